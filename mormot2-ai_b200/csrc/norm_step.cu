// The step from one sublayer to the next in a layer that norms both what a sublayer reads and
// what it gives back:
//     x[t] += N_out(y[t])           the sublayer's output y, normed, joins the residual
//     h[t]  = N_in(x[t])            and the next sublayer reads the residual, normed
// in one pass over the row. Either half may be missing: without y it is the norm of the residual
// (of the rows that `rows` names), without h it settles what is pending. y is the sum of `parts`
// float32 rows that may lie anywhere (a stored output, the split sums of a product, the rows of a
// token's experts), added up in order.
//
// A norm is one of two kinds, each with weights w and an optional bias b:
//     layer norm   (v - mean) / sqrt(var + eps) * w + b, var the mean of the squared deviations
//     RMS norm     v / sqrt(mean(v^2) + eps) * w + b
// Everything is float32; the variance takes a pass of its own over the row, which stays in
// registers (or in shared memory), so no sum of squares is ever reduced by one nearly as large.
#include "common.cuh"

MB_DEFINE_LAST_ERROR

struct NsNorm {
  const void* w;
  const void* b;      // or null
  int bf16;           // of w and b
  int layer;          // 1: layer norm, 0: RMS norm
  float eps;
};

// The sum over the block; every thread gets it. `red`: 32 floats that no other call of this kernel
// uses (so one barrier is enough).
__device__ __forceinline__ float ns_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  if (lane == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  return warp_sum(lane < warps ? red[lane] : 0.f);
}

// What a norm takes off a value (`off`) and multiplies it by (`inv`): `sum` of the values, or of
// their squares, is formed by the caller's function of an offset.
template <typename F>
__device__ __forceinline__ void ns_scale(const NsNorm& norm, int H, float* red, float& off,
                                         float& inv, F sum) {
  off = norm.layer ? ns_sum(sum(false, 0.f), red) / (float)H : 0.f;
  inv = 1.0f / sqrtf(ns_sum(sum(true, off), red + 32) / (float)H + norm.eps);
}

__device__ __forceinline__ float4 ns_load4(const void* p, int bf16, int c) {
  return bf16 ? load4<__nv_bfloat16>((const __nv_bfloat16*)p + c) : *(const float4*)((const float*)p + c);
}
__device__ __forceinline__ float ns_load1(const void* p, int bf16, int c) {
  return bf16 ? __bfloat162float(((const __nv_bfloat16*)p)[c]) : ((const float*)p)[c];
}

__device__ __forceinline__ float4 ns_apply4(float4 v, float off, float inv, float4 w, float4 b) {
  return make_float4(fmaf((v.x - off) * inv, w.x, b.x), fmaf((v.y - off) * inv, w.y, b.y),
                     fmaf((v.z - off) * inv, w.z, b.z), fmaf((v.w - off) * inv, w.w, b.w));
}

__device__ __forceinline__ float4 ns_apply4(float4 v, float off, float inv, const NsNorm& n, int c) {
  float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
  if (n.b) b = ns_load4(n.b, n.bf16, c);
  return ns_apply4(v, off, inv, ns_load4(n.w, n.bf16, c), b);
}

// The sum of a thread's 4 * VEC values (those inside the row), or of their squared distances from
// `off`
template <int VEC, int THREADS>
__device__ __forceinline__ float ns_mine(const float4* v, int H, bool squares, float off) {
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    if ((i * THREADS + (int)threadIdx.x) * 4 >= H) continue;
    if (squares) {
      const float a = v[i].x - off, b = v[i].y - off, c = v[i].z - off, d = v[i].w - off;
      t = fmaf(a, a, fmaf(b, b, fmaf(c, c, fmaf(d, d, t))));
    } else {
      t += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    }
  }
  return t;
}

// Rows of at most 4 * THREADS * VEC values (a multiple of 4, everything on 16-byte boundaries).
// FLAT: y has at most that many parts (0: any number), whose loads are all asked for at once.
template <typename TO, int VEC, int THREADS, int FLAT>
__global__ void __launch_bounds__(THREADS, THREADS <= 256 ? 4 : 1)
norm_step_vec_kernel(float* __restrict__ x, const float* __restrict__ y, int parts,
                     size_t part_stride, size_t row_stride, const __grid_constant__ NsNorm out_norm,
                     const __grid_constant__ NsNorm in_norm, TO* __restrict__ h,
                     const int* __restrict__ rows, int H) {
  __shared__ float red[2][64];
  const int r = blockIdx.x;
  float4 xv[VEC];
  // short rows a thread: the weights of both norms ahead of the wait too
  constexpr bool EARLY = VEC == 1 && FLAT > 0 && FLAT <= 4;
  float4 ow, ob, iw, ib;
  ow = ob = iw = ib = make_float4(0.f, 0.f, 0.f, 0.f);
  if (EARLY && (int)threadIdx.x * 4 < H) {
    const int c = threadIdx.x * 4;
    if (y != nullptr) {
      ow = ns_load4(out_norm.w, out_norm.bf16, c);
      if (out_norm.b) ob = ns_load4(out_norm.b, out_norm.bf16, c);
    }
    if (h != nullptr) {
      iw = ns_load4(in_norm.w, in_norm.bf16, c);
      if (in_norm.b) ib = ns_load4(in_norm.b, in_norm.bf16, c);
    }
  }
  // with a sublayer's output, the kernel before this one wrote that and nothing else: the
  // residual row can be asked for ahead of the wait
  const float* xr0 = x + (size_t)r * H;
  if (y != nullptr) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int c = (i * THREADS + threadIdx.x) * 4;
      xv[i] = c < H ? *(const float4*)(xr0 + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  mb_grid_wait();
  mb_grid_launch_next();
  float* xr = x + (size_t)(rows ? rows[r] : r) * H;
  if (y != nullptr) {
    float4 v[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int c = (i * THREADS + threadIdx.x) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c >= H) continue;
      const float* pp = y + (size_t)r * row_stride + c;
      if (FLAT > 0) {
        float4 a[FLAT > 0 ? FLAT : 1];
#pragma unroll
        for (int j = 0; j < FLAT; ++j)
          if (j < parts) a[j] = __ldg((const float4*)(pp + (size_t)j * part_stride));
#pragma unroll
        for (int j = 0; j < FLAT; ++j)
          if (j < parts) { v[i].x += a[j].x; v[i].y += a[j].y; v[i].z += a[j].z; v[i].w += a[j].w; }
        continue;
      }
      for (int p0 = 0; p0 < parts; p0 += 8) {      // up to eight loads in flight
        float4 a[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (p0 + j < parts) a[j] = __ldg((const float4*)(pp + (size_t)(p0 + j) * part_stride));
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (p0 + j < parts) { v[i].x += a[j].x; v[i].y += a[j].y; v[i].z += a[j].z; v[i].w += a[j].w; }
      }
    }
    float off, inv;
    ns_scale(out_norm, H, red[0], off, inv,
             [&](bool sq, float o) { return ns_mine<VEC, THREADS>(v, H, sq, o); });
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int c = (i * THREADS + threadIdx.x) * 4;
      if (c >= H) continue;
      const float4 n = EARLY ? ns_apply4(v[i], off, inv, ow, ob) : ns_apply4(v[i], off, inv, out_norm, c);
      xv[i].x += n.x; xv[i].y += n.y; xv[i].z += n.z; xv[i].w += n.w;
      *(float4*)(xr + c) = xv[i];
    }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int c = (i * THREADS + threadIdx.x) * 4;
      xv[i] = c < H ? *(const float4*)(xr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  if (h == nullptr) return;
  float off, inv;
  ns_scale(in_norm, H, red[1], off, inv,
           [&](bool sq, float o) { return ns_mine<VEC, THREADS>(xv, H, sq, o); });
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int c = (i * THREADS + threadIdx.x) * 4;
    if (c < H)
      store4<TO>(h + (size_t)r * H + c, EARLY ? ns_apply4(xv[i], off, inv, iw, ib)
                                              : ns_apply4(xv[i], off, inv, in_norm, c));
  }
}

// The same for any row: one value at a time, the row kept in shared memory.
template <typename TO>
__global__ void __launch_bounds__(256)
norm_step_kernel(float* __restrict__ x, const float* __restrict__ y, int parts, size_t part_stride,
                 size_t row_stride, const __grid_constant__ NsNorm out_norm,
                 const __grid_constant__ NsNorm in_norm, TO* __restrict__ h,
                 const int* __restrict__ rows, int H) {
  mb_grid_wait();
  mb_grid_launch_next();
  __shared__ float red[2][64];
  extern __shared__ float ns_row[];   // H values
  const int r = blockIdx.x;
  float* xr = x + (size_t)(rows ? rows[r] : r) * H;
  // a thread only ever reads the places of the row that it wrote
  auto sum = [&](bool squares, float o) {
    float t = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
      const float d = ns_row[c] - o;
      t = squares ? fmaf(d, d, t) : t + d;
    }
    return t;
  };
  float off, inv;
  if (y != nullptr) {
    for (int c = threadIdx.x; c < H; c += blockDim.x)
      ns_row[c] = sum_parts(y + (size_t)r * row_stride + c, parts, part_stride);
    ns_scale(out_norm, H, red[0], off, inv, sum);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
      const float b = out_norm.b ? ns_load1(out_norm.b, out_norm.bf16, c) : 0.f;
      const float v = xr[c] + fmaf((ns_row[c] - off) * inv, ns_load1(out_norm.w, out_norm.bf16, c), b);
      xr[c] = v;
      ns_row[c] = v;
    }
  } else {
    for (int c = threadIdx.x; c < H; c += blockDim.x) ns_row[c] = xr[c];
  }
  if (h == nullptr) return;
  ns_scale(in_norm, H, red[1], off, inv, sum);
  for (int c = threadIdx.x; c < H; c += blockDim.x) {
    const float b = in_norm.b ? ns_load1(in_norm.b, in_norm.bf16, c) : 0.f;
    h[(size_t)r * H + c] =
        from_f32<TO>(fmaf((ns_row[c] - off) * inv, ns_load1(in_norm.w, in_norm.bf16, c), b));
  }
}

template <typename TO>
static int norm_step_launch(float* x, const float* y, int parts, size_t part_stride,
                            size_t row_stride, const NsNorm& on, const NsNorm& in, void* h,
                            const int* rows, int R, int H, cudaStream_t s) {
  const uintptr_t bits = (uintptr_t)x | (uintptr_t)y | (uintptr_t)on.w | (uintptr_t)on.b |
                         (uintptr_t)in.w | (uintptr_t)in.b | (uintptr_t)h;
  if (H % 4 == 0 && H <= 4 * 1024 * 4 && (bits & 15) == 0 && ((part_stride | row_stride) & 3) == 0) {
#define NS_GO_F(V_, T_, F_)                                                                    \
  mb_launch(norm_step_vec_kernel<TO, V_, T_, F_>, dim3(R), dim3(T_), 0, s, x, y, parts,        \
            part_stride, row_stride, on, in, (TO*)h, rows, H)
#define NS_GO(V_, T_)                                                                          \
  {                                                                                            \
    if (parts <= 2) NS_GO_F(V_, T_, 2);                                                        \
    else if (parts <= 4) NS_GO_F(V_, T_, 4);                                                   \
    else if (V_ == 1 && parts <= 8) NS_GO_F(V_, T_, (V_ == 1 ? 8 : 0));                        \
    else NS_GO_F(V_, T_, 0);                                                                   \
  }
    // few rows (a decode step): as many threads a row as it has groups of four values, so that a
    // thread waits for few loads; many rows: 256 threads a row and more rows per SM
    if ((R <= 256 && H > 1024) || H > 4 * 256 * 4) {
      const int vec = (H + 4 * 1024 - 1) / (4 * 1024);
      if (vec <= 1) { if (H <= 2048) NS_GO(1, 512) else NS_GO(1, 1024) }
      else if (vec <= 2) NS_GO(2, 1024)
      else NS_GO(4, 1024)
    } else {
      const int vec = (H + 4 * 256 - 1) / (4 * 256);
      if (vec <= 1) { if (H <= 512) NS_GO(1, 128) else NS_GO(1, 256) }
      else if (vec <= 2) NS_GO(2, 256)
      else NS_GO(4, 256)
    }
#undef NS_GO
#undef NS_GO_F
    MB_CHECK_LAUNCH("mb_norm_step");
  }
  const size_t smem = (size_t)H * sizeof(float);
  static size_t configured = 47 * 1024;   // beside the kernel's static shared memory
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(norm_step_kernel<TO>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) MB_FAIL("mb_norm_step: a row of %d values: %s", H, cudaGetErrorString(e));
    configured = 200 * 1024;
  }
  mb_launch(norm_step_kernel<TO>, dim3(R), dim3(256), smem, s, x, y, parts, part_stride, row_stride,
            on, in, (TO*)h, rows, H);
  MB_CHECK_LAUNCH("mb_norm_step");
}

// x [T, H] float32; y (or null): `parts` rows a token at y + p * part_stride + t * row_stride; h
// (or null): [R, H]. Norms: weights, bias (or null), their type, layer norm (1) or RMS norm (0).
// rows [R] (or null: R = T rows in order) only without y.
MB_EXPORT int mb_norm_step(float* x, const float* y, int parts, long long part_stride,
                           long long row_stride, const void* out_w, const void* out_b,
                           int out_bf16, int out_layer, float out_eps, const void* in_w,
                           const void* in_b, int in_bf16, int in_layer, float in_eps, void* h,
                           int h_dtype, const int* rows, int R, int H, void* stream) {
  if (R <= 0) return 0;
  if (y == nullptr && h == nullptr) return 0;
  if (y != nullptr && (rows != nullptr || parts < 1 || out_w == nullptr))
    MB_FAIL("mb_norm_step: a sublayer's output of %d parts%s%s", parts,
            rows ? " with a row gather" : "", out_w ? "" : " without a norm");
  if (h != nullptr && in_w == nullptr) MB_FAIL("mb_norm_step: an operand without a norm");
  if ((size_t)H * sizeof(float) > 200 * 1024) MB_FAIL("mb_norm_step: rows of %d values", H);
  const NsNorm on = {out_w, out_b, out_bf16, out_layer, out_eps};
  const NsNorm in = {in_w, in_b, in_bf16, in_layer, in_eps};
  cudaStream_t s = (cudaStream_t)stream;
  if (h_dtype == MB_F32)
    return norm_step_launch<float>(x, y, parts, (size_t)part_stride, (size_t)row_stride, on, in, h,
                                   rows, R, H, s);
  return norm_step_launch<__nv_bfloat16>(x, y, parts, (size_t)part_stride, (size_t)row_stride, on,
                                         in, h, rows, R, H, s);
}
