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
// Everything is float32. A row's mean and squared deviations are formed in one reduction: every
// thread has its values' mean and their squared deviations from it, and two such triples
// (count, mean, deviations) merge exactly into that of both (Chan, Golub and LeVeque's pairwise
// update), so no sum of squares is ever reduced by a mean that nearly equals it.
#include "common.cuh"

MB_DEFINE_LAST_ERROR

struct NsNorm {
  const void* w;
  const void* b;      // or null
  int bf16;           // of w and b
  int layer;          // 1: layer norm, 0: RMS norm
  float eps;
};

struct NsMoments {
  float n, mean, dev;
};

__device__ __forceinline__ NsMoments ns_merge(const NsMoments& a, const NsMoments& b) {
  NsMoments m;
  m.n = a.n + b.n;
  const float share = m.n > 0.f ? b.n / m.n : 0.f, d = b.mean - a.mean;
  m.mean = fmaf(d, share, a.mean);
  m.dev = a.dev + b.dev + d * d * a.n * share;
  return m;
}

__device__ __forceinline__ NsMoments ns_warp(NsMoments m) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    NsMoments other;
    other.n = __shfl_down_sync(0xffffffffu, m.n, o);
    other.mean = __shfl_down_sync(0xffffffffu, m.mean, o);
    other.dev = __shfl_down_sync(0xffffffffu, m.dev, o);
    m = ns_merge(m, other);
  }
  return m;   // lane 0's is the warp's
}

// The moments of the whole block's values; every thread gets them. `red`: 3 x 32 floats that no
// other call of this kernel uses.
__device__ __forceinline__ NsMoments ns_block(NsMoments m, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
  m = ns_warp(m);
  if (lane == 0) {
    red[warp] = m.n;
    red[32 + warp] = m.mean;
    red[64 + warp] = m.dev;
  }
  __syncthreads();
  m.n = lane < warps ? red[lane] : 0.f;
  m.mean = lane < warps ? red[32 + lane] : 0.f;
  m.dev = lane < warps ? red[64 + lane] : 0.f;
  m = ns_warp(m);
  m.n = __shfl_sync(0xffffffffu, m.n, 0);
  m.mean = __shfl_sync(0xffffffffu, m.mean, 0);
  m.dev = __shfl_sync(0xffffffffu, m.dev, 0);
  return m;
}

// What a norm takes off a value and multiplies it by
__device__ __forceinline__ void ns_scale(const NsNorm& norm, const NsMoments& m, int H, float& off,
                                         float& inv) {
  const float var = m.dev / (float)H;
  off = norm.layer ? m.mean : 0.f;
  inv = 1.0f / sqrtf((norm.layer ? var : fmaf(m.mean, m.mean, var)) + norm.eps);
}

__device__ __forceinline__ float4 ns_load4(const void* p, int bf16, int c) {
  return bf16 ? load4<__nv_bfloat16>((const __nv_bfloat16*)p + c) : *(const float4*)((const float*)p + c);
}
__device__ __forceinline__ float ns_load1(const void* p, int bf16, int c) {
  return bf16 ? __bfloat162float(((const __nv_bfloat16*)p)[c]) : ((const float*)p)[c];
}

__device__ __forceinline__ float4 ns_apply4(float4 v, float off, float inv, const NsNorm& n, int c) {
  const float4 w = ns_load4(n.w, n.bf16, c);
  float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
  if (n.b) b = ns_load4(n.b, n.bf16, c);
  return make_float4(fmaf((v.x - off) * inv, w.x, b.x), fmaf((v.y - off) * inv, w.y, b.y),
                     fmaf((v.z - off) * inv, w.z, b.z), fmaf((v.w - off) * inv, w.w, b.w));
}

// The moments of a thread's 4 * VEC values (those inside the row)
template <int VEC, int THREADS>
__device__ __forceinline__ NsMoments ns_mine(const float4* v, int H) {
  NsMoments m = {0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    if ((i * THREADS + (int)threadIdx.x) * 4 >= H) continue;
    m.n += 4.f;
    m.mean += (v[i].x + v[i].y) + (v[i].z + v[i].w);
  }
  if (m.n > 0.f) m.mean /= m.n;
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    if ((i * THREADS + (int)threadIdx.x) * 4 >= H) continue;
    const float a = v[i].x - m.mean, b = v[i].y - m.mean, c = v[i].z - m.mean, d = v[i].w - m.mean;
    m.dev = fmaf(a, a, fmaf(b, b, fmaf(c, c, fmaf(d, d, m.dev))));
  }
  return m;
}

// Rows of at most 4 * THREADS * VEC values (a multiple of 4, everything on 16-byte boundaries).
template <typename TO, int VEC, int THREADS>
__global__ void __launch_bounds__(THREADS)
norm_step_vec_kernel(float* __restrict__ x, const float* __restrict__ y, int parts,
                     size_t part_stride, size_t row_stride, const __grid_constant__ NsNorm out_norm,
                     const __grid_constant__ NsNorm in_norm, TO* __restrict__ h,
                     const int* __restrict__ rows, int H) {
  __shared__ float red[2][96];
  const int r = blockIdx.x;
  float4 xv[VEC];
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
    ns_scale(out_norm, ns_block(ns_mine<VEC, THREADS>(v, H), red[0]), H, off, inv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int c = (i * THREADS + threadIdx.x) * 4;
      if (c >= H) continue;
      const float4 n = ns_apply4(v[i], off, inv, out_norm, c);
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
  ns_scale(in_norm, ns_block(ns_mine<VEC, THREADS>(xv, H), red[1]), H, off, inv);
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int c = (i * THREADS + threadIdx.x) * 4;
    if (c < H) store4<TO>(h + (size_t)r * H + c, ns_apply4(xv[i], off, inv, in_norm, c));
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
  __shared__ float red[2][96];
  extern __shared__ float ns_row[];   // H values
  const int r = blockIdx.x;
  float* xr = x + (size_t)(rows ? rows[r] : r) * H;
  // a thread only ever reads the places of the row that it wrote
  auto moments = [&](float* buf) {
    NsMoments m = {0.f, 0.f, 0.f};
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
      const NsMoments one = {1.f, ns_row[c], 0.f};
      m = ns_merge(m, one);
    }
    return ns_block(m, buf);
  };
  float off, inv;
  if (y != nullptr) {
    for (int c = threadIdx.x; c < H; c += blockDim.x)
      ns_row[c] = sum_parts(y + (size_t)r * row_stride + c, parts, part_stride);
    ns_scale(out_norm, moments(red[0]), H, off, inv);
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
  ns_scale(in_norm, moments(red[1]), H, off, inv);
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
#define NS_GO(V_, T_)                                                                          \
  mb_launch(norm_step_vec_kernel<TO, V_, T_>, dim3(R), dim3(T_), 0, s, x, y, parts,            \
            part_stride, row_stride, on, in, (TO*)h, rows, H)
    // few rows (a decode step): as many threads a row as it has groups of four values, so that a
    // thread waits for few loads; many rows: 256 threads a row and more rows per SM
    if ((R <= 256 && H > 1024) || H > 4 * 256 * 4) {
      const int vec = (H + 4 * 1024 - 1) / (4 * 1024);
      if (vec <= 1) { if (H <= 2048) NS_GO(1, 512); else NS_GO(1, 1024); }
      else if (vec <= 2) { NS_GO(2, 1024); }
      else { NS_GO(4, 1024); }
    } else {
      const int vec = (H + 4 * 256 - 1) / (4 * 256);
      if (vec <= 1) { if (H <= 512) NS_GO(1, 128); else NS_GO(1, 256); }
      else if (vec <= 2) { NS_GO(2, 256); }
      else { NS_GO(4, 256); }
    }
#undef NS_GO
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
