// Per-head RMSNorm of q and k, rotary position encoding, and the write of k and v into the
// paged cache, in one kernel after the fused q/k/v product, for float32 and bfloat16
// activations; sums, norms and angles are float32 in both.
//
// Formulas as the reference computes them (paths within the reference project):
//   q/k norm + RoPE + cache store   tools/cuda/ops.cu:211-314,
//             angles src/infer/mormot.ai.infer.decoder.pas:2539-2561
#include "common.cuh"

MB_DEFINE_LAST_ERROR

// a norm weight that is float32 or bfloat16 (the two fast kernels take either at run time)
__device__ __forceinline__ float norm_w(const void* w, int w_bf16, int i) {
  return w_bf16 ? __bfloat162float(((const __nv_bfloat16*)w)[i]) : ((const float*)w)[i];
}

// qkv [T, (nh + nkv) hd + nkv vd]: q heads, then k heads, then v heads (of vd values each) of a
// token. One warp per
// (token, head): RMSNorm over the head with q_norm / k_norm (null: no norm), rotate_half over
// the first rot_dim values with angle = f32(inv_freq[i] * pos), q written back in place, k and
// v (when write_kv) stored in the cache at the token's slot and position. `ld`: the row pitch
// of qkv (columns behind the heads belong to someone else). `unit_after`: instead of a weighted
// norm before the rotation, q and k are divided by their root mean square after it.
#define QK_WARPS 4
template <typename T, typename TW>
__global__ void qk_norm_rope_store_kernel(
    T* __restrict__ qkv, const TW* __restrict__ q_norm, const TW* __restrict__ k_norm, float eps,
    const float* __restrict__ inv_freq, int rot_dim, const int* __restrict__ tok_slot,
    const int* __restrict__ tok_pos,
    const int* __restrict__ page_table, int max_pages, int ring_pages, T* __restrict__ kpool,
    T* __restrict__ vpool, int nh, int nkv, int hd, int write_kv, int vd, int ld,
    int unit_after) {
  mb_grid_wait();
  mb_grid_launch_next();
  extern __shared__ float heads[];  // QK_WARPS x hd
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int head = blockIdx.y * QK_WARPS + warp;
  const int total = nh + 2 * nkv;
  if (head >= total) return;
  const bool is_q = head < nh, is_k = !is_q && head < nh + nkv;
  if (!is_q && !write_kv) return;
  T* src = qkv + (size_t)t * ld +
           (head < nh + nkv ? (size_t)head * hd
                            : (size_t)(nh + nkv) * hd + (size_t)(head - nh - nkv) * vd);
  float* buf = heads + warp * hd;
  const int pos = tok_pos[t];
  T* dst = src;
  if (!is_q) {
    const int g = is_k ? head - nh : head - nh - nkv;
    const size_t row = kv_row(page_table, max_pages, ring_pages, tok_slot[t], pos, nkv, g);
    if (!is_k) {  // values are stored as they are
      dst = vpool + row * vd;
      for (int i = lane; i < vd; i += 32) dst[i] = src[i];
      return;
    }
    dst = kpool + row * hd;
  }
  const TW* w = is_q ? q_norm : k_norm;
  float sum = 0.f;
  for (int i = lane; i < hd; i += 32) {
    const float v = to_f32<T>(src[i]);
    buf[i] = v;
    sum = fmaf(v, v, sum);
  }
  sum = warp_sum(sum);
  if (w && !unit_after) {
    const float inv = 1.0f / sqrtf(sum / (float)hd + eps);
    for (int i = lane; i < hd; i += 32) buf[i] = to_f32<TW>(w[i]) * (buf[i] * inv);
  }
  __syncwarp();
  const int half = rot_dim >> 1;
  float after = 0.f;   // the sum of squares of the head as it is after the rotation
  for (int i = lane; i < hd; i += 32) {
    float v = buf[i];
    if (i < rot_dim) {
      const int f = i < half ? i : i - half;
      const float angle = inv_freq[f] * (float)pos;  // float32 product, as the reference
      const float c = cosf(angle), s = sinf(angle);
      v = i < half ? buf[i] * c - buf[i + half] * s : buf[i] * c + buf[i - half] * s;
    }
    if (unit_after) after = fmaf(v, v, after);
    else dst[i] = from_f32<T>(v);
  }
  if (!unit_after) return;
  // the head over its root mean square, formed after the rotation, without a weight: the
  // rotated values are formed once more (buf still holds the unrotated head)
  const float inv = 1.0f / sqrtf(warp_sum(after) / (float)hd + eps);
  for (int i = lane; i < hd; i += 32) {
    float v = buf[i];
    if (i < rot_dim) {
      const int f = i < half ? i : i - half;
      const float angle = inv_freq[f] * (float)pos;
      const float c = cosf(angle), s = sinf(angle);
      v = i < half ? buf[i] * c - buf[i + half] * s : buf[i] * c + buf[i - half] * s;
    }
    dst[i] = from_f32<T>(v * inv);
  }
}


// The same for bfloat16 heads of 64, 128 or 256 values that rotate as a whole, for steps of few
// tokens (as many small warps in flight as possible): one warp per (token, head), every lane holds V = hd / 64 neighbouring values of the first half and their
// rotation partners of the second half, so nothing goes through shared memory. The source is
// the fused qkv row, or (PARTIAL) the float32 partial sums of a split product
// [parts][T][width], which are added up here in split order. q goes to q_out [T, nh * hd] when
// given, else back in place.
template <int V, bool PARTIAL>
__global__ void __launch_bounds__(QK_WARPS * 32)
qk_narrow_kernel(__nv_bfloat16* __restrict__ qkv, const float* __restrict__ partial, int parts,
               size_t part_stride, __nv_bfloat16* __restrict__ q_out,
               const void* __restrict__ q_norm, const void* __restrict__ k_norm, int w_bf16,
               float eps,
               const float* __restrict__ inv_freq, const int* __restrict__ tok_slot,
               const int* __restrict__ tok_pos,
               const int* __restrict__ page_table, int max_pages, int ring_pages,
               __nv_bfloat16* __restrict__ kpool, __nv_bfloat16* __restrict__ vpool, int nh,
               int nkv, int write_kv, int ld, int unit_after) {
  MB_TRACE_BEGIN();
  constexpr int HD = 64 * V, HALF = 32 * V;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int head = blockIdx.y * QK_WARPS + warp;
  const int total = nh + 2 * nkv;
  const bool is_q = head < nh, is_k = !is_q && head < nh + nkv;
  const bool live = head < total && (is_q || write_kv);
  const size_t col = (size_t)head * HD + V * lane;
  // Before the wait for the kernel before (which wrote the values of q, k and v, nothing
  // else): everything that does not depend on them. The token's position and slot, the page
  // table, the norm weights and the frequencies were settled by kernels further back, which
  // are complete once this kernel runs (every kernel of the stream waits for the one before it
  // ahead of letting its successor start). So the only loads after the wait are the values.
  __nv_bfloat16* dst = nullptr;
  float wa[V], wb[V], sn[V], cs[V];
  bool normed = false;
  if (live) {
    const int pos = tok_pos[t];
    if (is_q) {
      dst = q_out ? q_out + (size_t)t * nh * HD + col : qkv + (size_t)t * ld + col;
    } else {
      const int g = is_k ? head - nh : head - nh - nkv;
      const size_t row = kv_row(page_table, max_pages, ring_pages, tok_slot[t], pos, nkv, g);
      dst = (is_k ? kpool : vpool) + row * HD + V * lane;
    }
    if (is_q || is_k) {
      const void* w = is_q ? q_norm : k_norm;
      normed = w != nullptr && !unit_after;
#pragma unroll
      for (int j = 0; j < V; ++j) {
        wa[j] = normed ? norm_w(w, w_bf16, V * lane + j) : 1.f;
        wb[j] = normed ? norm_w(w, w_bf16, HALF + V * lane + j) : 1.f;
        const float angle = inv_freq[V * lane + j] * (float)pos;  // float32 product
        sincosf(angle, &sn[j], &cs[j]);
      }
    }
  }
  mb_grid_wait();
  mb_grid_launch_next();
  if (!live) return;
  float a[V], b[V];
  if (PARTIAL) {
    const float* src0 = partial + (size_t)t * ld + col;
    // up to eight parts asked for at once, then added in split order
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = b[j] = 0.f;
    for (int p0 = 0; p0 < parts; p0 += 8) {
      float pa[8][V], pb[8][V];
#pragma unroll
      for (int p = 0; p < 8; ++p) {
        const float* src = src0 + (size_t)(p0 + p) * part_stride;
#pragma unroll
        for (int j = 0; j < V; ++j) {
          pa[p][j] = p0 + p < parts ? __ldg(src + j) : 0.f;
          pb[p][j] = p0 + p < parts ? __ldg(src + HALF + j) : 0.f;
        }
      }
#pragma unroll
      for (int p = 0; p < 8; ++p)
#pragma unroll
        for (int j = 0; j < V; ++j) {
          a[j] += pa[p][j];
          b[j] += pb[p][j];
        }
    }
  } else {
    const __nv_bfloat16* src = qkv + (size_t)t * ld + col;
#pragma unroll
    for (int j = 0; j < V; ++j) {
      a[j] = __bfloat162float(src[j]);
      b[j] = __bfloat162float(src[HALF + j]);
    }
  }
  if (is_q || is_k) {
    if (normed) {
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < V; ++j) sum = fmaf(a[j], a[j], fmaf(b[j], b[j], sum));
      sum = warp_sum(sum);
      const float inv = 1.0f / sqrtf(sum / (float)HD + eps);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        a[j] = wa[j] * (a[j] * inv);
        b[j] = wb[j] * (b[j] * inv);
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float ra = a[j] * cs[j] - b[j] * sn[j], rb = b[j] * cs[j] + a[j] * sn[j];
      a[j] = ra;
      b[j] = rb;
    }
    if (unit_after) {   // over the root mean square of the rotated head, no weight
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < V; ++j) sum = fmaf(a[j], a[j], fmaf(b[j], b[j], sum));
      sum = warp_sum(sum);
      const float inv = 1.0f / sqrtf(sum / (float)HD + eps);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        a[j] *= inv;
        b[j] *= inv;
      }
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) {
    dst[j] = __float2bfloat16_rn(a[j]);
    dst[HALF + j] = __float2bfloat16_rn(b[j]);
  }
  MB_TRACE_END(3);  // by thread 0: warp 0's head is a q head, which is always live
}

// And for steps of many tokens, with 16-byte accesses: hd / 16 neighbouring lanes share a head, each holds eight neighbouring values of
// the first half and their rotation partners of the second half, so nothing goes through
// shared memory and a warp works on 512 / hd heads at once. A warp takes `passes` such groups
// of heads of its token one after another and forms the sines and cosines once. The source is
// the fused qkv row, or (PARTIAL) the float32 partial sums of a split product
// [parts][T][width], which are added up here in split order. q goes to q_out [T, nh * hd] when
// given, else back in place.
__device__ __forceinline__ void unpack8(const uint4& u, float* f) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 v = __bfloat1622float2(h[i]);
    f[2 * i] = v.x;
    f[2 * i + 1] = v.y;
  }
}
__device__ __forceinline__ uint4 pack8(const float* f) {
  uint4 u;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  return u;
}

#define QK_PASSES 3  // groups of heads that a warp of the wide form takes, at most
template <int HD, bool PARTIAL>
__global__ void __launch_bounds__(QK_WARPS * 32)
qk_wide_kernel(__nv_bfloat16* __restrict__ qkv, const float* __restrict__ partial, int parts,
               size_t part_stride, __nv_bfloat16* __restrict__ q_out,
               const void* __restrict__ q_norm, const void* __restrict__ k_norm, int w_bf16,
               float eps,
               const float* __restrict__ inv_freq, const int* __restrict__ tok_slot,
               const int* __restrict__ tok_pos,
               const int* __restrict__ page_table, int max_pages, int ring_pages,
               __nv_bfloat16* __restrict__ kpool, __nv_bfloat16* __restrict__ vpool, int nh,
               int nkv, int write_kv, int passes, int ld, int unit_after) {
  mb_grid_wait();
  mb_grid_launch_next();
  constexpr int HALF = HD / 2, L = HALF / 8, HPP = 32 / L;  // lanes a head, heads a pass
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sl = lane % L, hl = lane / L;
  const int t = blockIdx.x;
  const int total = nh + 2 * nkv;
  const int pos = tok_pos[t];
  const int group0 = (blockIdx.y * (blockDim.x >> 5) + warp) * passes;
  float cs[8], sn[8];
  bool have_angles = false;
  // every pass's values are asked for before the first pass is worked on: a pass's stores
  // may lie over the next one's source (q is rotated in place), so the compiler would not
  // move the loads up by itself, and three round trips to memory in a row would set the time
  uint4 raw[QK_PASSES][2];
  if (!PARTIAL) {
#pragma unroll
    for (int i = 0; i < QK_PASSES; ++i) {
      const int head = (group0 + i) * HPP + hl;
      raw[i][0] = raw[i][1] = make_uint4(0u, 0u, 0u, 0u);
      if (i < passes && head < total && (head < nh || write_kv)) {
        const __nv_bfloat16* src = qkv + (size_t)t * ld + (size_t)head * HD + 8 * sl;
        raw[i][0] = *reinterpret_cast<const uint4*>(src);
        raw[i][1] = *reinterpret_cast<const uint4*>(src + HALF);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < QK_PASSES; ++i) {
    if (i >= passes) break;
    const int head0 = (group0 + i) * HPP;
    if (head0 >= total) break;  // the whole warp
    const int head = head0 + hl;
    const bool is_q = head < nh, is_k = !is_q && head < nh + nkv;
    const bool live = head < total && (is_q || write_kv);
    const size_t col = (size_t)head * HD + 8 * sl;
    float a[8], b[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] = b[j] = 0.f;
    if (live) {
      if (PARTIAL) {
        const float* src0 = partial + (size_t)t * ld + col;
#pragma unroll 2
        for (int p = 0; p < parts; ++p) {
          const float4* sa = reinterpret_cast<const float4*>(src0 + (size_t)p * part_stride);
          const float4* sb = reinterpret_cast<const float4*>(src0 + (size_t)p * part_stride + HALF);
          const float4 a0 = __ldg(sa), a1 = __ldg(sa + 1), b0 = __ldg(sb), b1 = __ldg(sb + 1);
          a[0] += a0.x; a[1] += a0.y; a[2] += a0.z; a[3] += a0.w;
          a[4] += a1.x; a[5] += a1.y; a[6] += a1.z; a[7] += a1.w;
          b[0] += b0.x; b[1] += b0.y; b[2] += b0.z; b[3] += b0.w;
          b[4] += b1.x; b[5] += b1.y; b[6] += b1.z; b[7] += b1.w;
        }
      } else {
        unpack8(raw[i][0], a);
        unpack8(raw[i][1], b);
      }
    }
    if (head0 < nh + nkv) {  // some head of this pass is a q or k head (uniform over the warp)
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) sum = fmaf(a[j], a[j], fmaf(b[j], b[j], sum));
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (!have_angles) {
        // the lanes that hold the same eight columns of different heads share the work: each
        // forms 8 / HPP of the eight sines and cosines and hands them round
        constexpr int PER = 8 / HPP;
        float my_sn[PER], my_cs[PER];
#pragma unroll
        for (int r = 0; r < PER; ++r) {
          const float angle = inv_freq[8 * sl + hl * PER + r] * (float)pos;  // float32 product
          sincosf(angle, &my_sn[r], &my_cs[r]);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          sn[j] = __shfl_sync(0xffffffffu, my_sn[j % PER], (j / PER) * L + sl);
          cs[j] = __shfl_sync(0xffffffffu, my_cs[j % PER], (j / PER) * L + sl);
        }
        have_angles = true;
      }
      if (live && (is_q || is_k)) {
        const void* w = is_q ? q_norm : k_norm;
        if (w && !unit_after) {
          const float inv = 1.0f / sqrtf(sum / (float)HD + eps);
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            a[j] = norm_w(w, w_bf16, 8 * sl + j) * (a[j] * inv);
            b[j] = norm_w(w, w_bf16, HALF + 8 * sl + j) * (b[j] * inv);
          }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float ra = a[j] * cs[j] - b[j] * sn[j], rb = b[j] * cs[j] + a[j] * sn[j];
          a[j] = ra;
          b[j] = rb;
        }
      }
      if (unit_after) {   // over the root mean square of the rotated head, no weight
        float after = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) after = fmaf(a[j], a[j], fmaf(b[j], b[j], after));
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) after += __shfl_xor_sync(0xffffffffu, after, o);
        if (live && (is_q || is_k)) {
          const float inv = 1.0f / sqrtf(after / (float)HD + eps);
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            a[j] *= inv;
            b[j] *= inv;
          }
        }
      }
    }
    if (!live) continue;
    __nv_bfloat16* dst;
    if (is_q) {
      dst = q_out ? q_out + (size_t)t * nh * HD + col : qkv + (size_t)t * ld + col;
    } else {
      const int g = is_k ? head - nh : head - nh - nkv;
      const size_t row =
          kv_row(page_table, max_pages, ring_pages, tok_slot[t], pos, nkv, g);
      dst = (is_k ? kpool : vpool) + row * HD + 8 * sl;
    }
    *reinterpret_cast<uint4*>(dst) = pack8(a);
    *reinterpret_cast<uint4*>(dst + HALF) = pack8(b);
  }
}

// `partial` (may be null): float32 [parts][T][(nh + 2 nkv) hd] partial sums that stand for qkv
// (bfloat16 heads of 64/128/256 values that rotate as a whole only); `q_out` (may be null):
// where q goes instead of back into qkv, [T, nh * hd].
MB_EXPORT int mb_qk_norm_rope_store(void* qkv, const float* partial, int parts,
                                    long long part_stride, void* q_out, int dtype,
                                    const void* q_norm, const void* k_norm,
                                    int w_dtype, float eps, const float* inv_freq, int rot_dim,
                                    const int* tok_slot, const int* tok_pos,
                                    const int* page_table, int max_pages, int ring_pages,
                                    void* kpool, void* vpool, int T, int nh, int nkv, int hd,
                                    int write_kv, int vd, int ld, int unit_after,
                                    void* stream) {
  if (T <= 0) return 0;
  if (vd <= 0) vd = hd;
  const int width = (nh + nkv) * hd + nkv * vd;
  if (ld <= 0) ld = width;
  if (ld < width) MB_FAIL("mb_qk_norm_rope_store: a row pitch of %d for %d values", ld, width);
  if (rot_dim < 0 || rot_dim > hd || (rot_dim & 1))
    MB_FAIL("mb_qk_norm_rope_store: %d of %d values rotate", rot_dim, hd);
  if (hd <= 0 || hd > 1024) MB_FAIL("mb_qk_norm_rope_store: heads of %d", hd);
  cudaStream_t s = (cudaStream_t)stream;
  dim3 grid(T, (nh + 2 * nkv + QK_WARPS - 1) / QK_WARPS);
  const bool aligned = !(((uintptr_t)qkv | (uintptr_t)partial | (uintptr_t)q_out |
                          (uintptr_t)kpool | (uintptr_t)vpool) & 15) && (part_stride & 3) == 0;
  const bool fast = dtype == MB_BF16 && rot_dim == hd && (hd == 64 || hd == 128 || hd == 256) &&
                    aligned && vd == hd && ld % 8 == 0;
  if ((partial || q_out) && !fast)
    MB_FAIL("mb_qk_norm_rope_store: partial sums or a separate q for heads of %d values "
            "(%d rotate)%s are not supported", hd, rot_dim, aligned ? "" : ", not 16-byte aligned,");
  if (fast) {
    typedef __nv_bfloat16 bf;
    const int w_bf16 = w_dtype == MB_BF16;
    if (T < 512) {
#define QKN(V_, P_)                                                                            \
  mb_launch(qk_narrow_kernel<V_, P_>, grid, dim3(QK_WARPS * 32), 0, s, (bf*)qkv, partial,      \
      parts, (size_t)part_stride, (bf*)q_out, q_norm, k_norm, w_bf16, eps, inv_freq, tok_slot, \
      tok_pos, page_table, max_pages, ring_pages, (bf*)kpool, (bf*)vpool, nh, nkv,   \
      write_kv, ld, unit_after)
#define QKN_V(P_)                                                                              \
  if (hd == 64) QKN(1, P_); else if (hd == 128) QKN(2, P_); else QKN(4, P_)
      if (partial) { QKN_V(true); } else { QKN_V(false); }
#undef QKN_V
#undef QKN
      MB_CHECK_LAUNCH("mb_qk_norm_rope_store");
    }
    // groups of 512 / hd heads: blocks of four warps that take three groups each
    const int groups = ((nh + 2 * nkv) * hd + 511) / 512;
    const int warps = QK_WARPS, passes = QK_PASSES;
    dim3 fgrid(T, (groups + warps * passes - 1) / (warps * passes));
#define QKF(HD_, P_)                                                                           \
  mb_launch(qk_wide_kernel<HD_, P_>, fgrid, dim3(warps * 32), 0, s, (bf*)qkv, partial, parts,  \
      (size_t)part_stride, (bf*)q_out, q_norm, k_norm, w_bf16, eps, inv_freq, tok_slot,        \
      tok_pos, page_table, max_pages, ring_pages, (bf*)kpool, (bf*)vpool, nh, nkv,   \
      write_kv, passes, ld, unit_after)
#define QKF_V(P_)                                                                              \
  if (hd == 64) QKF(64, P_); else if (hd == 128) QKF(128, P_); else QKF(256, P_)
    if (partial) { QKF_V(true); } else { QKF_V(false); }
#undef QKF_V
#undef QKF
    MB_CHECK_LAUNCH("mb_qk_norm_rope_store");
  }
  const size_t smem = (size_t)QK_WARPS * hd * sizeof(float);
#define QK_LAUNCH(T_, TW_)                                                                     \
  mb_launch(qk_norm_rope_store_kernel<T_, TW_>, dim3(grid), dim3(QK_WARPS * 32), smem, s,                         \
      (T_*)qkv, (const TW_*)q_norm, (const TW_*)k_norm, eps, inv_freq, rot_dim, tok_slot,      \
      tok_pos, page_table, max_pages, ring_pages, (T_*)kpool, (T_*)vpool, nh, nkv,   \
      hd, write_kv, vd, ld, unit_after)
  if (dtype == MB_F32 && w_dtype == MB_F32) QK_LAUNCH(float, float);
  else if (dtype == MB_F32) QK_LAUNCH(float, __nv_bfloat16);
  else if (w_dtype == MB_F32) QK_LAUNCH(__nv_bfloat16, float);
  else QK_LAUNCH(__nv_bfloat16, __nv_bfloat16);
#undef QK_LAUNCH
  MB_CHECK_LAUNCH("mb_qk_norm_rope_store");
}


// ------------------------------------------------------------------ heads of several maps
// Rows [q | k | v] of a product (or its float32 split sums [parts][T][ld], added up in split
// order) for attention whose heads have `maps` queries and keys each: q holds nh * maps vectors
// of `dim`, k nkv * maps, v nkv of `vd`. A warp takes one vector at a time: the bias is added
// (float32, may be null), a map of q or k is normed (x / sqrt(mean(x^2) + eps) * w, one weight
// for all) and its first rot_dim values turn, pair (i, i + rot_dim / 2), cosine and sine times
// `amp`. q goes to q_out [T][nh * maps * dim]; the maps of a key head lie one after the other
// in the head's cache row of maps * dim values. A lane holds two neighbouring values of every
// 64 (PAIRS; the sizes and row pitches are then even) or one of every 32. A block takes
// `per_block` vectors of one token and forms the token's sines and cosines once.
#define MP_WARPS 4
#define MP_MAX 8    // rounds of a lane over a vector: 512 values in pairs, 256 single ones

template <typename T> __device__ __forceinline__ float2 load2(const T* p);
template <> __device__ __forceinline__ float2 load2<float>(const float* p) { return *(const float2*)p; }
template <> __device__ __forceinline__ float2 load2<__nv_bfloat16>(const __nv_bfloat16* p) {
  return __bfloat1622float2(*(const __nv_bfloat162*)p);
}
__device__ __forceinline__ void store2(float* p, float2 v) { *(float2*)p = v; }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float2 v) {
  *(__nv_bfloat162*)p = __floats2bfloat162_rn(v.x, v.y);
}

template <typename TI, typename TO, bool PAIRS>
__global__ void __launch_bounds__(MP_WARPS * 32)
maps_norm_rope_store_kernel(const TI* __restrict__ rows, int parts, size_t part_stride, int ld,
                            const float* __restrict__ bias, const float* __restrict__ q_norm,
                            const float* __restrict__ k_norm, float eps,
                            const float* __restrict__ inv_freq, int rot_dim, float amp,
                            const int* __restrict__ tok_slot, const int* __restrict__ tok_pos,
                            const int* __restrict__ page_table, int max_pages, int ring_pages,
                            TO* __restrict__ kpool, TO* __restrict__ vpool, TO* __restrict__ q_out,
                            int nh, int nkv, int maps, int dim, int vd, int per_block) {
  constexpr int PER = PAIRS ? 2 : 1, STEP = 32 * PER;
  extern __shared__ float mp_smem[];   // [rot_dim / 2] cosines, then sines, then [warps][dim]
  const int half = rot_dim >> 1;
  float* cs = mp_smem;
  float* sn = cs + half;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* buf = sn + half + warp * dim;
  const int t = blockIdx.x;
  // before the wait: what does not depend on the kernel before
  const int pos = tok_pos[t], slot = tok_slot[t];
  for (int i = threadIdx.x; i < half; i += MP_WARPS * 32) {
    float s, c;
    sincosf(inv_freq[i] * (float)pos, &s, &c);
    cs[i] = c * amp;
    sn[i] = s * amp;
  }
  __syncthreads();
  mb_grid_wait();
  mb_grid_launch_next();
  const int nq = nh * maps, nk = nkv * maps, total = nq + nk + nkv;
  const int first = blockIdx.y * per_block, last = min(first + per_block, total);
  for (int n = first + warp; n < last; n += MP_WARPS) {
    const bool is_q = n < nq, is_k = !is_q && n < nq + nk;
    const int size = is_q || is_k ? dim : vd;
    const int col = is_q || is_k ? n * dim : (nq + nk) * dim + (n - nq - nk) * vd;
    const TI* src = rows + (size_t)t * ld + col;
    float2 v[MP_MAX];
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < MP_MAX; ++j) {
      v[j] = make_float2(0.f, 0.f);
      const int i = STEP * j + PER * lane;
      if (i >= size) continue;
      for (int p0 = 0; p0 < parts; p0 += 8) {
        float2 a[8];
#pragma unroll
        for (int p = 0; p < 8; ++p) {
          if (p0 + p >= parts) continue;
          const TI* at = src + (size_t)(p0 + p) * part_stride + i;
          a[p] = PAIRS ? load2<TI>(at) : make_float2(to_f32<TI>(*at), 0.f);
        }
#pragma unroll
        for (int p = 0; p < 8; ++p)
          if (p0 + p < parts) { v[j].x += a[p].x; v[j].y += a[p].y; }
      }
      if (bias) {
        v[j].x += bias[col + i];
        if (PAIRS) v[j].y += bias[col + i + 1];
      }
      sum = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, sum));
    }
    TO* dst;
    if (is_q) {
      dst = q_out + (size_t)t * nq * dim + col;
    } else {
      const int m = n - nq, g = is_k ? m / maps : m - nk;
      const size_t row = kv_row(page_table, max_pages, ring_pages, slot, pos, nkv, g);
      dst = is_k ? kpool + (row * maps + (m - g * maps)) * dim : vpool + row * vd;
    }
    if (is_q || is_k) {
      const float* w = is_q ? q_norm : k_norm;
      const float inv = 1.0f / sqrtf(warp_sum(sum) / (float)dim + eps);
#pragma unroll
      for (int j = 0; j < MP_MAX; ++j) {
        const int i = STEP * j + PER * lane;
        if (i >= size) continue;
        v[j].x = w[i] * (v[j].x * inv);
        buf[i] = v[j].x;
        if (PAIRS) {
          v[j].y = w[i + 1] * (v[j].y * inv);
          buf[i + 1] = v[j].y;
        }
      }
      __syncwarp();
      auto turn = [&](int i, float x) {
        if (i >= rot_dim) return x;
        return i < half ? x * cs[i] - buf[i + half] * sn[i]
                        : x * cs[i - half] + buf[i - half] * sn[i - half];
      };
#pragma unroll
      for (int j = 0; j < MP_MAX; ++j) {
        const int i = STEP * j + PER * lane;
        if (i >= size) continue;
        v[j].x = turn(i, v[j].x);
        if (PAIRS) v[j].y = turn(i + 1, v[j].y);
      }
      __syncwarp();      // buf is written again by the warp's next vector
    }
#pragma unroll
    for (int j = 0; j < MP_MAX; ++j) {
      const int i = STEP * j + PER * lane;
      if (i >= size) continue;
      if (PAIRS) store2(dst + i, v[j]);
      else dst[i] = from_f32<TO>(v[j].x);
    }
  }
}

// The same for steps of many tokens, with 16-byte accesses: bfloat16 rows, maps of 64 or 128 values
// that rotate as a whole, value rows that are whole multiples of a map's size (taken as that
// many vectors). HD / 16 neighbouring lanes share a vector, each holds eight neighbouring values
// of the first half and their rotation partners of the second half; a warp works on 512 / HD
// vectors at once, takes up to QK_PASSES such groups of its token and forms the angles once.
template <int HD>
__global__ void __launch_bounds__(QK_WARPS * 32)
maps_wide_kernel(const __nv_bfloat16* __restrict__ rows, int ld, const float* __restrict__ bias,
                 const float* __restrict__ q_norm, const float* __restrict__ k_norm, float eps,
                 const float* __restrict__ inv_freq, float amp, const int* __restrict__ tok_slot,
                 const int* __restrict__ tok_pos, const int* __restrict__ page_table,
                 int max_pages, int ring_pages, __nv_bfloat16* __restrict__ kpool,
                 __nv_bfloat16* __restrict__ vpool, __nv_bfloat16* __restrict__ q_out, int nh,
                 int nkv, int maps, int vd) {
  constexpr int HALF = HD / 2, L = HALF / 8, HPP = 32 / L;  // lanes a vector, vectors a group
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sl = lane % L, hl = lane / L;
  const int t = blockIdx.x;
  const int nq = nh * maps, nk = nkv * maps, per_v = vd / HD, total = nq + nk + nkv * per_v;
  const int pos = tok_pos[t], slot = tok_slot[t];
  const int group0 = (blockIdx.y * QK_WARPS + warp) * QK_PASSES;
  // ahead of the wait: the angles (each lane that holds the same columns of another vector forms
  // 8 / HPP of the eight sines and cosines and hands them round)
  float cs[8], sn[8];
  {
    constexpr int PER = 8 / HPP > 0 ? 8 / HPP : 1;
    float my_sn[PER], my_cs[PER];
#pragma unroll
    for (int r = 0; r < PER; ++r) {
      const int f = 8 * sl + (hl * PER + r) % 8;
      sincosf(inv_freq[f] * (float)pos, &my_sn[r], &my_cs[r]);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      sn[j] = amp * __shfl_sync(0xffffffffu, my_sn[j % PER], (j / PER) * L + sl);
      cs[j] = amp * __shfl_sync(0xffffffffu, my_cs[j % PER], (j / PER) * L + sl);
    }
  }
  mb_grid_wait();
  mb_grid_launch_next();
  uint4 raw[QK_PASSES][2];       // every group's values are asked for before the first is worked on
#pragma unroll
  for (int i = 0; i < QK_PASSES; ++i) {
    const int n = (group0 + i) * HPP + hl;
    raw[i][0] = raw[i][1] = make_uint4(0u, 0u, 0u, 0u);
    if (n < total) {
      const __nv_bfloat16* src = rows + (size_t)t * ld + (size_t)n * HD + 8 * sl;
      raw[i][0] = *reinterpret_cast<const uint4*>(src);
      raw[i][1] = *reinterpret_cast<const uint4*>(src + HALF);
    }
  }
#pragma unroll
  for (int i = 0; i < QK_PASSES; ++i) {
    const int n0 = (group0 + i) * HPP, n = n0 + hl;
    if (n0 >= total) break;  // the whole warp
    const bool live = n < total, is_q = n < nq, is_k = !is_q && n < nq + nk;
    float a[8], b[8];
    unpack8(raw[i][0], a);
    unpack8(raw[i][1], b);
    if (bias && live) {
      const float* bp = bias + (size_t)n * HD + 8 * sl;
#pragma unroll
      for (int j = 0; j < 8; j += 4) {
        const float4 x = __ldg((const float4*)(bp + j)), y = __ldg((const float4*)(bp + HALF + j));
        a[j] += x.x; a[j + 1] += x.y; a[j + 2] += x.z; a[j + 3] += x.w;
        b[j] += y.x; b[j + 1] += y.y; b[j + 2] += y.z; b[j + 3] += y.w;
      }
    }
    if (n0 < nq + nk) {  // some vector of this group is a query or key (uniform over the warp)
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) sum = fmaf(a[j], a[j], fmaf(b[j], b[j], sum));
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (is_q || is_k) {
        const float* w = (is_q ? q_norm : k_norm) + 8 * sl;
        const float inv = 1.0f / sqrtf(sum / (float)HD + eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float x = __ldg(w + j) * (a[j] * inv), y = __ldg(w + HALF + j) * (b[j] * inv);
          a[j] = x * cs[j] - y * sn[j];
          b[j] = y * cs[j] + x * sn[j];
        }
      }
    }
    if (!live) continue;
    __nv_bfloat16* dst;
    if (is_q) {
      dst = q_out + ((size_t)t * nq + n) * HD;
    } else {
      const int m = is_k ? n - nq : n - nq - nk, per = is_k ? maps : per_v, g = m / per;
      const size_t row = kv_row(page_table, max_pages, ring_pages, slot, pos, nkv, g);
      dst = (is_k ? kpool : vpool) + (row * per + (m - g * per)) * HD;
    }
    *reinterpret_cast<uint4*>(dst + 8 * sl) = pack8(a);
    *reinterpret_cast<uint4*>(dst + 8 * sl + HALF) = pack8(b);
  }
}

MB_EXPORT int mb_maps_norm_rope_store(const void* rows, int in_dtype, int parts,
                                      long long part_stride, int ld, const float* bias,
                                      const float* q_norm, const float* k_norm, float eps,
                                      const float* inv_freq, int rot_dim, float amp,
                                      const int* tok_slot, const int* tok_pos,
                                      const int* page_table, int max_pages, int ring_pages,
                                      void* kpool, void* vpool, void* q_out, int dtype, int T,
                                      int nh, int nkv, int maps, int dim, int vd, void* stream) {
  if (T <= 0) return 0;
  if (rot_dim < 0 || rot_dim > dim || (rot_dim & 1))
    MB_FAIL("mb_maps_norm_rope_store: %d of %d values rotate", rot_dim, dim);
  if (nh <= 0 || nkv <= 0 || maps <= 0 || nh % nkv || parts < 1)
    MB_FAIL("mb_maps_norm_rope_store: %d heads on %d KV heads, %d maps, %d parts", nh, nkv, maps, parts);
  if (ld < (nh + nkv) * maps * dim + nkv * vd)
    MB_FAIL("mb_maps_norm_rope_store: a row pitch of %d", ld);
  if (in_dtype == MB_BF16 && dtype != MB_BF16)
    MB_FAIL("mb_maps_norm_rope_store: bfloat16 rows for float32 activations");
  const uintptr_t in_bytes = in_dtype == MB_F32 ? 8 : 4, out_bytes = dtype == MB_F32 ? 8 : 4;
  const bool pairs = !(dim & 1) && !(vd & 1) && !(ld & 1) && !(part_stride & 1) &&
                     ((uintptr_t)rows % in_bytes) == 0 &&
                     (((uintptr_t)kpool | (uintptr_t)vpool | (uintptr_t)q_out) % out_bytes) == 0;
  const int most = (pairs ? 64 : 32) * MP_MAX;
  if (dim <= 0 || vd <= 0 || dim > most || vd > most)
    MB_FAIL("mb_maps_norm_rope_store: vectors of %d and %d values (at most %d)", dim, vd, most);
  if (T >= 128 && in_dtype == MB_BF16 && dtype == MB_BF16 && parts == 1 &&
      (dim == 64 || dim == 128) && rot_dim == dim && vd % dim == 0 && ld % 8 == 0 &&
      (((uintptr_t)rows | (uintptr_t)kpool | (uintptr_t)vpool | (uintptr_t)q_out |
        (uintptr_t)bias) & 15) == 0) {
    typedef __nv_bfloat16 bf;
    const int vectors = (nh + nkv) * maps + nkv * (vd / dim), each = QK_WARPS * QK_PASSES * (512 / dim);
    dim3 wide(T, (vectors + each - 1) / each);
#define GOW(HD_)                                                                               \
  mb_launch(maps_wide_kernel<HD_>, wide, dim3(QK_WARPS * 32), 0, (cudaStream_t)stream,         \
            (const bf*)rows, ld, bias, q_norm, k_norm, eps, inv_freq, amp, tok_slot, tok_pos,  \
            page_table, max_pages, ring_pages, (bf*)kpool, (bf*)vpool, (bf*)q_out, nh, nkv,    \
            maps, vd)
    if (dim == 64) GOW(64); else GOW(128);
#undef GOW
    MB_CHECK_LAUNCH("mb_maps_norm_rope_store");
  }
  const size_t smem = (size_t)(rot_dim + MP_WARPS * dim) * sizeof(float);
  const int total = (nh + nkv) * maps + nkv;
  // few tokens: a vector a warp; many: four a warp, so that a block's angles serve sixteen
  const int per_block = T < 256 ? MP_WARPS : 4 * MP_WARPS;
  dim3 grid(T, (total + per_block - 1) / per_block);
  cudaStream_t s = (cudaStream_t)stream;
#define GO(TI_, TO_, P_)                                                                        \
  mb_launch(maps_norm_rope_store_kernel<TI_, TO_, P_>, grid, dim3(MP_WARPS * 32), smem, s,      \
            (const TI_*)rows, parts, (size_t)part_stride, ld, bias, q_norm, k_norm, eps,        \
            inv_freq, rot_dim, amp, tok_slot, tok_pos, page_table, max_pages, ring_pages,       \
            (TO_*)kpool, (TO_*)vpool, (TO_*)q_out, nh, nkv, maps, dim, vd, per_block)
#define GO_P(TI_, TO_) { if (pairs) GO(TI_, TO_, true); else GO(TI_, TO_, false); }
  if (dtype == MB_F32) GO_P(float, float)
  else if (in_dtype == MB_F32) GO_P(float, __nv_bfloat16)
  else GO_P(__nv_bfloat16, __nv_bfloat16)
#undef GO_P
#undef GO
  MB_CHECK_LAUNCH("mb_maps_norm_rope_store");
}

// ------------------------------------------------------------------ heads without a norm
// Rows [q | k | v | gates] of a product (or its float32 split sums [parts][T][ld], added up in
// split order) for attention that norms neither q nor k: the first rot_dim values of every q and k
// head turn, pair (i, i + rot_dim / 2), cosine and sine times `amp`; q goes to q_out (rows of q_ld
// values; it may be the product's row itself), k and v into the cache.
// `first` [T, nkv * vd] (or null) is what values are blended with across layers: without `lam` it
// receives this layer's values, with it (one float32 on the device) the values become
// (1 - lam) v + lam first before they are stored. `gate_out` (or null) [T, gate_n]: receives the
// gate_n columns behind v (of split sums; a product's own row is read where it lies).
// V neighbouring values a thread (8: everything on 16-byte boundaries; 1: any sizes).
template <typename T, int V> struct RsVec {
  static __device__ __forceinline__ void load(const T* p, float* v) {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = to_f32<T>(p[i]);
  }
  static __device__ __forceinline__ void store(T* p, const float* v) {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = from_f32<T>(v[i]);
  }
};
template <> struct RsVec<__nv_bfloat16, 8> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* v) {
    unpack8(*(const uint4*)p, v);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
    *(uint4*)p = pack8(v);
  }
};
template <> struct RsVec<float, 8> {
  static __device__ __forceinline__ void load(const float* p, float* v) {
    const float4 a = *(const float4*)p, b = *(const float4*)(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
    *(float4*)(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
};

template <typename TI, typename TO, int V>
__global__ void __launch_bounds__(256)
rope_store_kernel(const TI* rows, int parts, size_t part_stride, int ld,
                  const float* __restrict__ inv_freq, int rot_dim, float amp,
                  const int* __restrict__ tok_slot, const int* __restrict__ tok_pos,
                  const int* __restrict__ page_table, int max_pages, int ring_pages,
                  TO* __restrict__ kpool, TO* __restrict__ vpool, TO* q_out, int q_ld,
                  TO* __restrict__ first, const float* __restrict__ lam, TO* __restrict__ gate_out,
                  int gate_n, int nh, int nkv, int dim, int vd) {
  extern __shared__ float rs_angles[];   // [rot_dim / 2] cosines, then sines
  const int half = rot_dim >> 1;
  float* cs = rs_angles;
  float* sn = cs + half;
  const int t = blockIdx.x;
  // ahead of the wait: what does not depend on the kernel before
  const int pos = tok_pos[t], slot = tok_slot[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(inv_freq[i] * (float)pos, &s, &c);
    cs[i] = c * amp;
    sn[i] = s * amp;
  }
  const float l = lam ? *lam : 0.f;
  __syncthreads();
  mb_grid_wait();
  mb_grid_launch_next();
  const TI* row = rows + (size_t)t * ld;
  auto read = [&](int col, float* v) {
    RsVec<TI, V>::load(row + col, v);
    for (int p = 1; p < parts; ++p) {
      float a[V];
      RsVec<TI, V>::load(row + (size_t)p * part_stride + col, a);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] += a[i];
    }
  };
  // a head of q or k: pairs of V values that turn together, then V values at a time that pass
  const int pairs = half / V, per_head = pairs + (dim - rot_dim) / V;
  const int n_heads = (nh + nkv) * per_head, per_v = vd / V, n_v = nkv * per_v;
  const int total = n_heads + n_v + (gate_out ? gate_n / V : 0);
  for (int n = blockIdx.y * blockDim.x + threadIdx.x; n < total; n += gridDim.y * blockDim.x) {
    if (n < n_heads) {
      const int head = n / per_head, i = n - head * per_head;
      TO* dst;
      if (head < nh) {
        dst = q_out + (size_t)t * q_ld + (size_t)head * dim;
      } else {
        dst = kpool + kv_row(page_table, max_pages, ring_pages, slot, pos, nkv, head - nh) * dim;
      }
      float a[V];
      if (i < pairs) {
        float b[V];
        read(head * dim + i * V, a);
        read(head * dim + half + i * V, b);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          const float c = cs[i * V + j], s = sn[i * V + j], u = a[j], w = b[j];
          a[j] = u * c - w * s;
          b[j] = w * c + u * s;
        }
        RsVec<TO, V>::store(dst + i * V, a);
        RsVec<TO, V>::store(dst + half + i * V, b);
      } else {
        const int at = rot_dim + (i - pairs) * V;
        read(head * dim + at, a);
        RsVec<TO, V>::store(dst + at, a);
      }
    } else if (n < n_heads + n_v) {
      const int m = n - n_heads, g = m / per_v, at = (m - g * per_v) * V;
      float v[V];
      read((nh + nkv) * dim + g * vd + at, v);
      if (first) {
        TO* f = first + ((size_t)t * nkv + g) * vd + at;
        if (lam) {
          float o[V];
          RsVec<TO, V>::load(f, o);
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = (1.0f - l) * v[j] + l * o[j];
        } else {
          RsVec<TO, V>::store(f, v);
        }
      }
      RsVec<TO, V>::store(
          vpool + kv_row(page_table, max_pages, ring_pages, slot, pos, nkv, g) * vd + at, v);
    } else {
      const int at = (n - n_heads - n_v) * V;
      float v[V];
      read((nh + nkv) * dim + nkv * vd + at, v);
      RsVec<TO, V>::store(gate_out + (size_t)t * gate_n + at, v);
    }
  }
}

MB_EXPORT int mb_rope_store(const void* rows, int in_dtype, int parts, long long part_stride, int ld,
                            const float* inv_freq, int rot_dim, float amp, const int* tok_slot,
                            const int* tok_pos, const int* page_table, int max_pages,
                            int ring_pages, void* kpool, void* vpool, void* q_out, int q_ld,
                            int dtype, void* first, const float* lam, void* gate_out, int gate_n,
                            int T, int nh, int nkv, int dim, int vd, void* stream) {
  if (T <= 0) return 0;
  if (rot_dim < 0 || rot_dim > dim || (rot_dim & 1) || (rot_dim > 0 && inv_freq == nullptr))
    MB_FAIL("mb_rope_store: %d of %d values rotate", rot_dim, dim);
  if (nh <= 0 || nkv <= 0 || nh % nkv || parts < 1 || dim <= 0 || vd <= 0)
    MB_FAIL("mb_rope_store: %d heads on %d KV heads, %d parts", nh, nkv, parts);
  if (ld < (nh + nkv) * dim + nkv * vd + (gate_out ? gate_n : 0) || q_ld < nh * dim)
    MB_FAIL("mb_rope_store: row pitches of %d and %d", ld, q_ld);
  if (in_dtype == MB_BF16 && dtype != MB_BF16)
    MB_FAIL("mb_rope_store: bfloat16 rows for float32 activations");
  if (lam != nullptr && first == nullptr) MB_FAIL("mb_rope_store: nothing to blend with");
  if (rot_dim > 8192) MB_FAIL("mb_rope_store: %d rotating values", rot_dim);
  cudaStream_t s = (cudaStream_t)stream;
  const uintptr_t bits = (uintptr_t)rows | (uintptr_t)kpool | (uintptr_t)vpool | (uintptr_t)q_out |
                         (uintptr_t)first | (uintptr_t)gate_out;
  const bool wide = dim % 8 == 0 && vd % 8 == 0 && (rot_dim / 2) % 8 == 0 && ld % 8 == 0 &&
                    q_ld % 8 == 0 && part_stride % 8 == 0 && (!gate_out || gate_n % 8 == 0) &&
                    (bits & 15) == 0;
  const int V = wide ? 8 : 1;
  const int items = (nh + nkv) * (dim - rot_dim / 2) / V + nkv * vd / V + (gate_out ? gate_n / V : 0);
  // few tokens: an item a thread; many: a block walks its token's items, the angles once
  const int threads = items >= 256 ? 256 : (items > 64 ? 128 : 64);
  const int most = (items + threads - 1) / threads;
  dim3 grid(T, T <= 64 ? most : (most + 3) / 4);
  const size_t smem = (size_t)rot_dim * sizeof(float);
#define GO(TI_, TO_, V_)                                                                        \
  mb_launch(rope_store_kernel<TI_, TO_, V_>, grid, dim3(threads), smem, s, (const TI_*)rows,    \
            parts, (size_t)part_stride, ld, inv_freq, rot_dim, amp, tok_slot, tok_pos,          \
            page_table, max_pages, ring_pages, (TO_*)kpool, (TO_*)vpool, (TO_*)q_out, q_ld,     \
            (TO_*)first, lam, (TO_*)gate_out, gate_n, nh, nkv, dim, vd)
#define GO_V(TI_, TO_) { if (wide) GO(TI_, TO_, 8); else GO(TI_, TO_, 1); }
  if (dtype == MB_F32) GO_V(float, float)
  else if (in_dtype == MB_F32) GO_V(float, __nv_bfloat16)
  else GO_V(__nv_bfloat16, __nv_bfloat16)
#undef GO_V
#undef GO
  MB_CHECK_LAUNCH("mb_rope_store");
}
