// Causal differential attention over the paged cache: every head has two queries and two keys
// (maps) over the same values; each map is a softmax attention of its own over the keys
// max(0, pos + 1 - window) .. pos, and the head's output is
//   o = a_1 - lam a_2,   factor * o / sqrt(mean(o^2) + eps).
// A key head's two maps lie one after the other in a cache row of 2 dim values (values in rows
// of vd), a query head's in 2 dim values of q. Head h reads KV head h div (heads div kv_heads).
//
// General kernel: float32 arithmetic on the CUDA cores for float32 or bfloat16 storage and any
// sizes up to 256 and 512. One warp per (token, head) walks the keys of the token's own
// sequence in tiles of 32 with an online softmax for each map (a lane has one key of the tile
// for both scores and values lane, lane + 32, ... of every key's row).
#include "common.cuh"

MB_DEFINE_LAST_ERROR

#define AD_WARPS 4
#define AD_MAX_V 16  // values of a row a lane keeps, for each map: rows of up to 512

template <typename T, int NV>
__global__ void __launch_bounds__(AD_WARPS * 32)
attention_diff_kernel(const T* __restrict__ q, T* __restrict__ out, const T* __restrict__ kpool,
                      const T* __restrict__ vpool, const int* __restrict__ page_table,
                      int max_pages, int ring_pages, const int* __restrict__ tok_slot,
                      const int* __restrict__ tok_pos, int nh, int nkv, int dim, int vd,
                      int window, float scale, float lam, float factor, float eps) {
  mb_grid_wait();
  mb_grid_launch_next();
  extern __shared__ __align__(16) float ad_q[];  // AD_WARPS x 2 dim
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, h = blockIdx.y * AD_WARPS + warp;
  if (h >= nh) return;
  const int g = h / (nh / nkv);
  const int pos = tok_pos[t], slot = tok_slot[t];
  float* qv = ad_q + warp * 2 * dim;
  const T* qp = q + ((size_t)t * nh + h) * 2 * dim;
  for (int i = lane; i < 2 * dim; i += 32) qv[i] = to_f32<T>(qp[i]);
  __syncwarp();
  const int lo = window > 0 && pos + 1 > window ? pos + 1 - window : 0;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float acc[2][NV];
#pragma unroll
  for (int d = 0; d < NV; ++d) acc[0][d] = acc[1][d] = 0.f;
  for (int k0 = lo; k0 <= pos; k0 += 32) {
    const int kp = k0 + lane;
    const bool valid = kp <= pos;
    size_t row = 0;
    float s[2] = {-INFINITY, -INFINITY};
    if (valid) {
      row = kv_row(page_table, max_pages, ring_pages, slot, kp, nkv, g);
      const T* kr = kpool + row * 2 * dim;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        float dot = 0.f;
        for (int i = 0; i < dim; ++i) dot = fmaf(qv[j * dim + i], to_f32<T>(kr[j * dim + i]), dot);
        s[j] = dot * scale;
      }
    }
    float p[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float m_new = fmaxf(m[j], warp_max(s[j]));
      const float corr = expf(m[j] - m_new);  // 0 on the first tile (m = -inf)
      p[j] = valid ? expf(s[j] - m_new) : 0.f;
      l[j] = l[j] * corr + warp_sum(p[j]);
#pragma unroll
      for (int d = 0; d < NV; ++d) acc[j][d] *= corr;
      m[j] = m_new;
    }
    const int n = min(32, pos - k0 + 1);
    for (int e = 0; e < n; ++e) {
      const float p0 = __shfl_sync(0xffffffffu, p[0], e), p1 = __shfl_sync(0xffffffffu, p[1], e);
      const unsigned lo32 = __shfl_sync(0xffffffffu, (unsigned)(row & 0xffffffffu), e);
      const unsigned hi32 = __shfl_sync(0xffffffffu, (unsigned)(row >> 32), e);
      const T* vr = vpool + (((size_t)hi32 << 32) | lo32) * vd;
#pragma unroll
      for (int d = 0; d < NV; ++d) {
        const int i = lane + 32 * d;
        if (i < vd) {
          const float v = to_f32<T>(vr[i]);
          acc[0][d] = fmaf(p0, v, acc[0][d]);
          acc[1][d] = fmaf(p1, v, acc[1][d]);
        }
      }
    }
  }
  const float i1 = 1.0f / l[0], i2 = lam / l[1];
  float sum = 0.f;
#pragma unroll
  for (int d = 0; d < NV; ++d) {        // places beyond vd hold zeros
    acc[0][d] = acc[0][d] * i1 - acc[1][d] * i2;
    sum = fmaf(acc[0][d], acc[0][d], sum);
  }
  const float f = factor / sqrtf(warp_sum(sum) / (float)vd + eps);
  T* op = out + ((size_t)t * nh + h) * vd;
#pragma unroll
  for (int d = 0; d < NV; ++d) {
    const int i = lane + 32 * d;
    if (i < vd) op[i] = from_f32<T>(acc[0][d] * f);
  }
}

MB_EXPORT int mb_attention_diff(const void* q, void* out, const void* kpool, const void* vpool,
                                int dtype, const int* page_table, int max_pages, int ring_pages,
                                const int* tok_slot, const int* tok_pos, int T, int nh, int nkv,
                                int dim, int vd, int window, float scale, float lam, float factor,
                                float eps, void* stream) {
  if (T <= 0) return 0;
  if (dim <= 0 || dim > 256 || vd <= 0 || vd > 32 * AD_MAX_V)
    MB_FAIL("mb_attention_diff: maps of %d and value rows of %d values (at most 256 and %d)", dim,
            vd, 32 * AD_MAX_V);
  if (nkv <= 0 || nh % nkv) MB_FAIL("mb_attention_diff: %d heads on %d KV heads", nh, nkv);
  const size_t smem = (size_t)AD_WARPS * 2 * dim * sizeof(float);
  dim3 grid(T, (nh + AD_WARPS - 1) / AD_WARPS);
  cudaStream_t s = (cudaStream_t)stream;
#define GO(T_, NV_)                                                                            \
  mb_launch(attention_diff_kernel<T_, NV_>, grid, dim3(AD_WARPS * 32), smem, s, (const T_*)q,  \
            (T_*)out, (const T_*)kpool, (const T_*)vpool, page_table, max_pages, ring_pages,   \
            tok_slot, tok_pos, nh, nkv, dim, vd, window, scale, lam, factor, eps)
#define GO_V(T_)                                                                               \
  {                                                                                            \
    if (vd <= 128) GO(T_, 4); else if (vd <= 256) GO(T_, 8); else GO(T_, AD_MAX_V);            \
  }
  if (dtype == MB_F32) GO_V(float) else GO_V(__nv_bfloat16)
#undef GO_V
#undef GO
  MB_CHECK_LAUNCH("mb_attention_diff");
}
