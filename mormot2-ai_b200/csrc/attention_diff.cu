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
//
// Tensor-core kernels (mma.sync, bfloat16; maps of up to 128 values and value rows of up to
// 256, both multiples of 8). Decode: a KV head's two maps are halves of one 16-row product, so
// keys and values stream once for all the heads that share them. Prefill: one set of warps for
// each map, both over the same tiles in shared memory. The sizes are rounded up to 64 or 128
// (values: 64, 128 or 256) in the loops: the queries are zero beyond a map's size, and output
// columns beyond the value row are never read.
#include "attention_mma.cuh"

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

// ------------------------------------------------------------------ tensor-core kernels
typedef __nv_bfloat16 bf16;
#define DD_WARPS 4
#define DD_STAGES 3
#define DD_HEADS 8       // query heads of a KV head that one CTA takes
#define DD_SLACK 256     // reads past a tile's end (rounded-up sizes) stay inside the allocation

// q fragments of one map: 8 consecutive values per 32-value chunk and thread, zero beyond `dim`
template <int DB>
__device__ __forceinline__ void load_map(const bf16* q, int dim, int c, uint4* out) {
#pragma unroll
  for (int ch = 0; ch < DB / 32; ++ch) {
    const int at = ch * 32 + c * 8;
    out[ch] = q != nullptr && at < dim ? ldg16(q + at) : make_uint4(0, 0, 0, 0);
  }
}

// Decode: one CTA per (token, KV head [x 8 query heads of its group], split). Rows r of the
// m16n8k16 product are map 1 of the heads, rows r + 8 map 2 of the same heads: the scores of a
// page come from two products that each leave the other map's rows zero, the weighted values
// from one. Warp 4 streams the split's pages (every `splits`-th) by bulk copies, three ahead;
// warps 0-3 take 16 keys of every page each and keep an online softmax of their own. The warps
// are merged in shared memory, the splits through the shared memory of their cluster, where a
// warp then has a whole head: it takes the maps' difference, norms it and stores it.
template <int DB, int VB>
__global__ void __launch_bounds__((DD_WARPS + 1) * 32)
diff_decode_kernel(const bf16* __restrict__ q, const bf16* __restrict__ kpool,
                   const bf16* __restrict__ vpool, const int* __restrict__ page_table,
                   int max_pages, int ring_pages, const int* __restrict__ tok_slot,
                   const int* __restrict__ tok_pos, int nh, int nkv, int dim, int vd, int window,
                   float scale_log2, float lam, float factor, float eps, bf16* __restrict__ out,
                   int* __restrict__ error) {
  constexpr int CH = DB / 32, DBV = VB / 64;
  extern __shared__ __align__(128) uint8_t dd_smem[];
  const uint32_t kbytes = (uint32_t)MB_PAGE * 2 * dim * 2, vbytes = (uint32_t)MB_PAGE * vd * 2;
  const uint32_t stage = kbytes + vbytes;
  const uint32_t tiles = smem_u32(dd_smem);
  // after the loop the tiles' memory holds the warps' partial results; the barriers lie behind
  const uint32_t merge = (DD_WARPS + 1) * 16 * VB * 4 + (DD_WARPS + 1) * 32 * 4;
  const uint32_t room = max(DD_STAGES * stage + DD_SLACK, merge);
  const uint32_t full0 = tiles + room, empty0 = full0 + 8 * DD_STAGES;

  const int s = blockIdx.x, S = gridDim.x, t = blockIdx.z;
  const int G = nh / nkv, subs = (G + DD_HEADS - 1) / DD_HEADS;
  const int g = blockIdx.y / subs, sub = blockIdx.y % subs;
  const int h0 = g * G + sub * DD_HEADS;
  const int heads = min(DD_HEADS, G - sub * DD_HEADS);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = lane >> 2, c = lane & 3;

  const int pos = tok_pos[t], slot = tok_slot[t];
  const int lo = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
  const int lo_page = lo / MB_PAGE, p_last = pos / MB_PAGE;
  const int listed = p_last - lo_page + 1;
  const int n_pages = s < listed ? (listed - 1 - s) / S + 1 : 0;

  if (threadIdx.x == 0) {
    for (int i = 0; i < DD_STAGES; ++i) {
      mbar_init(full0 + 8 * i, 1);
      mbar_init(empty0 + 8 * i, DD_WARPS);
    }
    mbar_fence_init();
  }
  __syncthreads();

  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  float o[DBV][8][4];
#pragma unroll
  for (int db = 0; db < DBV; ++db)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[db][j][e] = 0.f;

  if (warp == DD_WARPS) {
    // only the newest page is written by the kernel before this one: the copies of older pages
    // start at once, the wait comes before the first copy of the newest page
    bool waited = false;
    int st = 0;
    uint32_t ph = 0;
    for (int i0 = 0; i0 < n_pages; i0 += 32) {
      int mine = 0;
      if (i0 + lane < n_pages) {
        const int p = lo_page + s + (i0 + lane) * S;
        const int entry = ring_pages > 0 ? p % ring_pages : p;
        mine = MB_INDEX_OK(entry < max_pages, 1, slot, p, max_pages)
                   ? page_table[(size_t)slot * max_pages + entry] : 0;
        if (!MB_INDEX_OK(mine >= 0, 2, slot, entry, mine)) mine = 0;
      }
      const int n = min(32, n_pages - i0);
      for (int i = 0; i < n; ++i) {
        const int page = __shfl_sync(0xffffffffu, mine, i);
        if (!waited && lo_page + s + (i0 + i) * S == p_last) {
          mb_grid_wait();
          waited = true;
        }
        if (lane == 0) {
          mbar_wait(empty0 + 8 * st, ph ^ 1, error, 4);
          mbar_expect_tx(full0 + 8 * st, stage);
          const size_t row = ((size_t)page * nkv + g) * MB_PAGE;
          bulk_copy(tiles + st * stage, kpool + row * 2 * dim, kbytes, full0 + 8 * st);
          bulk_copy(tiles + st * stage + kbytes, vpool + row * vd, vbytes, full0 + 8 * st);
        }
        if (++st == DD_STAGES) { st = 0; ph ^= 1; }
      }
    }
    if (!waited) mb_grid_wait();
    mb_grid_launch_next();
  } else {
    mb_grid_wait();  // q comes from the kernel before
    uint4 qa[CH], qb[CH];
    const bf16* qrow = r < heads ? q + ((size_t)t * nh + h0 + r) * 2 * dim : nullptr;
    load_map<DB>(qrow, dim, c, qa);
    load_map<DB>(qrow ? qrow + dim : nullptr, dim, c, qb);
    int st = 0;
    uint32_t ph = 0;
    for (int i = 0; i < n_pages; ++i) {
      const int key0 = (lo_page + s + i * S) * MB_PAGE + 16 * warp;  // this warp's 16 keys
      mbar_wait(full0 + 8 * st, ph, error, 5);
      const uint32_t ks = tiles + st * stage + (uint32_t)(16 * warp) * dim * 4;
      const uint32_t vs = tiles + st * stage + kbytes + (uint32_t)(16 * warp) * vd * 2;
      float sc[2][4];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        sc[u][0] = sc[u][1] = sc[u][2] = sc[u][3] = 0.f;
        const uint32_t krow = ks + (uint32_t)(u * 8 + r) * dim * 4 + c * 16;
#pragma unroll
        for (int ch = 0; ch < CH; ++ch) {
          const uint4 k1 = lds16(krow + ch * 64), k2 = lds16(krow + dim * 2 + ch * 64);
          mma_bf16(sc[u], qa[ch].x, 0u, qa[ch].y, 0u, k1.x, k1.y);
          mma_bf16(sc[u], qa[ch].z, 0u, qa[ch].w, 0u, k1.z, k1.w);
          mma_bf16(sc[u], 0u, qb[ch].x, 0u, qb[ch].y, k2.x, k2.y);
          mma_bf16(sc[u], 0u, qb[ch].z, 0u, qb[ch].w, k2.z, k2.w);
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int key = key0 + u * 8 + 2 * c + e;
          const bool ok = key <= pos && key >= lo;
          sc[u][e] = ok ? sc[u][e] * scale_log2 : -INFINITY;
          sc[u][2 + e] = ok ? sc[u][2 + e] * scale_log2 : -INFINITY;
          mx0 = fmaxf(mx0, sc[u][e]);
          mx1 = fmaxf(mx1, sc[u][2 + e]);
        }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);
      // this warp's 16 keys of the page may all lie outside [lo, pos]: keep exp2 off inf - inf
      const float base0 = n0 == -INFINITY ? 0.f : n0, base1 = n1 == -INFINITY ? 0.f : n1;
      const float c0 = exp2f(m0 - base0), c1 = exp2f(m1 - base1);
      m0 = n0;
      m1 = n1;
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          sc[u][e] = exp2f(sc[u][e] - base0);
          sc[u][2 + e] = exp2f(sc[u][2 + e] - base1);
          s0 += sc[u][e];
          s1 += sc[u][2 + e];
        }
      l0 = l0 * c0 + s0;
      l1 = l1 * c1 + s1;
      const uint32_t a0 = pack_bf16(sc[0][0], sc[0][1]), a1 = pack_bf16(sc[0][2], sc[0][3]);
      const uint32_t a2 = pack_bf16(sc[1][0], sc[1][1]), a3 = pack_bf16(sc[1][2], sc[1][3]);
      const uint32_t vrow = vs + (uint32_t)(2 * c) * vd * 2 + r * 16;
#pragma unroll
      for (int db = 0; db < DBV; ++db) {
        const uint4 va = lds16(vrow + db * 128);
        const uint4 vb = lds16(vrow + vd * 2 + db * 128);
        const uint4 vc = lds16(vrow + 16 * vd + db * 128);
        const uint4 ve = lds16(vrow + 18 * vd + db * 128);
        const uint32_t wa[4] = {va.x, va.y, va.z, va.w}, wb[4] = {vb.x, vb.y, vb.z, vb.w};
        const uint32_t wc[4] = {vc.x, vc.y, vc.z, vc.w}, wd[4] = {ve.x, ve.y, ve.z, ve.w};
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          o[db][j][0] *= c0;
          o[db][j][1] *= c0;
          o[db][j][2] *= c1;
          o[db][j][3] *= c1;
          const int w = j >> 1;
          const uint32_t b0 = (j & 1) ? pack_hi(wa[w], wb[w]) : pack_lo(wa[w], wb[w]);
          const uint32_t b1 = (j & 1) ? pack_hi(wc[w], wd[w]) : pack_lo(wc[w], wd[w]);
          mma_bf16(o[db][j], a0, a1, a2, a3, b0, b1);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(empty0 + 8 * st);  // this warp is done with the stage
      if (++st == DD_STAGES) { st = 0; ph ^= 1; }
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  }
  // every copy has landed and been read: the tiles' memory now holds the warps' results
  __syncthreads();
  float* sm_o = (float*)dd_smem;                        // [DD_WARPS][16][VB]
  float* sm_c = sm_o + DD_WARPS * 16 * VB;              // [16][VB] the CTA's own result
  float* sm_m = sm_c + 16 * VB;                         // [DD_WARPS][16]
  float* sm_l = sm_m + DD_WARPS * 16;                   // [DD_WARPS][16]
  float* sm_cml = sm_l + DD_WARPS * 16;                 // [16] its maxima, [16] its sums
  if (warp < DD_WARPS) {
    if (c == 0) {
      sm_m[warp * 16 + r] = m0;
      sm_m[warp * 16 + r + 8] = m1;
      sm_l[warp * 16 + r] = l0;
      sm_l[warp * 16 + r + 8] = l1;
    }
#pragma unroll
    for (int db = 0; db < DBV; ++db)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int d0 = db * 64 + (2 * c) * 8 + j, d1 = d0 + 8;
        sm_o[(warp * 16 + r) * VB + d0] = o[db][j][0];
        sm_o[(warp * 16 + r) * VB + d1] = o[db][j][1];
        sm_o[(warp * 16 + r + 8) * VB + d0] = o[db][j][2];
        sm_o[(warp * 16 + r + 8) * VB + d1] = o[db][j][3];
      }
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < 2 * heads * VB; idx += blockDim.x) {
    const int hr = idx / VB, d = idx - hr * VB;
    const int row = hr < heads ? hr : hr - heads + 8;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < DD_WARPS; ++w) M = fmaxf(M, sm_m[w * 16 + row]);
    float L = 0.f, acc = 0.f;
    if (M > -INFINITY) {
#pragma unroll
      for (int w = 0; w < DD_WARPS; ++w) {
        const float f = exp2f(sm_m[w * 16 + row] - M);  // 0 for a warp without keys
        if (f == 0.f) continue;
        L += sm_l[w * 16 + row] * f;
        acc += sm_o[(w * 16 + row) * VB + d] * f;
      }
    }
    sm_c[row * VB + d] = acc;
    if (d == 0) {
      sm_cml[row] = M;
      sm_cml[16 + row] = L;
    }
  }
  if (S > 1) cluster_sync_all(); else __syncthreads();
  // the heads of the group are dealt over the cluster's warps; the splits add up in order
  const uint32_t c_addr = smem_u32(sm_c), ml_addr = smem_u32(sm_cml);
  for (int n = s + S * warp; n < heads; n += S * (DD_WARPS + 1)) {
    float f[2][8], L[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      float M = -INFINITY, mk[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        mk[k] = k < S ? ld_cluster_f32(cluster_addr_of(ml_addr + 4 * (n + 8 * j), k)) : -INFINITY;
        M = fmaxf(M, mk[k]);
      }
      L[j] = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        f[j][k] = mk[k] == -INFINITY ? 0.f : exp2f(mk[k] - M);
        if (k < S) L[j] += f[j][k] * ld_cluster_f32(cluster_addr_of(ml_addr + 4 * (16 + n + 8 * j), k));
      }
    }
    const float i1 = 1.0f / L[0], i2 = lam / L[1];
    float v[VB / 32], sum = 0.f;
#pragma unroll
    for (int i = 0; i < VB / 32; ++i) {
      const int d = lane + 32 * i;
      float a1 = 0.f, a2 = 0.f;
      if (d < vd) {
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (k < S) {
            a1 += f[0][k] * ld_cluster_f32(cluster_addr_of(c_addr + 4 * (n * VB + d), k));
            a2 += f[1][k] * ld_cluster_f32(cluster_addr_of(c_addr + 4 * ((n + 8) * VB + d), k));
          }
      }
      v[i] = a1 * i1 - a2 * i2;
      sum = fmaf(v[i], v[i], sum);
    }
    const float scale = factor / sqrtf(warp_sum(sum) / (float)vd + eps);
    bf16* op = out + ((size_t)t * nh + h0 + n) * vd;
#pragma unroll
    for (int i = 0; i < VB / 32; ++i)
      if (lane + 32 * i < vd) op[lane + 32 * i] = __float2bfloat16_rn(v[i] * scale);
  }
  if (S > 1) cluster_sync_all();  // no CTA leaves while another may still read its shared memory
}

static int diff_checks(const char* who, const void* q, const void* out, const void* kpool,
                       const void* vpool, int T, int nh, int nkv, int dim, int vd) {
  if (dim <= 0 || dim > 128 || dim % 8 || vd <= 0 || vd > 256 || vd % 8)
    MB_FAIL("%s: maps of %d and value rows of %d values (multiples of 8, at most 128 and 256)",
            who, dim, vd);
  if (nkv <= 0 || nh % nkv) MB_FAIL("%s: %d heads on %d KV heads", who, nh, nkv);
  if (((uintptr_t)q | (uintptr_t)out | (uintptr_t)kpool | (uintptr_t)vpool) & 15)
    MB_FAIL("%s: q, out or the cache pools are not 16-byte aligned", who);
  if (T > 65535) MB_FAIL("%s: %d tokens or sequences are too many for one launch", who, T);
  return 0;
}

#define DIFF_SIZES(GO)                                                        \
  if (dim <= 64) {                                                            \
    if (vd <= 64) GO(64, 64) else if (vd <= 128) GO(64, 128) else GO(64, 256) \
  } else {                                                                    \
    if (vd <= 128) GO(128, 128) else GO(128, 256)                             \
  }

// out[t, h, :] for every token t, each with its own sequence and position (a decode step).
// `splits` (at most 8) CTAs share a sequence's pages; the caller chooses it from the batch and
// the cache's capacity, not from the lengths of the moment, so that a captured launch stays
// valid. `error`: a device word that receives 4 or 5 if a wait of the copy pipeline ran out.
MB_EXPORT int mb_attention_diff_decode(const void* q, void* out, const void* kpool,
                                       const void* vpool, const int* page_table, int max_pages,
                                       int ring_pages, const int* tok_slot, const int* tok_pos,
                                       int T, int nh, int nkv, int dim, int vd, int window,
                                       float scale, float lam, float factor, float eps,
                                       int splits, int* error, void* stream) {
  if (T <= 0) return 0;
  if (diff_checks("mb_attention_diff_decode", q, out, kpool, vpool, T, nh, nkv, dim, vd)) return -1;
  if (splits < 1 || splits > 8) MB_FAIL("mb_attention_diff_decode: %d splits (1 to 8)", splits);
  const int G = nh / nkv, subs = (G + DD_HEADS - 1) / DD_HEADS;
  const float scale_log2 = scale * 1.4426950408889634f;
  const size_t stage = (size_t)MB_PAGE * (2 * dim + vd) * 2;
  dim3 grid(splits, nkv * subs, T), block((DD_WARPS + 1) * 32);
  cudaStream_t s = (cudaStream_t)stream;
#define GO(D_, V_)                                                                             \
  {                                                                                            \
    const size_t merge = (DD_WARPS + 1) * 16 * V_ * 4 + (DD_WARPS + 1) * 32 * 4;               \
    const size_t room = DD_STAGES * stage + DD_SLACK;                                          \
    const size_t smem = (room > merge ? room : merge) + 16 * DD_STAGES;                        \
    static bool configured = false;                                                            \
    if (!configured) {                                                                         \
      cudaError_t e = cudaFuncSetAttribute(diff_decode_kernel<D_, V_>,                         \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize,        \
                                           220 * 1024);                                        \
      if (e != cudaSuccess) MB_FAIL("mb_attention_diff_decode: %s", cudaGetErrorString(e));    \
      configured = true;                                                                       \
    }                                                                                          \
    if (splits > 1)                                                                            \
      mb_launch_clusters(diff_decode_kernel<D_, V_>, grid, block, smem, s, splits,             \
                         (const bf16*)q, (const bf16*)kpool, (const bf16*)vpool, page_table,   \
                         max_pages, ring_pages, tok_slot, tok_pos, nh, nkv, dim, vd, window,   \
                         scale_log2, lam, factor, eps, (bf16*)out, error);                     \
    else                                                                                       \
      mb_launch(diff_decode_kernel<D_, V_>, grid, block, smem, s, (const bf16*)q,              \
                (const bf16*)kpool, (const bf16*)vpool, page_table, max_pages, ring_pages,     \
                tok_slot, tok_pos, nh, nkv, dim, vd, window, scale_log2, lam, factor, eps,     \
                (bf16*)out, error);                                                            \
  }
  DIFF_SIZES(GO)
#undef GO
  MB_CHECK_LAUNCH("mb_attention_diff_decode");
}

// ------------------------------------------------------------------ prefill
// A CTA takes 64 consecutive new tokens of one sequence and one query head: warps 0-3 map 1,
// warps 4-7 map 2, each 16 tokens as the rows of the product with an online softmax per row. The
// pages that any of the tokens may see come to shared memory by 16-byte asynchronous copies,
// two pages ahead; the two maps' keys lie at fixed places of a padded row. At the end the
// second map's warps hand their outputs (times lambda over the row sums) to the first's, which
// take the difference, norm it over the head and store it.
template <int DB, int VB>
__global__ void __launch_bounds__(256, (DB == 64 && VB <= 128) ? 2 : 1)
diff_prefill_kernel(const bf16* __restrict__ q, const bf16* __restrict__ kpool,
                    const bf16* __restrict__ vpool, const int* __restrict__ page_table,
                    int max_pages, int ring_pages, const int* __restrict__ seq_start,
                    const int* __restrict__ seq_past, const int* __restrict__ seq_slot, int nh,
                    int nkv, int dim, int vd, int window, float scale_log2, float lam,
                    float factor, float eps, bf16* __restrict__ out) {
  mb_grid_wait();
  mb_grid_launch_next();
  constexpr int CH = DB / 32, DBV = VB / 64;
  constexpr int KP = 4 * DB + 64, VP = 2 * VB + 16;     // row pitches in bytes
  constexpr uint32_t STAGE = MB_PAGE * (KP + VP);
  extern __shared__ __align__(128) uint8_t dp_smem[];
  const uint32_t tiles = smem_u32(dp_smem);

  const int b = blockIdx.z, h = blockIdx.y;
  const int start = seq_start[b], n_new = seq_start[b + 1] - start;
  if ((int)blockIdx.x * 64 >= n_new) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = lane >> 2, c = lane & 3;
  const int map = warp >> 2, wrow = warp & 3;
  const int past = seq_past[b], slot = seq_slot[b];
  const int g = h / (nh / nkv);
  const int cta_first = past + blockIdx.x * 64;
  const int cta_last = past + min((int)blockIdx.x * 64 + 63, n_new - 1);
  const int cta_lo = (window > 0 && cta_first + 1 > window) ? cta_first + 1 - window : 0;
  const int page0 = cta_lo / MB_PAGE, n_pages = cta_last / MB_PAGE - page0 + 1;

  if (dim < DB) {   // what a map's rows are rounded up by stays zero
    for (int e = threadIdx.x; e < (int)(DD_STAGES * STAGE / 16); e += 256)
      *(uint4*)(dp_smem + 16 * e) = make_uint4(0, 0, 0, 0);
    __syncthreads();
  }
  const int kch = dim / 8, vch = vd / 8;                // 16-byte chunks of a map, of a value row
  auto issue = [&](int i) {  // page i of the CTA into stage i % DD_STAGES
    if (i < n_pages) {
      const int p = page0 + i;
      const int entry = ring_pages > 0 ? p % ring_pages : p;
      int page = MB_INDEX_OK(entry < max_pages, 1, slot, p, max_pages)
                     ? page_table[(size_t)slot * max_pages + entry] : 0;
      if (!MB_INDEX_OK(page >= 0, 2, slot, entry, page)) page = 0;
      const size_t row0 = ((size_t)page * nkv + g) * MB_PAGE;
      const uint32_t kd = tiles + (i % DD_STAGES) * STAGE, vdst = kd + MB_PAGE * KP;
      for (int e = threadIdx.x; e < MB_PAGE * 2 * kch; e += 256) {
        const int row = e / (2 * kch), ch = e - row * 2 * kch;
        const int j = ch >= kch;
        cp_async16(kd + row * KP + j * (2 * DB) + (ch - j * kch) * 16,
                   kpool + (row0 + row) * 2 * dim + ch * 8);
      }
      for (int e = threadIdx.x; e < MB_PAGE * vch; e += 256) {
        const int row = e / vch, ch = e - row * vch;
        cp_async16(vdst + row * VP + ch * 16, vpool + (row0 + row) * vd + ch * 8);
      }
    }
    cp_async_commit();
  };

  const int row0 = blockIdx.x * 64 + wrow * 16;
  const bool live = row0 < n_new;  // a warp without rows still loads and synchronizes
  const int ra = row0 + r, rb = ra + 8;
  const bool has_a = ra < n_new, has_b = rb < n_new;
  const int pa = past + ra, pb = past + rb;  // positions of the two rows
  const int la = (window > 0 && pa + 1 > window) ? pa + 1 - window : 0;
  const int lb = (window > 0 && pb + 1 > window) ? pb + 1 - window : 0;
  const int first_pos = past + row0, last_pos = past + min(row0 + 15, n_new - 1);
  const int lo_w = (window > 0 && first_pos + 1 > window) ? first_pos + 1 - window : 0;

#pragma unroll
  for (int i = 0; i < DD_STAGES - 1; ++i) issue(i);

  uint4 qa[CH], qb[CH];
  {
    const size_t token = (size_t)2 * nh * dim;
    const bf16* qrow = q + (size_t)(start + ra) * token + (size_t)(2 * h + map) * dim;
    load_map<DB>(has_a ? qrow : nullptr, dim, c, qa);
    load_map<DB>(has_b ? qrow + 8 * token : nullptr, dim, c, qb);
  }
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  float o[DBV][8][4];
#pragma unroll
  for (int db = 0; db < DBV; ++db)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[db][j][e] = 0.f;

  for (int i = 0; i < n_pages; ++i) {
    cp_async_wait<DD_STAGES - 2>();  // page i has landed (for this thread's copies)
    __syncthreads();                 // ... for everyone's; and page i - 1 has been read by all
    issue(i + DD_STAGES - 1);        // into the stage that page i - 1 occupied
    const int p = page0 + i;
    if (live && p >= lo_w / MB_PAGE && p <= last_pos / MB_PAGE) {
      const uint32_t ks = tiles + (i % DD_STAGES) * STAGE, vs = ks + MB_PAGE * KP;
      const int key0 = p * MB_PAGE;
      float sc[8][4];
      qk_page_smem<DB, KP>(qa, qb, ks + map * (2 * DB), r, c, sc);
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int key = key0 + u * 8 + 2 * c + e;
          sc[u][e] = key <= pa && key >= la ? sc[u][e] * scale_log2 : -INFINITY;
          sc[u][2 + e] = key <= pb && key >= lb ? sc[u][2 + e] * scale_log2 : -INFINITY;
          mx0 = fmaxf(mx0, sc[u][e]);
          mx1 = fmaxf(mx1, sc[u][2 + e]);
        }
      }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);
      // a row may have no key in this page (and none so far): keep exp2 away from inf - inf
      const float base0 = n0 == -INFINITY ? 0.f : n0, base1 = n1 == -INFINITY ? 0.f : n1;
      const float c0 = exp2f(m0 - base0), c1 = exp2f(m1 - base1);
      m0 = n0;
      m1 = n1;
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          sc[u][e] = exp2f(sc[u][e] - base0);
          sc[u][2 + e] = exp2f(sc[u][2 + e] - base1);
          s0 += sc[u][e];
          s1 += sc[u][2 + e];
        }
      }
      l0 = l0 * c0 + s0;
      l1 = l1 * c1 + s1;
#pragma unroll
      for (int db = 0; db < DBV; ++db)
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          o[db][j][0] *= c0;
          o[db][j][1] *= c0;
          o[db][j][2] *= c1;
          o[db][j][3] *= c1;
        }
      pv_page_smem<VB, VP>(sc, vs, r, c, o);
    }
  }
  cp_async_wait<0>();
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  __syncthreads();                   // the tiles' memory is free
  // a thread of a second-map warp and the same thread of the first-map warp four before it hold
  // the same places: value k of lane l of row block w at [(w * places + k) * 32 + l]
  constexpr int PLACES = DBV * 32;
  float* hand = (float*)dp_smem + (size_t)wrow * PLACES * 32 + lane;
  if (map == 1) {
    const float i0 = lam / l0, i1 = lam / l1;
#pragma unroll
    for (int db = 0; db < DBV; ++db)
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          hand[((db * 8 + j) * 4 + e) * 32] = o[db][j][e] * (e < 2 ? i0 : i1);
  }
  __syncthreads();
  if (map == 1 || !live) return;
  const float i0 = 1.0f / l0, i1 = 1.0f / l1;
  float q0 = 0.f, q1 = 0.f;
  // a thread holds the dims db*64 + 16c .. + 15 of its two rows
#pragma unroll
  for (int db = 0; db < DBV; ++db)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float v = o[db][j][e] * (e < 2 ? i0 : i1) - hand[((db * 8 + j) * 4 + e) * 32];
        o[db][j][e] = v;
        if (db * 64 + 16 * c + 8 * (e & 1) < vd) {     // columns beyond the row count nothing
          if (e < 2) q0 = fmaf(v, v, q0);
          else q1 = fmaf(v, v, q1);
        }
      }
  q0 += __shfl_xor_sync(0xffffffffu, q0, 1);
  q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
  q1 += __shfl_xor_sync(0xffffffffu, q1, 1);
  q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
  const float f0 = factor / sqrtf(q0 / (float)vd + eps), f1 = factor / sqrtf(q1 / (float)vd + eps);
#pragma unroll
  for (int db = 0; db < DBV; ++db) {
    uint32_t w[4][4];  // [row a lo, row a hi, row b lo, row b hi][4 registers of 2 bf16]
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      w[0][j >> 1] = pack_bf16(o[db][j][0] * f0, o[db][j + 1][0] * f0);
      w[1][j >> 1] = pack_bf16(o[db][j][1] * f0, o[db][j + 1][1] * f0);
      w[2][j >> 1] = pack_bf16(o[db][j][2] * f1, o[db][j + 1][2] * f1);
      w[3][j >> 1] = pack_bf16(o[db][j][3] * f1, o[db][j + 1][3] * f1);
    }
    const int d = db * 64 + 16 * c;
    bf16* oa = out + ((size_t)(start + ra) * nh + h) * vd + d;
    bf16* ob = oa + (size_t)8 * nh * vd;
    if (has_a && d < vd) *(uint4*)oa = make_uint4(w[0][0], w[0][1], w[0][2], w[0][3]);
    if (has_a && d + 8 < vd) *(uint4*)(oa + 8) = make_uint4(w[1][0], w[1][1], w[1][2], w[1][3]);
    if (has_b && d < vd) *(uint4*)ob = make_uint4(w[2][0], w[2][1], w[2][2], w[2][3]);
    if (has_b && d + 8 < vd) *(uint4*)(ob + 8) = make_uint4(w[3][0], w[3][1], w[3][2], w[3][3]);
  }
}

// out[t, h, :] for the new tokens of B sequences (packed one after another: sequence b holds
// the rows seq_start[b] .. seq_start[b + 1]) over the cache. `max_new`: the most new tokens of
// one sequence.
MB_EXPORT int mb_attention_diff_prefill(const void* q, void* out, const void* kpool,
                                        const void* vpool, const int* page_table, int max_pages,
                                        int ring_pages, const int* seq_start, const int* seq_past,
                                        const int* seq_slot, int B, int max_new, int nh, int nkv,
                                        int dim, int vd, int window, float scale, float lam,
                                        float factor, float eps, void* stream) {
  if (B <= 0 || max_new <= 0) return 0;
  if (diff_checks("mb_attention_diff_prefill", q, out, kpool, vpool, B, nh, nkv, dim, vd)) return -1;
  if (nh > 65535) MB_FAIL("mb_attention_diff_prefill: %d heads", nh);
  dim3 grid((max_new + 63) / 64, nh, B);
  const float scale_log2 = scale * 1.4426950408889634f;
  cudaStream_t s = (cudaStream_t)stream;
#define GO(D_, V_)                                                                             \
  {                                                                                            \
    constexpr int smem = DD_STAGES * MB_PAGE * (4 * D_ + 64 + 2 * V_ + 16);                    \
    static bool configured = false;                                                            \
    if (!configured) {                                                                         \
      cudaError_t e = cudaFuncSetAttribute(diff_prefill_kernel<D_, V_>,                        \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, smem); \
      if (e != cudaSuccess) MB_FAIL("mb_attention_diff_prefill: %s", cudaGetErrorString(e));   \
      configured = true;                                                                       \
    }                                                                                          \
    mb_launch(diff_prefill_kernel<D_, V_>, grid, dim3(256), smem, s, (const bf16*)q,           \
              (const bf16*)kpool, (const bf16*)vpool, page_table, max_pages, ring_pages,       \
              seq_start, seq_past, seq_slot, nh, nkv, dim, vd, window, scale_log2, lam,        \
              factor, eps, (bf16*)out);                                                        \
  }
  DIFF_SIZES(GO)
#undef GO
  MB_CHECK_LAUNCH("mb_attention_diff_prefill");
}
