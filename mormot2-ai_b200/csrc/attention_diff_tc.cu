// Causal differential prefill attention over the paged cache on the fifth-generation tensor
// cores, for bfloat16 maps of 64 values and value rows of 64 or 128 (attention_diff.cu has the
// formula and the other sizes): S_m = Q_m · K_mᵀ and O_m += P_m · V of both maps are
// tcgen05.mma instructions with their accumulators in tensor memory, the tiles of Q, K and V
// come by TMA (128-byte swizzle; a head's two maps are the two 64-column halves of its Q and K
// tiles), and each map's softmax runs in float32 on four warps of its own that read S from
// tensor memory, one row a thread.
//
// A CTA takes 128 consecutive new tokens of one sequence and one query head (the only CTA of
// its SM: the two maps fill tensor memory) and walks the pages that these tokens see:
//   warp 0      loads Q once, then K and V of page after page into rings of stages;
//   warp 1      issues S of both maps two pages ahead, each into one of two buffers of its
//               map, and O_m += P_m · V when P_m of a page is ready: the products of one map run
//               under the softmax of the other;
//   warps 2-5   map 1's softmax, warps 6-9 map 2's, as in attention_tc.cu (P over the S just
//               read, O rescaled only when a row's maximum has grown by more than 2^8).
// At the end the eight warps share a row's columns between the two that hold its tensor-memory
// lanes: each takes O_1 / l_1 - lam O_2 / l_2 of its half, the halves' sums of squares meet in
// shared memory, and the normed head is stored.
#include "attention_tc.cuh"

MB_DEFINE_LAST_ERROR

typedef __nv_bfloat16 bf16;

#define DT_ROWS 128
#define DT_K_STAGES 4
#define DT_V_STAGES 3
#define DT_THREADS 320
#define DT_Q_BYTES (DT_ROWS * 128 * 2)      // 32 KB: the two maps' 128 x 64 halves
#define DT_K_BYTES (MB_PAGE * 128 * 2)      // 16 KB: the two maps' 64 x 64 halves
#define DT_HALF (MB_PAGE * 64 * 2)          // 8 KB: 64 rows x 64 columns
#define DT_TMEM_COLS 512                    // S of map m: 128 m, two buffers of 64; O of map m: 256 + 128 m
#define DT_FIXED (DT_Q_BYTES + DT_K_STAGES * DT_K_BYTES)
// l and the sums of squares of the two maps' (halves') rows, then the barriers
#define DT_TAIL (4 * DT_ROWS * 4 + 256)

// threads of the softmax warps meet (named barrier 1)
__device__ __forceinline__ void softmax_sync() {
  asm volatile("bar.sync 1, 256;" ::: "memory");
}

template <int VD>
__global__ void __launch_bounds__(DT_THREADS, 1)
diff_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ,
                       const __grid_constant__ CUtensorMap tmK,
                       const __grid_constant__ CUtensorMap tmV, bf16* __restrict__ out,
                       const int* __restrict__ page_table, int max_pages, int ring_pages,
                       const int* __restrict__ seq_start, const int* __restrict__ seq_past,
                       const int* __restrict__ seq_slot, int nh, int nkv, int window,
                       float scale_log2, float lam, float factor, float eps,
                       int* __restrict__ error) {
  constexpr int VH = VD / 64;                  // 64-column blocks of a value row
  constexpr int V_BYTES = VH * DT_HALF;
  extern __shared__ __align__(1024) uint8_t dt_smem[];
  const uint32_t raw = smem_u32(dt_smem);
  if (raw & 1023u) {  // swizzled tiles need it; never seen, but a wrong result must not follow
    if (threadIdx.x == 0 && error) atomicCAS(error, 0, 19);
    return;
  }
  const uint32_t sQ = raw;
  const uint32_t sK = sQ + DT_Q_BYTES;                  // [stage][16 KB]
  const uint32_t sV = sK + DT_K_STAGES * DT_K_BYTES;    // [stage][V_BYTES]
  const uint32_t rowsums = sV + DT_V_STAGES * V_BYTES;
  float* sm_rows = (float*)(dt_smem + (rowsums - raw)); // [2][128] 1 / l, [2][128] sums of squares
  const uint32_t bars = rowsums + 4 * DT_ROWS * 4;
  const uint32_t q_full = bars, k_full0 = bars + 8, k_empty0 = k_full0 + 8 * DT_K_STAGES;
  const uint32_t v_full0 = k_empty0 + 8 * DT_K_STAGES, v_empty0 = v_full0 + 8 * DT_V_STAGES;
  // for each map m and buffer b, at 16 m + 8 b: S ready, P ready, the second product done
  const uint32_t s_full0 = v_empty0 + 8 * DT_V_STAGES, p_full0 = s_full0 + 32;
  const uint32_t o_done0 = p_full0 + 32, slot = o_done0 + 32;
  volatile uint32_t* slot_ptr = (volatile uint32_t*)(dt_smem + (slot - raw));

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // heads fastest (the query heads of one KV head run side by side and share its pages in L2),
  // and the last row tiles, which see the most pages, first
  const int b = blockIdx.z, h = blockIdx.x;
  const int start = seq_start[b], n_new = seq_start[b + 1] - start;
  const int row0 = (int)(gridDim.y - 1 - blockIdx.y) * DT_ROWS;
  if (row0 >= n_new) return;  // the whole CTA, before anything is set up
  const int past = seq_past[b], slot_of_seq = seq_slot[b];
  const int g = h / (nh / nkv);
  const int first_pos = past + row0, last_pos = past + min(row0 + DT_ROWS - 1, n_new - 1);
  const int cta_lo = (window > 0 && first_pos + 1 > window) ? first_pos + 1 - window : 0;
  const int page0 = cta_lo / MB_PAGE, n_pages = last_pos / MB_PAGE - page0 + 1;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < DT_K_STAGES; ++i) {
      mbar_init(k_full0 + 8 * i, 1);
      mbar_init(k_empty0 + 8 * i, 1);
    }
    for (int i = 0; i < DT_V_STAGES; ++i) {
      mbar_init(v_full0 + 8 * i, 1);
      mbar_init(v_empty0 + 8 * i, 1);
    }
    for (int i = 0; i < 4; ++i) {
      mbar_init(s_full0 + 8 * i, 1);
      mbar_init(p_full0 + 8 * i, 4);
      mbar_init(o_done0 + 8 * i, 1);
    }
    mbar_fence_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) tmem_alloc(slot, DT_TMEM_COLS);
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *slot_ptr;
  mb_grid_wait();  // q and the newest keys and values come from the kernel before
  mb_grid_launch_next();

  if (warp == 0) {
    if (elect_one()) {
      mbar_expect_tx(q_full, DT_Q_BYTES);
      tma_load_2d(sQ, &tmQ, h * 128, start + row0, q_full);
      tma_load_2d(sQ + DT_Q_BYTES / 2, &tmQ, h * 128 + 64, start + row0, q_full);
      auto row_of = [&](int j) {
        const int p = page0 + j;
        const int entry = ring_pages > 0 ? p % ring_pages : p;
        int page = MB_INDEX_OK(entry < max_pages, 1, slot_of_seq, p, max_pages)
                       ? page_table[(size_t)slot_of_seq * max_pages + entry] : 0;
        if (!MB_INDEX_OK(page >= 0, 2, slot_of_seq, entry, page)) page = 0;
        return (page * nkv + g) * MB_PAGE;
      };
      auto load_k = [&](int j) {
        const int st = j % DT_K_STAGES, y = row_of(j);
        mbar_wait(k_empty0 + 8 * st, ((j / DT_K_STAGES) & 1) ^ 1, error, 11);
        mbar_expect_tx(k_full0 + 8 * st, DT_K_BYTES);
        tma_load_2d(sK + st * DT_K_BYTES, &tmK, 0, y, k_full0 + 8 * st);
        tma_load_2d(sK + st * DT_K_BYTES + DT_HALF, &tmK, 64, y, k_full0 + 8 * st);
      };
      // the first products run two pages ahead of the second ones: so do the loads of K
      load_k(0);
      if (n_pages > 1) load_k(1);
      for (int j = 0; j < n_pages; ++j) {
        if (j + 2 < n_pages) load_k(j + 2);
        const int st = j % DT_V_STAGES, y = row_of(j);
        mbar_wait(v_empty0 + 8 * st, ((j / DT_V_STAGES) & 1) ^ 1, error, 10);
        mbar_expect_tx(v_full0 + 8 * st, V_BYTES);
        for (int i = 0; i < VH; ++i)
          tma_load_2d(sV + st * V_BYTES + i * DT_HALF, &tmV, 64 * i, y, v_full0 + 8 * st);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(DT_ROWS, MB_PAGE);             // K-major both
      constexpr uint32_t idesc_o = umma_idesc_bf16(DT_ROWS, 64) | (1u << 16);     // B MN-major
      mbar_wait(q_full, 0, error, 12);
      // S of map m and page j goes into buffer j % 2 of the map, which held S and then P of
      // page j - 2
      auto issue_s = [&](int j, int m) {
        const int st = j % DT_K_STAGES;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const uint64_t da = umma_desc_k128(sQ + m * (DT_Q_BYTES / 2) + k * 32);
          const uint64_t db = umma_desc_k128(sK + st * DT_K_BYTES + m * DT_HALF + k * 32);
          umma_bf16(tmem + 128 * m + 64 * (j & 1), da, db, idesc_s, k > 0);
        }
        umma_commit(s_full0 + 16 * m + 8 * (j & 1));
      };
      auto wait_k = [&](int j) {
        mbar_wait(k_full0 + 8 * (j % DT_K_STAGES), (j / DT_K_STAGES) & 1, error, 13);
        tc_fence_after_sync();
      };
      for (int j = 0; j < min(2, n_pages); ++j) {
        wait_k(j);
        issue_s(j, 0);
        issue_s(j, 1);
        umma_commit(k_empty0 + 8 * (j % DT_K_STAGES));
      }
      for (int j = 0; j < n_pages; ++j) {
        const int st = j % DT_V_STAGES, buf = j & 1;
        mbar_wait(v_full0 + 8 * st, (j / DT_V_STAGES) & 1, error, 9);
        for (int m = 0; m < 2; ++m) {
          mbar_wait(p_full0 + 16 * m + 8 * buf, (j >> 1) & 1, error, 15);
          tc_fence_after_sync();
          const uint32_t tP = tmem + 128 * m + 64 * buf;
#pragma unroll
          for (int i = 0; i < VH; ++i)
#pragma unroll
            for (int k = 0; k < MB_PAGE / 16; ++k) {
              const uint64_t db =
                  umma_desc_mn128(sV + st * V_BYTES + i * DT_HALF + k * 2048, DT_HALF);
              umma_bf16_ts(tmem + 256 + 128 * m + 64 * i, tP + 8 * k, db, idesc_o, (j | k) != 0);
            }
          umma_commit(o_done0 + 16 * m + 8 * buf);
        }
        umma_commit(v_empty0 + 8 * st);  // V of this page has been read by both
        if (j + 2 < n_pages) {
          // S of page j + 2 overwrites the P that the product just issued reads as an operand:
          // wait until that product is done
          wait_k(j + 2);
          for (int m = 0; m < 2; ++m) {
            mbar_wait(o_done0 + 16 * m + 8 * buf, (j >> 1) & 1, error, 14);
            tc_fence_after_sync();
            issue_s(j + 2, m);
          }
          umma_commit(k_empty0 + 8 * ((j + 2) % DT_K_STAGES));
        }
      }
    }
  } else {
    const int m = warp >= 6;     // the map
    const int q = warp & 3;      // the TMEM lanes of this warp
    const int row = q * 32 + lane;
    const int pos = past + row0 + row;  // position of this thread's token
    const int lo = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const uint32_t tS = tmem + 128 * m + lane_addr, tO = tmem + 256 + 128 * m + lane_addr;
    const uint32_t s_full = s_full0 + 16 * m, p_full = p_full0 + 16 * m, o_done = o_done0 + 16 * m;
    float m_ref = -INFINITY, l = 0.f;
    for (int j = 0; j < n_pages; ++j) {
      const uint32_t tSj = tS + 64 * (j & 1);
      mbar_wait(s_full + 8 * (j & 1), (j >> 1) & 1, error, 16);
      tc_fence_after_sync();
      float s[MB_PAGE];
      tmem_ld64(tSj, s);
      const int key0 = (page0 + j) * MB_PAGE;
      // a page that every row of the warp sees whole needs no mask (uniform over the warp)
      const bool whole = key0 + MB_PAGE - 1 <= pos - lane &&
                         (window == 0 || key0 >= lo + (31 - lane));
      if (!whole) {
#pragma unroll
        for (int c = 0; c < MB_PAGE; ++c) {
          const int key = key0 + c;
          if (!(key >= lo && key <= pos)) s[c] = -INFINITY;
        }
      }
      // the scale is positive: the maximum of the raw scores is the scaled ones' maximum too
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < MB_PAGE; c += 2) mx4[(c >> 1) & 3] = max3(mx4[(c >> 1) & 3], s[c], s[c + 1]);
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;
      // O is rescaled only when this row's maximum has grown by more than 2^8 (or appears for
      // the first time); until then the old reference stays and P may reach 2^8
      const bool grow = mx > m_ref + 8.0f || (m_ref == -INFINITY && mx > -INFINITY);
      if (__any_sync(0xffffffffu, grow)) {
        const float f = grow ? (m_ref == -INFINITY ? 0.f : exp2f(m_ref - mx)) : 1.f;
        if (j > 0) {
          // the second product of the page before adds into O: it must be done
          mbar_wait(o_done + 8 * ((j - 1) & 1), ((j - 1) >> 1) & 1, error, 17);
          tc_fence_after_sync();
#pragma unroll 1
          for (int c0 = 0; c0 < VD; c0 += 16) {
            float o[16];
            tmem_ld16(tO + c0, o);
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] *= f;
            tmem_st16(tO + c0, o);
          }
        }
        l *= f;
        if (grow) m_ref = mx;
      }
      const float ref = m_ref == -INFINITY ? 0.f : m_ref;
      // P over the S just read, as the first operand of the second product: this thread's row,
      // two bfloat16 values a column, keys in order
      const unsigned long long scale2 = pack2(scale_log2, scale_log2), ref2 = pack2(-ref, -ref);
      unsigned long long l4[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
      for (int c16 = 0; c16 < 2; ++c16) {
        uint32_t w[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float x0, x1;
          unpack2(fma2(pack2(s[c16 * 32 + 2 * i], s[c16 * 32 + 2 * i + 1]), scale2, ref2), x0, x1);
          const float p0 = ex2(x0), p1 = ex2(x1);
          l4[i & 3] = add2(l4[i & 3], pack2(p0, p1));
          __nv_bfloat162 v = __floats2bfloat162_rn(p0, p1);
          w[i] = *reinterpret_cast<uint32_t*>(&v);
        }
        tmem_st16_u32(tSj + 16 * c16, w);
      }
      {
        float a0, a1;
        unpack2(add2(add2(l4[0], l4[1]), add2(l4[2], l4[3])), a0, a1);
        l += a0 + a1;
      }
      tmem_wait_st();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full + 8 * (j & 1));
    }
    // the map's last product done means all of its are (the tensor core works in the order of
    // issue); its warps tell the other map's at the barrier
    mbar_wait(o_done + 8 * ((n_pages - 1) & 1), ((n_pages - 1) >> 1) & 1, error, 18);
    sm_rows[m * DT_ROWS + row] = (m ? lam : 1.0f) / l;
    tc_fence_before_sync();
    softmax_sync();
    tc_fence_after_sync();
    const float i1 = sm_rows[row], i2 = sm_rows[DT_ROWS + row];
    constexpr int COLS = VD / 2;           // this thread's columns: COLS * m ..
    float v[COLS], sum = 0.f;
#pragma unroll
    for (int c0 = 0; c0 < COLS; c0 += 16) {
      float a[16], d[16];
      tmem_ld16(tmem + 256 + lane_addr + COLS * m + c0, a);
      tmem_ld16(tmem + 384 + lane_addr + COLS * m + c0, d);
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        v[c0 + i] = a[i] * i1 - d[i] * i2;
        sum = fmaf(v[c0 + i], v[c0 + i], sum);
      }
    }
    sm_rows[(2 + m) * DT_ROWS + row] = sum;
    softmax_sync();
    const float f = factor / sqrtf((sm_rows[2 * DT_ROWS + row] + sm_rows[3 * DT_ROWS + row]) /
                                       (float)VD + eps);
    // Q's shared memory is free now: a warp lays its 32 half rows there (16-byte piece p of row
    // r at p ^ (r & 7), pieces per half row a power of two) and writes whole half rows out
    constexpr int PIECES = COLS / 8, RPI = 32 / PIECES;    // rows an instruction writes
    const uint32_t stage = sQ + (uint32_t)(m * 4 + q) * (32 * COLS * 2);
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
      uint32_t w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        __nv_bfloat162 x = __floats2bfloat162_rn(v[8 * p + 2 * i] * f, v[8 * p + 2 * i + 1] * f);
        w[i] = *reinterpret_cast<uint32_t*>(&x);
      }
      st_shared_v4(stage + lane * (COLS * 2) + ((p ^ (lane & (PIECES - 1))) << 4),
                   make_uint4(w[0], w[1], w[2], w[3]));
    }
    __syncwarp();
    const int p = lane % PIECES;
#pragma unroll 4
    for (int i = 0; i < PIECES; ++i) {
      const int r = RPI * i + lane / PIECES;
      if (row0 + q * 32 + r < n_new) {
        const uint4 x = ld_shared_v4(stage + r * (COLS * 2) + ((p ^ (r & (PIECES - 1))) << 4));
        *(uint4*)(out + ((size_t)(start + row0 + q * 32 + r) * nh + h) * VD + COLS * m + 8 * p) = x;
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, DT_TMEM_COLS);
}

// out[t, h, :] for the new tokens of B sequences over the cache. q [T, nh * 128] bfloat16 (a
// head's two maps of 64 one after the other); kpool [pool_rows, 128], vpool [pool_rows, vd] with
// pool_rows = pages * kv_heads * 64; out [T, nh * vd]. `error`: a device word that receives
// 9..19 if a wait in the kernel ran out.
MB_EXPORT int mb_attention_diff_prefill_tc(const void* q, void* out, const void* kpool,
                                           const void* vpool, long long pool_rows,
                                           const int* page_table, int max_pages, int ring_pages,
                                           const int* seq_start, const int* seq_past,
                                           const int* seq_slot, int B, int T, int max_new, int nh,
                                           int nkv, int dim, int vd, int window, float scale,
                                           float lam, float factor, float eps, int* error,
                                           void* stream) {
  if (B <= 0 || max_new <= 0) return 0;
  if (dim != 64 || (vd != 64 && vd != 128))
    MB_FAIL("mb_attention_diff_prefill_tc: maps of %d and value rows of %d (64; 64 or 128)", dim, vd);
  if (nkv <= 0 || nh % nkv) MB_FAIL("mb_attention_diff_prefill_tc: %d heads on %d KV heads", nh, nkv);
  if ((uintptr_t)out & 15) MB_FAIL("mb_attention_diff_prefill_tc: out is not 16-byte aligned");
  const int row_tiles = (max_new + DT_ROWS - 1) / DT_ROWS;
  if (B > 65535 || row_tiles > 65535)
    MB_FAIL("mb_attention_diff_prefill_tc: %d sequences, %d new tokens in one", B, max_new);
  if (!(scale > 0.f))  // the row maximum is taken over the scores before they are scaled
    MB_FAIL("mb_attention_diff_prefill_tc: a scale of %g (it must be positive)", (double)scale);
  CUtensorMap tmQ, tmK, tmV;
  const char* who = "mb_attention_diff_prefill_tc";
  if (!mb_make_map_bf16(&tmQ, q, T, nh * 128, nh * 128, DT_ROWS, who)) return -1;
  if (!mb_make_map_bf16(&tmK, kpool, pool_rows, 128, 128, MB_PAGE, who)) return -1;
  if (!mb_make_map_bf16(&tmV, vpool, pool_rows, vd, vd, MB_PAGE, who)) return -1;
  dim3 grid(nh, row_tiles, B);
#define GO(VD_)                                                                                \
  {                                                                                            \
    constexpr int smem = DT_FIXED + DT_V_STAGES * (VD_ / 64) * DT_HALF + DT_TAIL;              \
    static bool configured = false;                                                            \
    if (!configured) {                                                                         \
      cudaError_t e = cudaFuncSetAttribute(diff_prefill_tc_kernel<VD_>,                        \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, smem); \
      if (e != cudaSuccess) MB_FAIL("%s: %s", who, cudaGetErrorString(e));                     \
      configured = true;                                                                       \
    }                                                                                          \
    mb_launch(diff_prefill_tc_kernel<VD_>, grid, dim3(DT_THREADS), smem, (cudaStream_t)stream, \
              tmQ, tmK, tmV, (bf16*)out, page_table, max_pages, ring_pages, seq_start,         \
              seq_past, seq_slot, nh, nkv, window, scale * 1.4426950408889634f, lam, factor,   \
              eps, error);                                                                     \
  }
  if (vd == 64) GO(64) else GO(128)
#undef GO
  MB_CHECK_LAUNCH("mb_attention_diff_prefill_tc");
}
