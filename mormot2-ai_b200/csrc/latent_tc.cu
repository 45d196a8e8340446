// Latent attention of long steps (prompts) on the fifth-generation tensor cores, with keys and
// values formed per head.
//
// The other kernels of latent attention (latent.cu, latent_mma.cu) never form them: every head
// scores rows of kv_rank + rot_dim values and sums rows of kv_rank. That reads the least memory,
// which counts for a decode step; a prompt's many queries pay for it with three to four times the
// multiply-adds. Here the latents that the step's queries can see are gathered from the cache into
// one matrix (latent_gather), one plain product with [W_uk ; W_uv] gives every head's keys and
// values for them, the queries' rotated parts turn in place (latent_q_rope), and
//     S = Q_plain Kᵀ + Q_rot rᵀ,   O += P V
// are tcgen05.mma instructions with their accumulators in tensor memory, the tiles by TMA
// (128-byte swizzle), as in attention_tc.cu. The rotated key part r, the same for all heads, is
// one more block of 64 columns of the K tile, filled up with zeros: what lies behind a head's
// rotated query part then counts nothing.
//
// A CTA takes 256 consecutive new tokens of one sequence and one query head (the only CTA of its
// SM) as two row tiles of 128 that share every K and V tile:
//   warp 0      loads Q once, then K and V of 64 keys after 64 keys into rings of stages;
//   warp 1      issues S of both row tiles two steps ahead, each into one of two buffers of its
//               tile, and O += P V when P of a step is ready: the products of one row tile run
//               under the softmax of the other;
//   warps 2-5   the first row tile's softmax, warps 6-9 the second's, a row a thread (P over the
//               S just read, O rescaled only when a row's maximum has grown by more than 2^8).
// A row tile takes part only in the steps whose keys one of its rows can see.
//
// Keys of sequence b: positions lo_b = max(0, past + 1 - window) .. past + new - 1, rows base_b ..
// of the gathered matrix, base_b the sum of the sequences before. Every block forms base_b from
// the step's index arrays.
#include "attention_tc.cuh"

MB_DEFINE_LAST_ERROR

typedef __nv_bfloat16 bf16;

#define LT_ROWS 128
#define LT_K_STAGES 3
#define LT_V_STAGES 2
#define LT_THREADS 320
#define LT_HALF (MB_PAGE * 64 * 2)          // 8 KB: 64 keys x 64 columns
#define LT_Q_HALF (LT_ROWS * 64 * 2)        // 16 KB: 128 rows x 64 columns
#define LT_TMEM_COLS 512                    // S of tile m: 128 m, two buffers of 64; O of tile m: 256 + 128 m

// The first gathered row of sequence b and the position that it holds.
__device__ __forceinline__ int gathered_base(const int* __restrict__ seq_start,
                                             const int* __restrict__ seq_past, int b, int window,
                                             int& lo) {
  int base = 0;
  for (int i = 0; i < b; ++i) {
    const int past = seq_past[i];
    const int first = window > 0 ? max(0, past + 1 - window) : 0;
    base += past + seq_start[i + 1] - seq_start[i] - first;
  }
  lo = window > 0 ? max(0, seq_past[b] + 1 - window) : 0;
  return base;
}

// ------------------------------------------------------------------ latent_gather
// Row r of the step's keys: its latent [kv_rank] into c_out, its rotated part [rot_dim] and zeros
// up to 64 values into r_out. A warp a row, 16 bytes a lane.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const bf16* __restrict__ pool, const int* __restrict__ page_table,
                     int max_pages, int ring_pages, const int* __restrict__ seq_start,
                     const int* __restrict__ seq_past, const int* __restrict__ seq_slot, int B,
                     int R, int kv_rank, int rot_dim, int window, bf16* __restrict__ c_out,
                     bf16* __restrict__ r_out) {
  mb_grid_wait();
  mb_grid_launch_next();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= R) return;
  int b = 0, base = 0, lo = 0;
  for (;; ++b) {
    const int past = seq_past[b];
    lo = window > 0 ? max(0, past + 1 - window) : 0;
    const int rows = past + seq_start[b + 1] - seq_start[b] - lo;
    if (r < base + rows || b + 1 >= B) break;
    base += rows;
  }
  const int dk = kv_rank + rot_dim;
  const bf16* src = pool + kv_row(page_table, max_pages, ring_pages, seq_slot[b], lo + r - base, 1, 0) * dk;
  for (int i = 8 * lane; i < kv_rank; i += 256)
    *(uint4*)(c_out + (size_t)r * kv_rank + i) = *(const uint4*)(src + i);
  if (lane < 8)
    *(uint4*)(r_out + (size_t)r * 64 + 8 * lane) =
        8 * lane < rot_dim ? *(const uint4*)(src + kv_rank + 8 * lane) : make_uint4(0, 0, 0, 0);
}

// `R`: the rows of all sequences together, as the host counts them.
MB_EXPORT int mb_latent_gather(const void* pool, const int* page_table, int max_pages,
                               int ring_pages, const int* seq_start, const int* seq_past,
                               const int* seq_slot, int B, int R, int kv_rank, int rot_dim,
                               int window, void* c_out, void* r_out, void* stream) {
  if (R <= 0 || B <= 0) return 0;
  if (kv_rank % 8 || rot_dim % 8 || rot_dim > 64 ||
      (((uintptr_t)pool | (uintptr_t)c_out | (uintptr_t)r_out) & 15))
    MB_FAIL("mb_latent_gather: rows of %d + %d values", kv_rank, rot_dim);
  mb_launch(latent_gather_kernel, dim3((R + 7) / 8), dim3(256), 0, (cudaStream_t)stream,
            (const bf16*)pool, page_table, max_pages, ring_pages, seq_start, seq_past, seq_slot, B,
            R, kv_rank, rot_dim, window, (bf16*)c_out, (bf16*)r_out);
  MB_CHECK_LAUNCH("mb_latent_gather");
}

// ------------------------------------------------------------------ latent_q_rope
// The rotated part of every head of q [T, nh * (dim + rot_dim)], in place: of its rot_dim values
// the first rot_dims turn, pair (i, i + rot_dims / 2), cosine and sine times `amp`.
__global__ void __launch_bounds__(256)
latent_q_rope_kernel(bf16* __restrict__ q, int ld, int nh, int dim, int rot_dim, int rot_dims,
                     const float* __restrict__ inv_freq, float amp,
                     const int* __restrict__ tok_pos) {
  extern __shared__ float lq_angles[];   // [rot_dims / 2] cosines, then sines
  const int half = rot_dims >> 1, t = blockIdx.x, pos = tok_pos[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(inv_freq[i] * (float)pos, &s, &c);
    lq_angles[i] = c * amp;
    lq_angles[half + i] = s * amp;
  }
  __syncthreads();
  mb_grid_wait();
  mb_grid_launch_next();
  if ((half & 1) == 0) {   // two neighbouring pairs at a time (dim and rot_dim are multiples of 8)
    const int quarter = half >> 1;
    for (int n = threadIdx.x; n < nh * quarter; n += blockDim.x) {
      const int h = n / quarter, i = 2 * (n - h * quarter);
      __nv_bfloat162* p = (__nv_bfloat162*)(q + (size_t)t * ld + (size_t)h * (dim + rot_dim) + dim + i);
      const float2 u = __bfloat1622float2(p[0]), v = __bfloat1622float2(p[quarter]);
      const float c0 = lq_angles[i], s0 = lq_angles[half + i];
      const float c1 = lq_angles[i + 1], s1 = lq_angles[half + i + 1];
      p[0] = __floats2bfloat162_rn(u.x * c0 - v.x * s0, u.y * c1 - v.y * s1);
      p[quarter] = __floats2bfloat162_rn(v.x * c0 + u.x * s0, v.y * c1 + u.y * s1);
    }
    return;
  }
  for (int n = threadIdx.x; n < nh * half; n += blockDim.x) {
    const int h = n / half, i = n - h * half;
    bf16* p = q + (size_t)t * ld + (size_t)h * (dim + rot_dim) + dim + i;
    const float u = __bfloat162float(p[0]), v = __bfloat162float(p[half]);
    const float c = lq_angles[i], s = lq_angles[half + i];
    p[0] = __float2bfloat16_rn(u * c - v * s);
    p[half] = __float2bfloat16_rn(v * c + u * s);
  }
}

MB_EXPORT int mb_latent_q_rope(void* q, int ld, int T, int nh, int dim, int rot_dim, int rot_dims,
                               const float* inv_freq, float amp, const int* tok_pos,
                               void* stream) {
  if (T <= 0 || rot_dims <= 0) return 0;
  if (rot_dims > rot_dim || (rot_dims & 1) || inv_freq == nullptr || dim % 8 || rot_dim % 8 ||
      ld % 8 || ((uintptr_t)q & 15))
    MB_FAIL("mb_latent_q_rope: %d of %d values rotate", rot_dims, rot_dim);
  mb_launch(latent_q_rope_kernel, dim3(T), dim3(256), (size_t)rot_dims * sizeof(float),
            (cudaStream_t)stream, (bf16*)q, ld, nh, dim, rot_dim, rot_dims, inv_freq, amp, tok_pos);
  MB_CHECK_LAUNCH("mb_latent_q_rope");
}

// ------------------------------------------------------------------ the attention
// DH: 64-column blocks of a head's plain part (dim = 64 DH); VH: of a value row.
template <int DH, int VH>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ,
                         const __grid_constant__ CUtensorMap tmKV,
                         const __grid_constant__ CUtensorMap tmR, bf16* __restrict__ out,
                         int out_stride, const int* __restrict__ seq_start,
                         const int* __restrict__ seq_past, int nh, int rot_dim, int window,
                         float scale_log2, int* __restrict__ error, const bf16* __restrict__ gate,
                         int gate_stride) {
  constexpr int VD = 64 * VH, DIM = 64 * DH;
  constexpr int Q_BYTES = (DH + 1) * LT_Q_HALF, K_BYTES = (DH + 1) * LT_HALF, V_BYTES = VH * LT_HALF;
  extern __shared__ __align__(1024) uint8_t lt_smem[];
  const uint32_t raw = smem_u32(lt_smem);
  if (raw & 1023u) {  // swizzled tiles need it; never seen, but a wrong result must not follow
    if (threadIdx.x == 0 && error) atomicCAS(error, 0, 19);
    return;
  }
  const uint32_t sQ = raw;                              // [row tile][Q_BYTES]
  const uint32_t sK = sQ + 2 * Q_BYTES;                 // [stage][K_BYTES]
  const uint32_t sV = sK + LT_K_STAGES * K_BYTES;       // [stage][V_BYTES]
  const uint32_t bars = sV + LT_V_STAGES * V_BYTES;
  const uint32_t q_full = bars, k_full0 = bars + 8, k_empty0 = k_full0 + 8 * LT_K_STAGES;
  const uint32_t v_full0 = k_empty0 + 8 * LT_K_STAGES, v_empty0 = v_full0 + 8 * LT_V_STAGES;
  // for each row tile m and buffer b, at 16 m + 8 b: S ready, P ready, the second product done
  const uint32_t s_full0 = v_empty0 + 8 * LT_V_STAGES, p_full0 = s_full0 + 32;
  const uint32_t o_done0 = p_full0 + 32, slot = o_done0 + 32;
  volatile uint32_t* slot_ptr = (volatile uint32_t*)(lt_smem + (slot - raw));

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.x;
  const int start = seq_start[b], n_new = seq_start[b + 1] - start;
  const int row0 = (int)(gridDim.y - 1 - blockIdx.y) * 2 * LT_ROWS;   // the longest first
  if (row0 >= n_new) return;  // the whole CTA, before anything is set up
  const int past = seq_past[b];
  int lo_b;
  const int base = gathered_base(seq_start, seq_past, b, window, lo_b);
  const int first_pos = past + row0, last_pos = past + min(row0 + 2 * LT_ROWS - 1, n_new - 1);
  const int key_lo = (window > 0 && first_pos + 1 > window) ? first_pos + 1 - window : 0;
  const int steps = (last_pos - key_lo) / MB_PAGE + 1;
  // the steps of row tile m: from the first key of its first row to its last row
  auto tile_lo = [&](int m) {
    const int p = first_pos + m * LT_ROWS;
    return p > last_pos ? 0 : ((window > 0 && p + 1 > window ? p + 1 - window : 0) - key_lo) / MB_PAGE;
  };
  auto tile_hi = [&](int m) {
    const int p = first_pos + m * LT_ROWS;
    return p > last_pos ? 0 : (min(p + LT_ROWS - 1, last_pos) - key_lo) / MB_PAGE + 1;
  };
  const int lo0 = tile_lo(0), hi0 = tile_hi(0), lo1 = tile_lo(1), hi1 = tile_hi(1);

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < LT_K_STAGES; ++i) {
      mbar_init(k_full0 + 8 * i, 1);
      mbar_init(k_empty0 + 8 * i, 1);
    }
    for (int i = 0; i < LT_V_STAGES; ++i) {
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
    tma_prefetch_desc(&tmKV);
    tma_prefetch_desc(&tmR);
  }
  if (warp == 1) tmem_alloc(slot, LT_TMEM_COLS);
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *slot_ptr;
  mb_grid_wait();  // queries, keys and values come from the kernels before
  mb_grid_launch_next();

  if (warp == 0) {
    if (elect_one()) {
      mbar_expect_tx(q_full, 2 * Q_BYTES);
      for (int m = 0; m < 2; ++m)
        for (int i = 0; i <= DH; ++i)
          tma_load_2d(sQ + m * Q_BYTES + i * LT_Q_HALF, &tmQ, h * (DIM + rot_dim) + 64 * i,
                      start + row0 + m * LT_ROWS, q_full);
      const int y0 = base + key_lo - lo_b;
      auto load_k = [&](int j) {
        const int st = j % LT_K_STAGES, y = y0 + j * MB_PAGE;
        mbar_wait(k_empty0 + 8 * st, ((j / LT_K_STAGES) & 1) ^ 1, error, 11);
        mbar_expect_tx(k_full0 + 8 * st, K_BYTES);
        for (int i = 0; i < DH; ++i)
          tma_load_2d(sK + st * K_BYTES + i * LT_HALF, &tmKV, h * DIM + 64 * i, y, k_full0 + 8 * st);
        tma_load_2d(sK + st * K_BYTES + DH * LT_HALF, &tmR, 0, y, k_full0 + 8 * st);
      };
      // the first products run two steps ahead of the second ones: so do the loads of K
      load_k(0);
      if (steps > 1) load_k(1);
      for (int j = 0; j < steps; ++j) {
        if (j + 2 < steps) load_k(j + 2);
        const int st = j % LT_V_STAGES, y = y0 + j * MB_PAGE;
        mbar_wait(v_empty0 + 8 * st, ((j / LT_V_STAGES) & 1) ^ 1, error, 10);
        mbar_expect_tx(v_full0 + 8 * st, V_BYTES);
        for (int i = 0; i < VH; ++i)
          tma_load_2d(sV + st * V_BYTES + i * LT_HALF, &tmKV, nh * DIM + h * VD + 64 * i, y,
                      v_full0 + 8 * st);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(LT_ROWS, MB_PAGE);             // K-major both
      constexpr uint32_t idesc_o = umma_idesc_bf16(LT_ROWS, 64) | (1u << 16);     // B MN-major
      mbar_wait(q_full, 0, error, 12);
      // S of row tile m and step j goes into the tile's buffer of its own step number i = j - lo,
      // which held S and then P of the step before last
      auto issue_s = [&](int j, int m, int i) {
        const int st = j % LT_K_STAGES;
#pragma unroll
        for (int k = 0; k < 4 * (DH + 1); ++k) {
          const uint64_t da =
              umma_desc_k128(sQ + m * Q_BYTES + (k / 4) * LT_Q_HALF + (k % 4) * 32);
          const uint64_t db = umma_desc_k128(sK + st * K_BYTES + (k / 4) * LT_HALF + (k % 4) * 32);
          umma_bf16(tmem + 128 * m + 64 * (i & 1), da, db, idesc_s, k > 0);
        }
        umma_commit(s_full0 + 16 * m + 8 * (i & 1));
      };
      // everything that step j's keys are multiplied with, then its stage is free
      auto first_products = [&](int j) {
        mbar_wait(k_full0 + 8 * (j % LT_K_STAGES), (j / LT_K_STAGES) & 1, error, 13);
        tc_fence_after_sync();
        for (int m = 0; m < 2; ++m) {
          const int lo = m ? lo1 : lo0, hi = m ? hi1 : hi0, i = j - lo;
          if (j < lo || j >= hi) continue;
          if (i >= 2) {
            // it overwrites the P that an earlier product reads as an operand: wait until that
            // product is done
            mbar_wait(o_done0 + 16 * m + 8 * (i & 1), ((i - 2) >> 1) & 1, error, 14);
            tc_fence_after_sync();
          }
          issue_s(j, m, i);
        }
        umma_commit(k_empty0 + 8 * (j % LT_K_STAGES));
      };
      for (int j = 0; j < min(2, steps); ++j) first_products(j);
      for (int j = 0; j < steps; ++j) {
        const int st = j % LT_V_STAGES;
        mbar_wait(v_full0 + 8 * st, (j / LT_V_STAGES) & 1, error, 9);
        for (int m = 0; m < 2; ++m) {
          const int lo = m ? lo1 : lo0, hi = m ? hi1 : hi0, i = j - lo;
          if (j < lo || j >= hi) continue;
          mbar_wait(p_full0 + 16 * m + 8 * (i & 1), (i >> 1) & 1, error, 15);
          tc_fence_after_sync();
          const uint32_t tP = tmem + 128 * m + 64 * (i & 1);
#pragma unroll
          for (int c = 0; c < VH; ++c)
#pragma unroll
            for (int k = 0; k < MB_PAGE / 16; ++k) {
              const uint64_t db = umma_desc_mn128(sV + st * V_BYTES + c * LT_HALF + k * 2048, LT_HALF);
              umma_bf16_ts(tmem + 256 + 128 * m + 64 * c, tP + 8 * k, db, idesc_o, (i | k) != 0);
            }
          umma_commit(o_done0 + 16 * m + 8 * (i & 1));
        }
        umma_commit(v_empty0 + 8 * st);  // V of this step has been read by both
        if (j + 2 < steps) first_products(j + 2);
      }
    }
  } else {
    const int m = warp >= 6;     // the row tile
    const int q = warp & 3;      // the TMEM lanes of this warp
    const int row = m * LT_ROWS + q * 32 + lane;
    const int pos = first_pos + row;    // position of this thread's token
    const int lo = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
    const int j_lo = m ? lo1 : lo0, n = (m ? hi1 : hi0) - j_lo;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const uint32_t tS = tmem + 128 * m + lane_addr, tO = tmem + 256 + 128 * m + lane_addr;
    const uint32_t s_full = s_full0 + 16 * m, p_full = p_full0 + 16 * m, o_done = o_done0 + 16 * m;
    float m_ref = -INFINITY, l = 0.f;
    for (int i = 0; i < n; ++i) {
      const uint32_t tSj = tS + 64 * (i & 1);
      mbar_wait(s_full + 8 * (i & 1), (i >> 1) & 1, error, 16);
      tc_fence_after_sync();
      float s[MB_PAGE];
      tmem_ld64(tSj, s);
      const int key0 = key_lo + (j_lo + i) * MB_PAGE;
      // a step that every row of the warp sees whole needs no mask (uniform over the warp)
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
      const bool grow = mx > m_ref + 8.0f || (m_ref == -INFINITY && mx > -INFINITY);
      if (__any_sync(0xffffffffu, grow)) {
        const float f = grow ? (m_ref == -INFINITY ? 0.f : exp2f(m_ref - mx)) : 1.f;
        if (i > 0) {
          // the second product of the step before adds into O: it must be done
          mbar_wait(o_done + 8 * ((i - 1) & 1), ((i - 1) >> 1) & 1, error, 17);
          tc_fence_after_sync();
#pragma unroll 1
          for (int c0 = 0; c0 < VD; c0 += 16) {
            float o[16];
            tmem_ld16(tO + c0, o);
#pragma unroll
            for (int k = 0; k < 16; ++k) o[k] *= f;
            tmem_st16(tO + c0, o);
          }
        }
        l *= f;
        if (grow) m_ref = mx;
      }
      const float ref = m_ref == -INFINITY ? 0.f : m_ref;
      // P over the S just read, as the first operand of the second product
      const unsigned long long scale2 = pack2(scale_log2, scale_log2), ref2 = pack2(-ref, -ref);
      unsigned long long l4[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
      for (int c16 = 0; c16 < 2; ++c16) {
        uint32_t w[16];
#pragma unroll
        for (int k = 0; k < 16; ++k) {
          float x0, x1;
          unpack2(fma2(pack2(s[c16 * 32 + 2 * k], s[c16 * 32 + 2 * k + 1]), scale2, ref2), x0, x1);
          const float p0 = ex2(x0), p1 = ex2(x1);
          l4[k & 3] = add2(l4[k & 3], pack2(p0, p1));
          __nv_bfloat162 v = __floats2bfloat162_rn(p0, p1);
          w[k] = *reinterpret_cast<uint32_t*>(&v);
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
      if (lane == 0) mbar_arrive(p_full + 8 * (i & 1));
    }
    if (n > 0) {
      // the last product done means all of the tile's are (the tensor core works in the order of
      // issue), those that read its Q among them
      mbar_wait(o_done + 8 * ((n - 1) & 1), ((n - 1) >> 1) & 1, error, 18);
      tc_fence_after_sync();
      const float inv = 1.0f / l;
      const bf16* gates = gate != nullptr && row0 + row < n_new
                              ? gate + (size_t)(start + row0 + row) * gate_stride + (size_t)h * VD
                              : nullptr;
      // the tile's Q memory is free now: a warp lays its 32 rows there (16-byte piece p of row r
      // at p ^ (r & 7): no bank conflicts either way) and writes whole rows out
      const uint32_t stage = sQ + m * Q_BYTES + (uint32_t)q * (32 * VD * 2);
#pragma unroll 1
      for (int c0 = 0; c0 < VD; c0 += 16) {
        float o[16];
        tmem_ld16(tO + c0, o);
        if (gates != nullptr) {
          const uint4 ga = *(const uint4*)(gates + c0), gb = *(const uint4*)(gates + c0 + 8);
          const uint32_t gw[8] = {ga.x, ga.y, ga.z, ga.w, gb.x, gb.y, gb.z, gb.w};
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const float2 gv = __bfloat1622float2(*(const __nv_bfloat162*)&gw[i]);
            o[2 * i] *= sigmoid_fast(gv.x);
            o[2 * i + 1] *= sigmoid_fast(gv.y);
          }
        }
        uint32_t w[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          __nv_bfloat162 v = __floats2bfloat162_rn(o[2 * i] * inv, o[2 * i + 1] * inv);
          w[i] = *reinterpret_cast<uint32_t*>(&v);
        }
        const int pc = c0 >> 3;
        st_shared_v4(stage + lane * (VD * 2) + ((pc ^ (lane & 7)) << 4),
                     make_uint4(w[0], w[1], w[2], w[3]));
        st_shared_v4(stage + lane * (VD * 2) + (((pc + 1) ^ (lane & 7)) << 4),
                     make_uint4(w[4], w[5], w[6], w[7]));
      }
      __syncwarp();
      constexpr int PIECES = VD / 8, AT_ONCE = 32 / PIECES;
      const int pc = lane % PIECES, first_row = row0 + m * LT_ROWS + q * 32;
#pragma unroll 4
      for (int i = 0; i < 32 / AT_ONCE; ++i) {
        const int r = AT_ONCE * i + lane / PIECES;
        if (first_row + r < n_new) {
          const uint4 v = ld_shared_v4(stage + r * (VD * 2) + ((pc ^ (r & 7)) << 4));
          *(uint4*)(out + (size_t)(start + first_row + r) * out_stride + (size_t)h * VD + 8 * pc) = v;
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, LT_TMEM_COLS);
}

// out[t, h, :] for the new tokens of B sequences. q [T, nh * (dim + rot_dim)] with its rotated
// parts turned; kv [R, nh * (dim + vd)]: the gathered rows' keys of all heads, then their values;
// rot [R, 64]; gate (may be null) [T, >= nh * vd]. `error`: a device word that receives 9..19 if
// a wait in the kernel ran out.
MB_EXPORT int mb_latent_prefill_tc(const void* q, int q_stride, const void* kv, int kv_stride,
                                   const void* rot, int R, void* out, int out_stride,
                                   const int* seq_start, const int* seq_past, int B, int T,
                                   int max_new, int nh, int dim, int rot_dim, int vd, int window,
                                   float scale, int* error, const void* gate, int gate_stride,
                                   void* stream) {
  if (B <= 0 || max_new <= 0) return 0;
  const char* who = "mb_latent_prefill_tc";
  if ((dim != 64 && dim != 128) || (vd != 64 && vd != 128) || rot_dim < 0 || rot_dim > 64 || rot_dim % 8)
    MB_FAIL("%s: heads of %d + %d and %d values", who, dim, rot_dim, vd);
  if (((uintptr_t)out & 15) || (out_stride & 7) ||
      (gate != nullptr && (((uintptr_t)gate & 15) || (gate_stride & 7))))
    MB_FAIL("%s: out or the gates are not 16-byte aligned", who);
  if (!(scale > 0.f))  // the row maximum is taken over the scores before they are scaled
    MB_FAIL("%s: a scale of %g (it must be positive)", who, (double)scale);
  const int row_tiles = (max_new + 2 * LT_ROWS - 1) / (2 * LT_ROWS);
  if (B > 65535 || row_tiles > 65535) MB_FAIL("%s: %d sequences, %d new tokens in one", who, B, max_new);
  CUtensorMap tmQ, tmKV, tmR;
  if (!mb_make_map_bf16(&tmQ, q, T, (long long)nh * (dim + rot_dim), q_stride, LT_ROWS, who)) return -1;
  if (!mb_make_map_bf16(&tmKV, kv, R, (long long)nh * (dim + vd), kv_stride, MB_PAGE, who)) return -1;
  if (!mb_make_map_bf16(&tmR, rot, R, 64, 64, MB_PAGE, who)) return -1;
  dim3 grid(nh, row_tiles, B);
#define GO(DH_, VH_)                                                                           \
  {                                                                                            \
    constexpr int smem = 2 * (DH_ + 1) * LT_Q_HALF + LT_K_STAGES * (DH_ + 1) * LT_HALF +       \
                         LT_V_STAGES * VH_ * LT_HALF + 256;                                    \
    static bool configured = false;                                                            \
    if (!configured) {                                                                         \
      cudaError_t e = cudaFuncSetAttribute(latent_prefill_tc_kernel<DH_, VH_>,                 \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, smem); \
      if (e != cudaSuccess) MB_FAIL("%s: %s", who, cudaGetErrorString(e));                     \
      configured = true;                                                                       \
    }                                                                                          \
    mb_launch(latent_prefill_tc_kernel<DH_, VH_>, grid, dim3(LT_THREADS), smem,                \
              (cudaStream_t)stream, tmQ, tmKV, tmR, (bf16*)out, out_stride, seq_start,         \
              seq_past, nh, rot_dim, window, scale * 1.4426950408889634f, error,               \
              (const bf16*)gate, gate_stride);                                                 \
  }
  if (dim == 128) { if (vd == 128) GO(2, 2) else GO(2, 1) }
  else { if (vd == 128) GO(1, 2) else GO(1, 1) }
#undef GO
  MB_CHECK_LAUNCH("mb_latent_prefill_tc");
}
