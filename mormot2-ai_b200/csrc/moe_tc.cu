// The routed experts' two products on the fifth-generation tensor cores (bfloat16), over the
// lists that moe.cu plans in tiles of 128 rows:
//   moe_gather    the rows that the first product reads, copied into list order (a TMA tile is
//                 128 rows that lie one after the other)
//   moe_gemm_tc   up:   act[r, :] = f(rows[r] · Wᵀ)           (f of one input, or gate and up)
//                 down: y[a(r), :] = weight[a(r)] * (act[r] · Wdᵀ)   (float32, scattered to the
//                       assignment's own row)
//
// moe_gemm_tc is persistent: a CTA walks tiles of 128 list rows x BN weight rows (up to 256).
// Warp 0 loads both operands' tiles by TMA into a ring of stages, warp 1 issues the tcgen05.mma
// with the accumulator in tensor memory (two of them, so that the products of a tile run under
// the epilogue of the one before), warps 2-5 read it, apply the activation or the weight and
// write whole pieces of rows. A tile's rows beyond the expert's list and weight rows beyond the
// expert's own are computed and dropped.
#include "tc_common.cuh"
#include "moe_act.cuh"

MB_DEFINE_LAST_ERROR

typedef __nv_bfloat16 bf16;

#define MQ_ROWS 128
#define MQ_BK 64
#define MQ_STAGES 4
#define MQ_THREADS 192
#define MQ_A_BYTES (MQ_ROWS * MQ_BK * 2)
#define MQ_B_BYTES (256 * MQ_BK * 2)
#define MQ_SMEM (1024 + MQ_STAGES * (MQ_A_BYTES + MQ_B_BYTES) + 1024 + 4 * 4096)

__global__ void __launch_bounds__(256)
moe_gather_kernel(const bf16* __restrict__ in, const int* __restrict__ plan, int A, int E, int top,
                  int K, bf16* __restrict__ out) {
  mb_grid_wait();
  mb_grid_launch_next();
  const int* offsets = plan + 1;
  const int r = blockIdx.x;
  if (r >= offsets[E]) return;
  const uint4* src = (const uint4*)(in + (size_t)(offsets[E + 1 + r] / top) * K);
  uint4* dst = (uint4*)(out + (size_t)r * K);
  for (int i = threadIdx.x; i < K / 8; i += blockDim.x) dst[i] = src[i];
}

// out[r] = in[perm[r] / top] for every row r of the plan's lists; K a multiple of 8
MB_EXPORT int mb_moe_gather(const void* in, const int* plan, int A, int E, int top, int K,
                            void* out, void* stream) {
  if (A <= 0) return 0;
  if (K % 8 || (((uintptr_t)in | (uintptr_t)out) & 15))
    MB_FAIL("mb_moe_gather: rows of %d values on 16-byte boundaries", K);
  mb_launch(moe_gather_kernel, dim3(A), dim3(256), 0, (cudaStream_t)stream, (const bf16*)in, plan,
            A, E, top, K, (bf16*)out);
  MB_CHECK_LAUNCH("mb_moe_gather");
}

template <int MODE>
__global__ void __launch_bounds__(MQ_THREADS, 1)
moe_gemm_tc_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB,
                   void* __restrict__ out, const int* __restrict__ plan, int A, int E,
                   int max_tiles, int N, int K, int BN, int n_tiles, int act,
                   const float* __restrict__ weight, float limit, int* __restrict__ error) {
  constexpr int NB = MODE == MOE_GATED_UP ? 2 : 1;
  extern __shared__ uint8_t mq_raw[];
  const uint32_t raw = smem_u32(mq_raw);
  const uint32_t sA = (raw + 1023u) & ~1023u;       // swizzled tiles need 1024-byte alignment
  const uint32_t sB = sA + MQ_STAGES * MQ_A_BYTES;
  const uint32_t bars = sB + MQ_STAGES * MQ_B_BYTES;
  const uint32_t full0 = bars, empty0 = bars + 8 * MQ_STAGES;
  const uint32_t acc_full0 = bars + 16 * MQ_STAGES, acc_empty0 = acc_full0 + 16;
  const uint32_t slot = acc_empty0 + 16;
  volatile uint32_t* slot_ptr = (volatile uint32_t*)(mq_raw + (slot - raw));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int BNO = BN / NB;                          // output columns of a tile
  const int nkb = (K + MQ_BK - 1) / MQ_BK;

  if (threadIdx.x == 0) {
    for (int s = 0; s < MQ_STAGES; ++s) {
      mbar_init(full0 + 8 * s, 1);
      mbar_init(empty0 + 8 * s, 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(acc_full0 + 8 * b, 1);
      mbar_init(acc_empty0 + 8 * b, 4);  // the four epilogue warps
    }
    mbar_fence_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmB);
  }
  if (warp == 1) tmem_alloc(slot, 512);  // two accumulators of 256 columns
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *slot_ptr;
  mb_grid_wait();
  mb_grid_launch_next();
  const int* offsets = plan + 1;
  const int* perm = offsets + E + 1;
  const int work = min(plan[0], max_tiles) * n_tiles;   // tile w: row tile w / n_tiles

  if (warp == 0) {
    if (elect_one()) {
      int s = 0;
      uint32_t ph = 0;
      for (int w = blockIdx.x; w < work; w += gridDim.x) {
        const int tile = w / n_tiles, n0 = (w - tile * n_tiles) * BNO;
        const int e = perm[A + tile], r0 = perm[A + max_tiles + tile];
        for (int i = 0; i < nkb; ++i) {
          mbar_wait(empty0 + 8 * s, ph ^ 1, error, 1);
          mbar_expect_tx(full0 + 8 * s, MQ_A_BYTES + BN * MQ_BK * 2);
          tma_load_2d(sA + s * MQ_A_BYTES, &tmA, i * MQ_BK, r0, full0 + 8 * s);
#pragma unroll
          for (int nb = 0; nb < NB; ++nb)
            tma_load_2d(sB + s * MQ_B_BYTES + nb * BNO * (MQ_BK * 2), &tmB, i * MQ_BK,
                        (e * NB + nb) * N + n0, full0 + 8 * s);
          if (++s == MQ_STAGES) { s = 0; ph ^= 1; }
        }
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      const uint32_t idesc = umma_idesc_bf16(MQ_ROWS, BN);
      int s = 0, it = 0;
      uint32_t ph = 0;
      for (int w = blockIdx.x; w < work; w += gridDim.x, ++it) {
        const int b = it & 1;
        mbar_wait(acc_empty0 + 8 * b, ((it >> 1) & 1) ^ 1, error, 2);  // the epilogue left it
        tc_fence_after_sync();
        const uint32_t acc = tmem + b * 256;
        for (int i = 0; i < nkb; ++i) {
          mbar_wait(full0 + 8 * s, ph, error, 2);
          tc_fence_after_sync();
          const uint64_t da = umma_desc_k128(sA + s * MQ_A_BYTES);
          const uint64_t db = umma_desc_k128(sB + s * MQ_B_BYTES);
#pragma unroll
          for (int k = 0; k < MQ_BK / 16; ++k)  // 16 values of K = 32 bytes further in the row
            umma_bf16(acc, da + 2 * k, db + 2 * k, idesc, (i | k) != 0);
          umma_commit(empty0 + 8 * s);  // the stage is free once these MMAs have read it
          if (++s == MQ_STAGES) { s = 0; ph ^= 1; }
        }
        umma_commit(acc_full0 + 8 * b);
      }
    }
  } else {
    const int q = warp & 3;  // the TMEM lanes a warp may read: 32 * (warp % 4) ..
    // a warp lays 32 rows x 128 bytes of finished output here (16-byte piece p of row r at
    // p ^ (r & 7)) and writes four rows of 128 bytes at a time
    const uint32_t stage_w = bars + 1024 + q * 4096;
    const uint32_t mine = stage_w + lane * 128;
    const int pc = lane & 7;
    int it = 0;
    for (int w = blockIdx.x; w < work; w += gridDim.x, ++it) {
      const int tile = w / n_tiles, n0 = (w - tile * n_tiles) * BNO;
      const int e = perm[A + tile], r0 = perm[A + max_tiles + tile];
      const int rows = min(MQ_ROWS, offsets[e + 1] - r0);
      // where the warp's rows go: down, the assignment of row `lane`; up, the list row itself
      int to = 0;
      float wt = 1.0f;
      if (MODE == MOE_DOWN && q * 32 + lane < rows) {
        to = perm[r0 + q * 32 + lane];
        if (weight) wt = weight[to];
      }
      const int b = it & 1;
      mbar_wait(acc_full0 + 8 * b, (it >> 1) & 1, error, 3);
      tc_fence_after_sync();
      const uint32_t taddr = tmem + b * 256 + ((uint32_t)(q * 32) << 16);
      constexpr int STEP = MODE == MOE_DOWN ? 32 : 64;      // output columns of 128 bytes
      if (q * 32 < rows)
#pragma unroll 1
      for (int c0 = 0; c0 < BNO; c0 += STEP) {
        const int ncols = min(STEP, min(BNO - c0, N - (n0 + c0)));
        if (ncols <= 0) break;
#pragma unroll 1
        for (int g = 0; g * 16 < ncols; ++g) {
          float v[16];
          tmem_ld16(taddr + c0 + 16 * g, v);
          if (MODE == MOE_DOWN) {
#pragma unroll
            for (int j = 0; j < 4; ++j)
              st_shared_v4(mine + (((4 * g + j) ^ (lane & 7)) << 4),
                           make_uint4(__float_as_uint(wt * v[4 * j]), __float_as_uint(wt * v[4 * j + 1]),
                                      __float_as_uint(wt * v[4 * j + 2]),
                                      __float_as_uint(wt * v[4 * j + 3])));
          } else {
            float u[16];
            if (NB == 2) tmem_ld16(taddr + BNO + c0 + 16 * g, u);
            __nv_bfloat162 h[8];
#pragma unroll
            for (int j = 0; j < 8; ++j)
              h[j] = __floats2bfloat162_rn(
                  moe_act<MODE>(v[2 * j], NB == 2 ? u[2 * j] : 0.f, act, limit),
                  moe_act<MODE>(v[2 * j + 1], NB == 2 ? u[2 * j + 1] : 0.f, act, limit));
            st_shared_v4(mine + (((2 * g) ^ (lane & 7)) << 4), *(uint4*)&h[0]);
            st_shared_v4(mine + (((2 * g + 1) ^ (lane & 7)) << 4), *(uint4*)&h[4]);
          }
        }
        __syncwarp();
        const int pieces = MODE == MOE_DOWN ? ncols >> 2 : ncols >> 3;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int r = 4 * i + (lane >> 3);
          const int row = MODE == MOE_DOWN ? __shfl_sync(0xffffffffu, to, r) : r0 + q * 32 + r;
          if (pc < pieces && q * 32 + r < rows) {
            const uint4 x = ld_shared_v4(stage_w + r * 128 + ((pc ^ (r & 7)) << 4));
            if (MODE == MOE_DOWN) *(uint4*)((float*)out + (size_t)row * N + n0 + c0 + 4 * pc) = x;
            else *(uint4*)((bf16*)out + (size_t)row * N + n0 + c0 + 8 * pc) = x;
          }
        }
        __syncwarp();  // the rows are read out before the next columns are laid over them
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(acc_empty0 + 8 * b);
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, 512);
}

// One of the experts' products over a plan in tiles of 128 rows. `in` [A, K]: list rows (gathered
// for the first product); W [E][N or 2N][K]; up 0: the second product, 1: the first with gate
// and up rows, 2: the first without a gate. N and K multiples of 8. `error`: a device word
// that receives a non-zero code if a wait ran out.
MB_EXPORT int mb_moe_gemm_tc(const void* in, const void* W, void* out, const int* plan, int A,
                             int E, int max_tiles, int N, int K, int up, int act,
                             const float* weight, float limit, int sms, int* error, void* stream) {
  if (A <= 0) return 0;
  if (up < 0 || up > 2) MB_FAIL("mb_moe_gemm_tc: product %d", up);
  if (up == MOE_PLAIN_UP && act != 0 && act != 1 && act != 3)
    MB_FAIL("mb_moe_gemm_tc: activation %d of one input", act);
  if (N % 8 || K % 8 || ((uintptr_t)out & 15))
    MB_FAIL("mb_moe_gemm_tc: %d x %d (multiples of 8, 16-byte boundaries)", N, K);
  const int nb = up == MOE_GATED_UP ? 2 : 1;
  // the tile's width (of output columns, a multiple of 16): the one whose rounds of tiles over
  // the SMs, each with a tile's fixed price, take least (whole rounds while they are few). How
  // many row tiles there will be is estimated: every expert's last tile half full, or one tile
  // an expert while lists are short
  const int used = min(E, A), row_tiles = max(used, A / MQ_ROWS + used / 2);
  int best = 0;
  double cost = 0;
  for (int bn = 256 / nb; bn >= 64 / nb; bn -= 16) {
    const long long tiles = (long long)((N + bn - 1) / bn) * row_tiles;
    const double rounds = tiles <= 3ll * sms ? (double)((tiles + sms - 1) / sms) : (double)tiles / sms;
    const double c = rounds * (bn * nb + 24);
    if (!best || c < cost) { best = bn; cost = c; }
  }
  const int n_tiles = (N + best - 1) / best;
  CUtensorMap tmA, tmB;
  if (!mb_make_map_bf16(&tmA, in, A, K, K, MQ_ROWS, "mb_moe_gemm_tc rows")) return -1;
  if (!mb_make_map_bf16(&tmB, W, (long long)E * nb * N, K, K, best, "mb_moe_gemm_tc weights")) return -1;
  const int grid = (int)min((long long)sms, (long long)max_tiles * n_tiles);
#define GO(M_)                                                                                 \
  {                                                                                            \
    static bool configured = false;                                                            \
    if (!configured) {                                                                         \
      cudaError_t e = cudaFuncSetAttribute(moe_gemm_tc_kernel<M_>,                             \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize,        \
                                           MQ_SMEM);                                           \
      if (e != cudaSuccess) MB_FAIL("mb_moe_gemm_tc: %s", cudaGetErrorString(e));              \
      configured = true;                                                                       \
    }                                                                                          \
    mb_launch(moe_gemm_tc_kernel<M_>, dim3(grid), dim3(MQ_THREADS), MQ_SMEM,                   \
              (cudaStream_t)stream, tmA, tmB, out, plan, A, E, max_tiles, N, K, best * nb,     \
              n_tiles, act, weight, limit, error);                                             \
  }
  if (up == MOE_GATED_UP) GO(MOE_GATED_UP)
  else if (up == MOE_PLAIN_UP) GO(MOE_PLAIN_UP)
  else GO(MOE_DOWN)
#undef GO
  MB_CHECK_LAUNCH("mb_moe_gemm_tc");
}
