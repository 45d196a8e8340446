// A feed-forward of routed experts on the device, without a round trip to the host: the
// router's choice, the lists of tokens per expert, the experts' two products over those lists
// and the weighted sum into the residual. float32 arithmetic on the CUDA cores for float32
// and bfloat16 storage.
//
//   moe_route    per token: the `top` largest router logits (the lower index on a tie), their
//                weights = softmax over the chosen logits only, and the shared expert's gate
//                sigmoid(logit) when the router's product carries that column
//   moe_plan     assignments (token, k) listed expert by expert, cut into tiles of rows (the
//                choices come from the router, or from a table by token id)
//   moe_gemm     for every tile the product with its expert's weight:
//                up:   act[r, :] = f(h[token(r)] · Wgᵀ) * (h[token(r)] · Wuᵀ)   (rows gathered)
//                down: y[a(r), :] = weight[a(r)] * (act[r] · Wdᵀ)              (float32, scattered
//                      to the assignment's own row, so the sum below has a fixed order)
//   moe_combine  x[t] += sum_k y[t·top + k] + gate[t] · shared[t]
//
// Experts may have no gate: act[r, :] = f(h[token(r)] · Wuᵀ). In bfloat16 the products of a step
// of more than 8 tokens are moe_tc.cu's.
//
// The order of an expert's rows in its list comes from atomic counters and may differ from run
// to run; no result depends on it (a row's sums are formed alone, in a fixed order).
#include "common.cuh"
#include "mma_common.cuh"
#include "moe_act.cuh"

MB_DEFINE_LAST_ERROR

// ------------------------------------------------------------------ route
// z [parts][T, ldz] float32, the split sums of the router's product (parts = 1: the product
// itself), added up as they are read: columns [0, E) the experts' logits, column shared_col
// (or -1) the shared expert's gate logit. One warp per token.
__device__ __forceinline__ float route_logit(const float* __restrict__ zr, int parts,
                                             size_t part_stride, int i) {
  return parts == 1 ? zr[i] : sum_parts(zr + i, parts, part_stride);
}

__device__ __forceinline__ void route_token(const float* __restrict__ zr, int parts,
                                            size_t part_stride, int E, int top, int shared_col,
                                            int* __restrict__ ids, float* __restrict__ w,
                                            float* __restrict__ sg, int lane) {
  float last_v = INFINITY;
  int last_i = -1;
  float first = 0.f, sum = 0.f, mine = 0.f;  // lane k keeps the k-th chosen logit
  // up to 256 experts: a lane adds its logits' split sums up once and keeps them
  const bool kept = E <= 256;
  float zl[8];
  if (kept) {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = lane + 32 * j;
      zl[j] = i < E ? route_logit(zr, parts, part_stride, i) : -INFINITY;
    }
  }
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int best_i = 0x7fffffff;
    if (kept) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int i = lane + 32 * j;
        const float v = zl[j];
        const bool open = i < E && (v < last_v || (v == last_v && i > last_i));
        if (open && (v > best || (v == best && i < best_i))) {
          best = v;
          best_i = i;
        }
      }
    } else {
      for (int i = lane; i < E; i += 32) {
        const float v = route_logit(zr, parts, part_stride, i);
        const bool open = v < last_v || (v == last_v && i > last_i);
        if (open && (v > best || (v == best && i < best_i))) {
          best = v;
          best_i = i;
        }
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
      if (ov > best || (ov == best && oi < best_i)) {
        best = ov;
        best_i = oi;
      }
    }
    if (best_i == 0x7fffffff) {  // nothing left that compares (NaNs): take the next index
      best_i = min(E - 1, last_i + 1);
      best = route_logit(zr, parts, part_stride, best_i);
    }
    if (k == 0) first = best;
    const float e = expf(best - first);
    sum += e;
    if (lane == k) mine = e;
    if (lane == 0) ids[k] = best_i;
    last_v = best;
    last_i = best_i;
  }
  if (lane < top) w[lane] = mine / sum;
  if (sg && lane == 0) *sg = 1.0f / (1.0f + expf(-route_logit(zr, parts, part_stride, shared_col)));
}

// The other scorings: s = softmax(z) over all E columns, or s = sigmoid(z) column by column
// (`sigmoid`); the choice goes by s + corr (the lower index on a tie), the weights are the chosen
// s times wscale, not renormalized. Up to 256 columns (a lane keeps eight).
// `groups` > 1: the columns are that many equal groups of neighbours; a group's score is the sum
// of its two largest choice scores, and only columns of the `keep` best groups (the lower group on
// a tie) can be chosen. At most 32 groups (lane g keeps group g's score).
__device__ __forceinline__ void route_token_scored(const float* __restrict__ zr, int parts,
                                                   size_t part_stride, int E, int top,
                                                   const float* __restrict__ corr, float wscale,
                                                   int* __restrict__ ids, float* __restrict__ w,
                                                   int lane, bool sigmoid, int groups, int keep) {
  float sc[8], ch[8];
  float mx = -INFINITY;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int i = lane + 32 * j;
    sc[j] = i < E ? route_logit(zr, parts, part_stride, i) : -INFINITY;
    mx = fmaxf(mx, sc[j]);
  }
  if (sigmoid) {
#pragma unroll
    for (int j = 0; j < 8; ++j) sc[j] = lane + 32 * j < E ? sigmoid_f32(sc[j]) : 0.f;
  } else {
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      sc[j] = lane + 32 * j < E ? expf(sc[j] - mx) : 0.f;
      sum += sc[j];
    }
    sum = warp_sum(sum);
#pragma unroll
    for (int j = 0; j < 8; ++j) sc[j] = sc[j] / sum;
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int i = lane + 32 * j;
    ch[j] = i < E ? sc[j] + (corr ? corr[i] : 0.f) : -INFINITY;
  }
  if (groups > 1) {
    const int size = E / groups;
    float mine = -INFINITY;
    for (int g = 0; g < groups; ++g) {
      float a = -INFINITY, b = -INFINITY;    // this lane's two largest of the group
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int i = lane + 32 * j;
        if (i >= g * size && i < (g + 1) * size) {
          b = fmaxf(b, fminf(a, ch[j]));
          a = fmaxf(a, ch[j]);
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float oa = __shfl_xor_sync(0xffffffffu, a, o);
        const float ob = __shfl_xor_sync(0xffffffffu, b, o);
        b = fmaxf(fmaxf(b, ob), fminf(a, oa));
        a = fmaxf(a, oa);
      }
      if (lane == g) mine = size > 1 ? a + b : a;
    }
    // a group is open when fewer than `keep` groups are ahead of it
    int ahead = 0;
    for (int g = 0; g < groups; ++g) {
      const float v = __shfl_sync(0xffffffffu, mine, g);
      ahead += v > mine || (v == mine && g < lane);
    }
    const unsigned open = __ballot_sync(0xffffffffu, lane < groups && ahead < keep);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = lane + 32 * j;
      if (i < E && !((open >> (i / size)) & 1u)) ch[j] = -INFINITY;
    }
  }
  float last_v = INFINITY, mine = 0.f;
  int last_i = -1;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY, best_s = 0.f;
    int best_i = 0x7fffffff;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = lane + 32 * j;
      const float v = ch[j];
      const bool open = i < E && (v < last_v || (v == last_v && i > last_i));
      if (open && v > -INFINITY && (v > best || (v == best && i < best_i))) {
        best = v;
        best_i = i;
        best_s = sc[j];
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const float os = __shfl_xor_sync(0xffffffffu, best_s, o);
      const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
      if (ov > best || (ov == best && oi < best_i)) {
        best = ov;
        best_i = oi;
        best_s = os;
      }
    }
    if (best_i == 0x7fffffff) {  // nothing left that compares (NaNs): take the next index
      best_i = min(E - 1, last_i + 1);
      best_s = 0.f;
    }
    if (lane == k) mine = best_s * wscale;
    if (lane == 0) ids[k] = best_i;
    last_v = best;
    last_i = best_i;
  }
  if (lane < top) w[lane] = mine;
}

__global__ void __launch_bounds__(128)
moe_route_kernel(const float* __restrict__ z, int ldz, int parts, size_t part_stride, int E,
                 int top, int shared_col, int* __restrict__ ids, float* __restrict__ w,
                 float* __restrict__ sg, int T, int mode, const float* __restrict__ corr,
                 float wscale, int groups, int keep) {
  mb_grid_wait();
  mb_grid_launch_next();
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (t >= T) return;
  if (mode != 0) {
    route_token_scored(z + (size_t)t * ldz, parts, part_stride, E, top, corr, wscale,
                       ids + (size_t)t * top, w + (size_t)t * top, lane, mode == 2, groups, keep);
    return;
  }
  route_token(z + (size_t)t * ldz, parts, part_stride, E, top, shared_col, ids + (size_t)t * top,
              w + (size_t)t * top, sg ? sg + t : nullptr, lane);
}

// mode 0: softmax over the chosen logits; 1: scores by a softmax over all; 2: by a sigmoid each
static int route_groups(const char* who, int mode, int E, int top, int groups, int keep) {
  if (mode < 0 || mode > 2) MB_FAIL("%s: scoring %d", who, mode);
  if (groups <= 1) return 0;
  if (mode == 0 || groups > 32 || E % groups || keep < 1 || keep > groups ||
      top > keep * (E / groups))
    MB_FAIL("%s: %d of %d columns from %d of %d groups", who, top, E, keep, groups);
  return 0;
}

MB_EXPORT int mb_moe_route(const float* z, int ldz, int parts, long long part_stride, int E,
                           int top, int shared_col, int* ids, float* w, float* sg, int T,
                           int mode, const float* corr, float wscale, int groups, int keep,
                           void* stream) {
  if (T <= 0) return 0;
  if (route_groups("mb_moe_route", mode, E, top, groups, keep)) return -1;
  if (mode != 0 && (E > 256 || sg != nullptr))
    MB_FAIL("mb_moe_route: scores over all of %d columns (at most 256, no gate column)", E);
  if (top <= 0 || top > 32 || top > E) MB_FAIL("mb_moe_route: %d of %d experts", top, E);
  if ((sg != nullptr) != (shared_col >= 0)) MB_FAIL("mb_moe_route: the shared gate and its column");
  if (parts < 1) MB_FAIL("mb_moe_route: %d parts", parts);
  mb_launch(moe_route_kernel, dim3((T + 3) / 4), dim3(128), 0, (cudaStream_t)stream, z, ldz,
            parts, (size_t)part_stride, E, top, shared_col, ids, w, sg, T, mode, corr, wscale, groups, keep);
  MB_CHECK_LAUNCH("mb_moe_route");
}

// ------------------------------------------------------------------ plan
// plan (int32): [0] number of tiles, [1 .. 1+E] first list row of every expert (E + 1 values),
// then perm[A] (the assignment a = t·top + k at every list row), then tile_expert[max_tiles]
// and tile_row0[max_tiles]. One block.
// With `table` given the choices come from it: token t's k-th expert is
// table[tok_ids[t] * top + k] (A = T * top; an id outside the table counts as 0).
// With z given (a step of at most 64 tokens) the block first routes the tokens itself, a warp a
// token, and writes ids, w and sg as moe_route does: one kernel instead of two.
__global__ void __launch_bounds__(1024)
moe_plan_kernel(int* __restrict__ ids, int A, int E, int bm, int max_tiles,
                int* __restrict__ plan, const float* __restrict__ z, int ldz, int parts,
                size_t part_stride, int top, int shared_col, float* __restrict__ w,
                float* __restrict__ sg, int mode, const float* __restrict__ corr, float wscale,
                int groups, int keep, int E_route, const int* __restrict__ table, const int* __restrict__ tok_ids,
                int V) {
  mb_grid_wait();
  mb_grid_launch_next();
  extern __shared__ int counts[];  // E counters, then E cursors
  if (z != nullptr) {
    const int T = A / top, lane = threadIdx.x & 31;
    for (int t = threadIdx.x >> 5; t < T; t += blockDim.x >> 5) {
      if (mode != 0)
        route_token_scored(z + (size_t)t * ldz, parts, part_stride, E_route, top, corr, wscale,
                           ids + (size_t)t * top, w + (size_t)t * top, lane, mode == 2, groups,
                           keep);
      else
        route_token(z + (size_t)t * ldz, parts, part_stride, E_route, top, shared_col,
                    ids + (size_t)t * top, w + (size_t)t * top, sg ? sg + t : nullptr, lane);
    }
    __syncthreads();  // the block's own writes of ids are visible to it
  }
  auto choice = [&](int a) {
    if (table == nullptr) return ids[a];
    const int t = a / top, id = tok_ids[t];
    return table[(size_t)(id < 0 || id >= V ? 0 : id) * top + (a - t * top)];
  };
  int* cursor = counts + E;
  int* offsets = plan + 1;
  int* perm = offsets + E + 1;
  int* tile_e = perm + A;
  int* tile_r0 = tile_e + max_tiles;
  for (int e = threadIdx.x; e < E; e += blockDim.x) counts[e] = 0;
  __syncthreads();
  for (int a = threadIdx.x; a < A; a += blockDim.x) {
    const int e = choice(a);
    if (e >= 0 && e < E) atomicAdd(&counts[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int at = 0, tiles = 0;
    for (int e = 0; e < E; ++e) {
      offsets[e] = at;
      cursor[e] = at;
      for (int r0 = 0; r0 < counts[e] && tiles < max_tiles; r0 += bm) {
        tile_e[tiles] = e;
        tile_r0[tiles] = at + r0;
        ++tiles;
      }
      at += counts[e];
    }
    offsets[E] = at;
    plan[0] = tiles;
  }
  __syncthreads();
  for (int a = threadIdx.x; a < A; a += blockDim.x) {
    const int e = choice(a);
    if (e >= 0 && e < E) perm[atomicAdd(&cursor[e], 1)] = a;
  }
}

MB_EXPORT int mb_moe_plan(int* ids, int A, int E, int bm, int max_tiles, int* plan,
                          void* stream) {
  if (A <= 0) return 0;
  if (E > 4096) MB_FAIL("mb_moe_plan: %d experts", E);
  if (max_tiles < (A + bm - 1) / bm + E) MB_FAIL("mb_moe_plan: room for %d tiles", max_tiles);
  mb_launch(moe_plan_kernel, dim3(1), dim3(1024), (size_t)2 * E * sizeof(int),
            (cudaStream_t)stream, ids, A, E, bm, max_tiles, plan, (const float*)nullptr, 0, 1,
            (size_t)0, 1, -1, (float*)nullptr, (float*)nullptr, 0, (const float*)nullptr, 1.0f, 1, 1, E,
            (const int*)nullptr, (const int*)nullptr, 0);
  MB_CHECK_LAUNCH("mb_moe_plan");
}

// The same for choices that a table [V, top] names by token id.
MB_EXPORT int mb_moe_table_plan(const int* table, int V, int top, const int* tok_ids, int A, int E,
                                int bm, int max_tiles, int* plan, void* stream) {
  if (A <= 0) return 0;
  if (E > 4096 || top <= 0 || top > E || A % top || V <= 0)
    MB_FAIL("mb_moe_table_plan: %d choices of %d experts, %d ids", top, E, V);
  if (max_tiles < (A + bm - 1) / bm + E) MB_FAIL("mb_moe_table_plan: room for %d tiles", max_tiles);
  mb_launch(moe_plan_kernel, dim3(1), dim3(1024), (size_t)2 * E * sizeof(int),
            (cudaStream_t)stream, (int*)nullptr, A, E, bm, max_tiles, plan, (const float*)nullptr, 0,
            1, (size_t)0, top, -1, (float*)nullptr, (float*)nullptr, 0, (const float*)nullptr, 1.0f,
            1, 1, E, table, tok_ids, V);
  MB_CHECK_LAUNCH("mb_moe_table_plan");
}

// moe_route and moe_plan in one kernel, for a step of at most 64 tokens.
MB_EXPORT int mb_moe_route_plan(const float* z, int ldz, int parts, long long part_stride, int E,
                                int top, int shared_col, int* ids, float* w, float* sg, int T,
                                int bm, int max_tiles, int* plan, int mode, const float* corr,
                                float wscale, int groups, int keep, int E_route, void* stream) {
  if (T <= 0) return 0;
  if (E_route < E) MB_FAIL("mb_moe_route_plan: %d routed columns for %d experts", E_route, E);
  if (route_groups("mb_moe_route_plan", mode, E_route, top, groups, keep)) return -1;
  if (mode != 0 && (E_route > 256 || sg != nullptr))
    MB_FAIL("mb_moe_route_plan: scores over all of %d columns (at most 256, no gate column)", E_route);
  if (T > 64) MB_FAIL("mb_moe_route_plan: %d tokens (at most 64)", T);
  if (top <= 0 || top > 32 || top > E_route) MB_FAIL("mb_moe_route_plan: %d of %d experts", top, E_route);
  if ((sg != nullptr) != (shared_col >= 0)) MB_FAIL("mb_moe_route_plan: the shared gate and its column");
  if (E > 4096 || parts < 1) MB_FAIL("mb_moe_route_plan: %d experts, %d parts", E, parts);
  const int A = T * top;
  if (max_tiles < (A + bm - 1) / bm + E) MB_FAIL("mb_moe_route_plan: room for %d tiles", max_tiles);
  mb_launch(moe_plan_kernel, dim3(1), dim3(1024), (size_t)2 * E * sizeof(int),
            (cudaStream_t)stream, ids, A, E, bm, max_tiles, plan, z, ldz, parts,
            (size_t)part_stride, top, shared_col, w, sg, mode, corr, wscale, groups, keep, E_route,
            (const int*)nullptr, (const int*)nullptr, 0);
  MB_CHECK_LAUNCH("mb_moe_route_plan");
}

// ------------------------------------------------------------------ the experts' products
#define MG_BN 64
#define MG_BK 16
// UP:   in = h [T, K] (row of list row r: perm[r] / top), W [E][2N][K] (gate rows, then up
//       rows; without a gate [E][N][K]), out = act [A, N] at list row r.
// DOWN: in = act [A, K] at list row r, W [E][N][K], out = y [A, N] float32 at row perm[r],
//       multiplied by weight[perm[r]] (null: by one).
template <typename T, typename TW, int BM, int MODE>
__global__ void __launch_bounds__(256)
moe_gemm_kernel(const T* __restrict__ in, const TW* __restrict__ W, void* __restrict__ out,
                const int* __restrict__ plan, int A, int E, int max_tiles, int top, int N, int K,
                int act, const float* __restrict__ weight, float limit) {
  mb_grid_wait();
  mb_grid_launch_next();
  constexpr bool UP = MODE != MOE_DOWN;
  constexpr int NW = MODE == MOE_GATED_UP ? 2 : 1;
  constexpr int TM = BM / 16;
  const int tile = blockIdx.y;
  if (tile >= plan[0]) return;
  const int* offsets = plan + 1;
  const int* perm = offsets + E + 1;
  const int e = perm[A + tile];
  const int r0 = perm[A + max_tiles + tile];
  const int rows = min(BM, offsets[e + 1] - r0);
  __shared__ float As[MG_BK][BM + 4];
  __shared__ float Ws[NW][MG_BK][MG_BN + 4];
  __shared__ int src[BM];
  const int tid = threadIdx.x;
  if (tid < BM) src[tid] = tid < rows ? perm[r0 + tid] : -1;
  __syncthreads();
  const int n0 = blockIdx.x * MG_BN;
  const TW* We = W + (size_t)e * NW * N * K;
  const int tr = (tid / 16) * TM, tc = (tid % 16) * 4;
  float acc[NW][TM][4];
#pragma unroll
  for (int w = 0; w < NW; ++w)
#pragma unroll
    for (int i = 0; i < TM; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[w][i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += MG_BK) {
    for (int el = tid; el < BM * MG_BK; el += 256) {
      const int r = el / MG_BK, c = el % MG_BK;
      const int gk = k0 + c;
      float v = 0.f;
      if (r < rows && gk < K) {
        const size_t row = UP ? (size_t)(src[r] / top) : (size_t)(r0 + r);
        v = to_f32<T>(in[row * K + gk]);
      }
      As[c][r] = v;
    }
    for (int el = tid; el < MG_BN * MG_BK; el += 256) {
      const int r = el / MG_BK, c = el % MG_BK;
      const int gn = n0 + r, gk = k0 + c;
#pragma unroll
      for (int w = 0; w < NW; ++w)
        Ws[w][c][r] = (gn < N && gk < K) ? to_f32<TW>(We[((size_t)w * N + gn) * K + gk]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < MG_BK; ++k) {
      float a[TM];
#pragma unroll
      for (int i = 0; i < TM; ++i) a[i] = As[k][tr + i];
#pragma unroll
      for (int w = 0; w < NW; ++w) {
        float b[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) b[j] = Ws[w][k][tc + j];
#pragma unroll
        for (int i = 0; i < TM; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[w][i][j] = fmaf(a[i], b[j], acc[w][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < TM; ++i) {
    const int r = tr + i;
    if (r >= rows) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int gn = n0 + tc + j;
      if (gn >= N) continue;
      if (UP) {
        ((T*)out)[(size_t)(r0 + r) * N + gn] =
            from_f32<T>(moe_act<MODE>(acc[0][i][j], acc[NW - 1][i][j], act, limit));
      } else {
        const int a = src[r];
        ((float*)out)[(size_t)a * N + gn] = (weight ? weight[a] : 1.0f) * acc[0][i][j];
      }
    }
  }
}

// The two products for a decode step of at most eight tokens (tiles of at most 8 rows, so an
// expert's weights are streamed exactly once): the WEIGHT rows are the 16 rows of the m16n8k16
// product and the tile's tokens its 8 columns. A warp owns 16 output features (for the first
// product their gate and their up rows) over all of K and reads its weight rows straight from
// global memory into the product's registers, 16 bytes a thread and row, several steps of K in
// flight; the tokens' rows wait in shared memory. Within a step of 32 values of K a thread
// holds values 8t .. 8t+7 of both operands: the products pair them up in another order than
// the instruction's own, which is the same sum. K must be a multiple of 32.
// GROUPS: how many groups of 16 features a warp of a product without a gate takes (two where there
// are blocks enough: the tokens' rows and the look-ups ahead of the first weight then serve twice
// as many weights).
#define MR_WARPS 4
template <int MODE, int GROUPS>
__global__ void __launch_bounds__(MR_WARPS * 32)
moe_rows_mma_kernel(const __nv_bfloat16* __restrict__ in, const __nv_bfloat16* __restrict__ W,
                    void* __restrict__ out, const int* __restrict__ plan, int A, int E,
                    int max_tiles, int top, int N, int K, int act,
                    const float* __restrict__ weight, float limit) {
  mb_grid_wait();
  mb_grid_launch_next();
  constexpr bool UP = MODE != MOE_DOWN;
  constexpr int NB = MODE == MOE_GATED_UP ? 2 : GROUPS;
  const int tile = blockIdx.y;
  if (tile >= plan[0]) return;
  const int* offsets = plan + 1;
  const int* perm = offsets + E + 1;
  const int e = perm[A + tile];
  const int r0 = perm[A + max_tiles + tile];
  const int rows = min(8, offsets[e + 1] - r0);
  extern __shared__ __align__(16) unsigned char mr_raw[];
  const int pitch = K + 8;
  __nv_bfloat16* xs = (__nv_bfloat16*)mr_raw;  // [8][pitch]
  __shared__ int src[8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  if (tid < 8) src[tid] = tid < rows ? perm[r0 + tid] : -1;
  __syncthreads();
  const int n0 = (blockIdx.x * MR_WARPS + warp) * (MODE == MOE_GATED_UP ? 16 : 16 * GROUPS);
  const __nv_bfloat16* We = W + (size_t)e * (MODE == MOE_GATED_UP ? 2 : 1) * N * K;
  // rows past N are read from row N - 1 and never stored
  const __nv_bfloat16* wa[NB];
  const __nv_bfloat16* wb[NB];
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) {
    const int row = n0 + (MODE == MOE_GATED_UP ? 0 : 16 * nb) + g;
    const size_t up = MODE == MOE_GATED_UP ? (size_t)nb * N : 0;
    wa[nb] = We + (up + min(row, N - 1)) * K + 8 * t;
    wb[nb] = We + (up + min(row + 8, N - 1)) * K + 8 * t;
  }
  for (int c = tid; c < 8 * (K / 8); c += MR_WARPS * 32) {
    const int r = c / (K / 8), kc = (c - r * (K / 8)) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < rows) v = ldg16(in + (UP ? (size_t)(src[r] / top) : (size_t)(r0 + r)) * K + kc);
    *(uint4*)(xs + r * pitch + kc) = v;
  }
  __syncthreads();
  if (n0 >= N) return;
  const __nv_bfloat16* xr = xs + g * pitch + 8 * t;
  float acc[NB][4];
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) acc[nb][0] = acc[nb][1] = acc[nb][2] = acc[nb][3] = 0.f;
  constexpr int UNROLL = NB == 2 ? 4 : 8;
  for (int k0 = 0; k0 < K; k0 += 32 * UNROLL) {
    uint4 a[UNROLL][NB], b[UNROLL][NB];
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
      const int k = k0 + 32 * u;
      if (k < K) {
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
          a[u][nb] = ldg16(wa[nb] + k);
          b[u][nb] = ldg16(wb[nb] + k);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
      const int k = k0 + 32 * u;
      if (k < K) {
        const uint4 x = *(const uint4*)(xr + k);
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
          mma_bf16(acc[nb], a[u][nb].x, b[u][nb].x, a[u][nb].y, b[u][nb].y, x.x, x.y);
          mma_bf16(acc[nb], a[u][nb].z, b[u][nb].z, a[u][nb].w, b[u][nb].w, x.z, x.w);
        }
      }
    }
  }
  // acc[.][0..1]: feature n0 + g, tokens 2t and 2t + 1; acc[.][2..3]: feature n0 + g + 8
#pragma unroll
  for (int nb = 0; nb < (MODE == MOE_GATED_UP ? 1 : NB); ++nb)
#pragma unroll
    for (int el = 0; el < 4; ++el) {
      const int gn = n0 + 16 * nb + g + (el >= 2 ? 8 : 0), r = 2 * t + (el & 1);
      if (gn >= N || r >= rows) continue;
      if (UP) {
        ((__nv_bfloat16*)out)[(size_t)(r0 + r) * N + gn] = __float2bfloat16_rn(
            moe_act<MODE>(acc[nb][el], acc[MODE == MOE_GATED_UP ? NB - 1 : nb][el], act, limit));
      } else {
        const int a_ = src[r];
        ((float*)out)[(size_t)a_ * N + gn] = (weight ? weight[a_] : 1.0f) * acc[nb][el];
      }
    }
}

MB_EXPORT int mb_moe_gemm(const void* in, int dtype, const void* W, int w_dtype, void* out,
                          const int* plan, int A, int E, int max_tiles, int bm, int top, int N,
                          int K, int up, int act, const float* weight, float limit, void* stream) {
  if (A <= 0) return 0;
  if (bm != 8 && bm != 16 && bm != 64) MB_FAIL("mb_moe_gemm: tiles of %d rows", bm);
  if (up < 0 || up > 2) MB_FAIL("mb_moe_gemm: product %d", up);
  if (up == MOE_PLAIN_UP && act != 0 && act != 1 && act != 3)
    MB_FAIL("mb_moe_gemm: activation %d of one input", act);
  cudaStream_t s = (cudaStream_t)stream;
  dim3 grid((N + MG_BN - 1) / MG_BN, max_tiles);
  if (bm == 8) {
    if (!(dtype == MB_BF16 && w_dtype == MB_BF16 && K % 32 == 0 &&
          (((uintptr_t)in | (uintptr_t)W) & 15) == 0))
      MB_FAIL("mb_moe_gemm: tiles of 8 rows are the decode kernel's (bfloat16, K %% 32 == 0)");
    const size_t smem = (size_t)8 * (K + 8) * 2;
    if (smem > 160 * 1024) MB_FAIL("mb_moe_gemm: rows of %d values", K);
    // two groups a warp while that still leaves two blocks an SM (as many experts as the step's
    // assignments can name)
    const int named = A < E ? A : E;
    const bool two = up != MOE_GATED_UP &&
                     (N + 32 * MR_WARPS - 1) / (32 * MR_WARPS) * named >= 2 * 148;
    const int per_block = (two ? 32 : 16) * MR_WARPS;
    dim3 g8((N + per_block - 1) / per_block, max_tiles);
#define GO8(M_, G_)                                                                           \
  {                                                                                           \
    static bool configured = false;                                                           \
    if (!configured) {                                                                        \
      cudaFuncSetAttribute(moe_rows_mma_kernel<M_, G_>,                                       \
                           cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);          \
      configured = true;                                                                      \
    }                                                                                         \
    mb_launch(moe_rows_mma_kernel<M_, G_>, g8, dim3(MR_WARPS * 32), smem, s,                 \
              (const __nv_bfloat16*)in, (const __nv_bfloat16*)W, out, plan, A, E, max_tiles,  \
              top, N, K, act, weight, limit);                                                 \
  }
    if (up == MOE_GATED_UP) GO8(MOE_GATED_UP, 1)
    else if (up == MOE_PLAIN_UP) { if (two) GO8(MOE_PLAIN_UP, 2) else GO8(MOE_PLAIN_UP, 1) }
    else { if (two) GO8(MOE_DOWN, 2) else GO8(MOE_DOWN, 1) }
#undef GO8
    MB_CHECK_LAUNCH("mb_moe_gemm");
  }
#define GO(T_, TW_, BM_, M_)                                                                 \
  mb_launch(moe_gemm_kernel<T_, TW_, BM_, M_>,  grid, dim3(256), 0, s, (const T_*)in,        \
            (const TW_*)W, out, plan, A, E, max_tiles, top, N, K, act, weight, limit)
#define GO2(T_, TW_, BM_)                                             \
  {                                                                   \
    if (up == MOE_GATED_UP) GO(T_, TW_, BM_, MOE_GATED_UP);           \
    else if (up == MOE_PLAIN_UP) GO(T_, TW_, BM_, MOE_PLAIN_UP);      \
    else GO(T_, TW_, BM_, MOE_DOWN);                                  \
  }
#define GO3(T_, TW_)                                                  \
  {                                                                   \
    if (bm == 16) GO2(T_, TW_, 16) else GO2(T_, TW_, 64)              \
  }
  if (dtype == MB_F32) {
    if (w_dtype == MB_F32) GO3(float, float) else GO3(float, __nv_bfloat16)
  } else {
    if (w_dtype == MB_F32) GO3(__nv_bfloat16, float) else GO3(__nv_bfloat16, __nv_bfloat16)
  }
#undef GO3
#undef GO2
#undef GO
  MB_CHECK_LAUNCH("mb_moe_gemm");
}

// ------------------------------------------------------------------ combine
// x[t, c] += sum_k y[(t·top + k), c] (k ascending) + sg[t] · shared[t, c]; shared
// [parts][T, H]: the split sums of the shared expert's last product, added up in split order.
// An assignment whose expert id is E or more names an identity expert: its term is
// w[a] · h[t, c] (h: the feed-forward's input, `h_bf16` says of which type). `store`: x = the
// sum instead of x += it.
__global__ void moe_combine_kernel(float* __restrict__ x, const float* __restrict__ y, int top,
                                   const float* __restrict__ shared, int parts,
                                   size_t part_stride, const float* __restrict__ sg, int H,
                                   const int* __restrict__ ids, const float* __restrict__ w,
                                   int E, const void* __restrict__ h, int h_bf16, int store) {
  mb_grid_wait();
  mb_grid_launch_next();
  const int t = blockIdx.x;
  const float g = sg ? sg[t] : 1.0f;
  for (int c = threadIdx.x; c < H; c += blockDim.x) {
    float v = 0.f;
    for (int k = 0; k < top; ++k) {
      const size_t a = (size_t)t * top + k;
      if (ids != nullptr && ids[a] >= E) {
        const float hv = h_bf16 ? __bfloat162float(((const __nv_bfloat16*)h)[(size_t)t * H + c])
                                : ((const float*)h)[(size_t)t * H + c];
        v = fmaf(w[a], hv, v);
      } else {
        v += y[a * H + c];
      }
    }
    if (shared) {
      v = fmaf(g, sum_parts(shared + (size_t)t * H + c, parts, part_stride), v);
    }
    if (store) x[(size_t)t * H + c] = v;
    else x[(size_t)t * H + c] += v;
  }
}

MB_EXPORT int mb_moe_combine(float* x, const float* y, int top, const float* shared, int parts,
                             long long part_stride, const float* sg, int T, int H,
                             const int* ids, const float* w, int E, const void* h, int h_dtype,
                             int store, void* stream) {
  if (T <= 0) return 0;
  if (ids != nullptr && (w == nullptr || h == nullptr))
    MB_FAIL("mb_moe_combine: identity experts need the weights and the input rows");
  mb_launch(moe_combine_kernel, dim3(T), dim3(H >= 1024 ? 256 : 128), 0, (cudaStream_t)stream, x,
            y, top, shared, parts, (size_t)part_stride, sg, H, ids, w, E, h,
            h_dtype == MB_BF16 ? 1 : 0, store);
  MB_CHECK_LAUNCH("mb_moe_combine");
}
