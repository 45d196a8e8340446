// Pieces that the attention kernels on mma.sync share: a page's tiles of keys and values in
// shared memory as operands, and the copies that bring them there.
#pragma once
#include "mma_common.cuh"
#include "tc_common.cuh"

// 16 bytes of a tile in shared memory
__device__ __forceinline__ uint4 lds16(uint32_t addr) {
  uint4 v;
  asm volatile("ld.shared.v4.u32 {%0, %1, %2, %3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "r"(addr));
  return v;
}

// `bytes` contiguous bytes from global to shared memory (both 16-byte aligned), completing `bar`
__device__ __forceinline__ void bulk_copy(uint32_t dst, const void* src, uint32_t bytes,
                                          uint32_t bar) {
  asm volatile(
      "cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
      ::"r"(dst), "l"(src), "r"(bytes), "r"(bar)
      : "memory");
}

__device__ __forceinline__ float ld_cluster_f32(uint32_t cluster_addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(cluster_addr) : "memory");
  return v;
}

// scores of one page whose keys lie in shared memory (rows KP bytes apart): sc[u][e] = q(row) ·
// k(key) for the keys u*8 + 2c + (e & 1) of the page and the rows r (e < 2) and r + 8 (e >= 2) of
// the warp's 16 query rows
template <int HD, int KP>
__device__ __forceinline__ void qk_page_smem(const uint4* qa, const uint4* qb, uint32_t ks, int r,
                                             int c, float sc[8][4]) {
#pragma unroll
  for (int u = 0; u < 8; ++u) {
    sc[u][0] = sc[u][1] = sc[u][2] = sc[u][3] = 0.f;
    const uint32_t krow = ks + (uint32_t)(u * 8 + r) * KP + c * 16;
#pragma unroll
    for (int ch = 0; ch < HD / 32; ++ch) {
      const uint4 kb = lds16(krow + ch * 64);
      mma_bf16(sc[u], qa[ch].x, qb[ch].x, qa[ch].y, qb[ch].y, kb.x, kb.y);
      mma_bf16(sc[u], qa[ch].z, qb[ch].z, qa[ch].w, qb[ch].w, kb.z, kb.w);
    }
  }
}

// o += p · v for one page whose values lie in shared memory (rows VP bytes apart): 16 keys a
// step; logical column q of output tile j is the dim db*64 + q*8 + j, so a thread ends up with 8
// consecutive dims per accumulator column
template <int HD, int VP>
__device__ __forceinline__ void pv_page_smem(const float sc[8][4], uint32_t vs, int r, int c,
                                             float o[HD / 64][8][4]) {
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    const uint32_t a0 = pack_bf16(sc[2 * kk][0], sc[2 * kk][1]);
    const uint32_t a1 = pack_bf16(sc[2 * kk][2], sc[2 * kk][3]);
    const uint32_t a2 = pack_bf16(sc[2 * kk + 1][0], sc[2 * kk + 1][1]);
    const uint32_t a3 = pack_bf16(sc[2 * kk + 1][2], sc[2 * kk + 1][3]);
    const uint32_t vrow = vs + (uint32_t)(kk * 16 + 2 * c) * VP + r * 16;
#pragma unroll
    for (int db = 0; db < HD / 64; ++db) {
      const uint4 va = lds16(vrow + db * 128);
      const uint4 vb = lds16(vrow + VP + db * 128);
      const uint4 vc = lds16(vrow + 8 * VP + db * 128);
      const uint4 vd = lds16(vrow + 9 * VP + db * 128);
      const uint32_t wa[4] = {va.x, va.y, va.z, va.w}, wb[4] = {vb.x, vb.y, vb.z, vb.w};
      const uint32_t wc[4] = {vc.x, vc.y, vc.z, vc.w}, wd[4] = {vd.x, vd.y, vd.z, vd.w};
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int w = j >> 1;
        const uint32_t b0 = (j & 1) ? pack_hi(wa[w], wb[w]) : pack_lo(wa[w], wb[w]);
        const uint32_t b1 = (j & 1) ? pack_hi(wc[w], wd[w]) : pack_lo(wc[w], wd[w]);
        mma_bf16(o[db][j], a0, a1, a2, a3, b0, b1);
      }
    }
  }
}

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
