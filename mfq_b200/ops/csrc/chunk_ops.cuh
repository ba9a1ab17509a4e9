// Pieces of the chunked recurrences (64 tokens at a time, bf16 tensor cores by mma.sync): copies, fragments, and fp32 operands as pairs
// of bf16 numbers.
#pragma once

#include "dense_common.cuh"

namespace mfq {

constexpr int kGc = 64;           // tokens per chunk
constexpr float kGcSpan = 100.f;  // widest decay (log2) of a 16-row block whose scores are formed as a product of two factors

__device__ __forceinline__ float gc_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void gc_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void gc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void gc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void gc_ldm(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void gc_ldm_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void gc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as a pair of bf16 numbers and the pair of what they leave
__device__ __forceinline__ void gc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 gc_pair(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

// 64 rows of `width` bf16 (a multiple of 16) to shared memory by `kWarps` warps, two rows of a warp at a time; rows from `n` on are
// zeros.
template <int kWarps>
__device__ __forceinline__ void gc_rows(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, int stride, int width, int n, int warp, int lane) {
  const int per = width / 8;
  for (int t0 = warp * 2; t0 < kGc; t0 += 2 * kWarps)
    for (int i = lane; i < 2 * per; i += 32) {
      const int t = t0 + (i >= per), c = (i >= per ? i - per : i) * 8;
      if (t < n) gc_cp16(dst + t * pitch + c, src + size_t(t) * stride + c);
      else *reinterpret_cast<uint4*>(dst + t * pitch + c) = make_uint4(0, 0, 0, 0);
    }
}

// z_tc = sum_r a_tr w_cr of a chunk's 64 tokens and the `dk` channels of a head: a [64][pitch] in shared memory, w [dk, rank] in global
// memory, rank a multiple of 16.  store(t, c, z_tc, z_t(c+1)).
template <int kWarps, typename Store>
__device__ __forceinline__ void gc_low_rank(const __nv_bfloat16* a, int pitch, const __nv_bfloat16* w, int rank, int dk, int warp, int lane, Store&& store) {
  const int g = lane >> 2, t4 = lane & 3, mat = lane >> 3, mrow = lane & 7;
  const uint32_t frag = smem_u32(a + ((mat & 1) * 8 + mrow) * pitch + (mat >> 1) * 8);
  for (int n0 = warp * 8; n0 < dk; n0 += kWarps * 8) {
    const __nv_bfloat16* row = w + size_t(n0 + g) * rank + t4 * 2;
    float acc[4][4] = {};
#pragma unroll 4
    for (int ks = 0; ks < rank / 16; ++ks) {
      const uint32_t b0 = *reinterpret_cast<const uint32_t*>(row + ks * 16), b1 = *reinterpret_cast<const uint32_t*>(row + ks * 16 + 8);
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) {
        uint32_t f[4];
        gc_ldm(frag + (mt * 16 * pitch + ks * 16) * 2, f);
        gc_mma(acc[mt], f, b0, b1);
      }
    }
#pragma unroll
    for (int mt = 0; mt < 4; ++mt) {
      store(mt * 16 + g, n0 + t4 * 2, acc[mt][0], acc[mt][1]);
      store(mt * 16 + g + 8, n0 + t4 * 2, acc[mt][2], acc[mt][3]);
    }
  }
}

}  // namespace mfq
