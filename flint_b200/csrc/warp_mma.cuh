// What warp-level tensor-core kernels share: 16-byte loads of eight numbers, ldmatrix, and mma.sync m16n8k16 (bfloat16
// in, float32 out).
#pragma once
#include "common.cuh"

namespace flint_attn {
using namespace flint;

template <typename TC>
__device__ __forceinline__ void load8(const TC* p, float* f);
template <>
__device__ __forceinline__ void load8<float>(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
template <>
__device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float* f) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}

// Warp-level tensor-core helpers (mma.sync m16n8k16, bf16 in, float32 out), first for the decode
// kernel in attention_tc.cu.  A decoded token brings only nq/nkv (typically 4) query rows per
// key/value head, far below the 128 rows of a tcgen05 tile, and the float32-pipe kernels here
// are bound by instruction issue; the warp-level MMA with 16 rows (the group's heads, zero
// padded) cuts the instruction count per byte of cache about tenfold:
//   S = Q K^T    ldmatrix (K rows are already the "col" operand), 2 x hd/16 MMAs per 16 keys
//   softmax      on the accumulator fragment: 4 lanes share a row; float32 max, sum, exp
//   O += P V     P re-packed from the S fragment as the A operand, V through ldmatrix.trans
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                         uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

}  // namespace flint_attn
