// Helpers for kernels that exist for two activation types, bfloat16 and float, and the warp-level bf16 tensor-core
// pieces (ldmatrix, mma.sync m16n8k16, cp.async) of the attention and per-head kernels.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace zse {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_exact(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_exact(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }

__device__ __forceinline__ float relu2(float z) { return z > 0.f ? z * z : 0.f; }
// g sigmoid(1.702 g) (u + 1), g clamped from above, u from both sides
__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
  g = fminf(g, limit);
  return g / (1.f + expf(-1.702f * g)) * (fminf(fmaxf(u, -limit), limit) + 1.f);
}

__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }

// 2^x on the special-function unit: softmax weights need no more than its fp32 accuracy, and no range handling around it
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// 1 / x on the special-function unit, for normal x (infinity gives zero)
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// sigmoid on the special-function unit, within a few units in the last place of fp32
__device__ __forceinline__ float sigmoid_fast(float z) { return rcp(1.f + ex2(z * -1.4426950408889634f)); }

// Gated activations of two products: kinds 0 clamped_glu, 1 silu(g) u, 2 gelu(g) u with the tanh form of gelu, which is
// z sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3)).  FAST: the special-function unit's sigmoid, for results in bfloat16.
template <bool FAST>
__device__ __forceinline__ float glu(int kind, float g, float u, float limit) {
  if (kind == 0 && !FAST) return clamped_glu(g, u, limit);
  if (kind == 0) {
    g = fminf(g, limit);
    return g * sigmoid_fast(1.702f * g) * (fminf(fmaxf(u, -limit), limit) + 1.f);
  }
  const float z = kind == 1 ? g : 1.5957691216057308f * (g + 0.044715f * g * g * g);
  return g * (FAST ? sigmoid_fast(z) : sigmoid_exact(z)) * u;
}

__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
// the part of (a, b) that pack_bf16(a, b) lost
__device__ __forceinline__ uint32_t pack_bf16_rest(float a, float b) {
  return pack_bf16(a - __bfloat162float(__float2bfloat16_rn(a)), b - __bfloat162float(__float2bfloat16_rn(b)));
}

// VEC consecutive values as fp32 (VEC 4: one access of 16 or 8 bytes)
template <int VEC>
struct F32Vec {
  float v[VEC];
};
template <int VEC>
__device__ __forceinline__ F32Vec<VEC> load_vec(const float* p) {
  F32Vec<VEC> r;
  if constexpr (VEC == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
  } else {
    r.v[0] = p[0];
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ F32Vec<VEC> load_vec(const bf16* p) {
  F32Vec<VEC> r;
  if constexpr (VEC == 4) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
    r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
  } else {
    r.v[0] = to_f32(p[0]);
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* p, const F32Vec<VEC>& r) {
  if constexpr (VEC == 4)
    *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else
    p[0] = r.v[0];
}
template <int VEC>
__device__ __forceinline__ void store_vec(bf16* p, const F32Vec<VEC>& r) {
  if constexpr (VEC == 4)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r.v[0], r.v[1]), pack_bf16(r.v[2], r.v[3]));
  else
    p[0] = from_f32<bf16>(r.v[0]);
}

__device__ __forceinline__ void cpa16(void* smem_dst, const void* gmem_src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gmem_src) : "memory");
}
__device__ __forceinline__ void cpa_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cpa_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldm_x4(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldm_x4_t(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr float kLog2E = 1.4426950408889634f;

enum DType : int { kBF16 = 1, kF32 = 2 };

}  // namespace zse
