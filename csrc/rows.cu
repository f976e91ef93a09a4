// Row kernels for activations of bfloat16 or float: embedding, residual sum + RMSNorm, logits epilogue, arg-max of
// fp32 logits.  Any row length.
#include "api.h"
#include "typed.cuh"

namespace zse {
namespace {

template <typename T>
__global__ void embedding_typed_kernel(const T* __restrict__ table, const int* __restrict__ ids,
                                       float* __restrict__ out, int H, int vocab, float scale, Status* st) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  int id = ids[row];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) report(st, kBadArgument, 61, unsigned(id));
    id = 0;
  }
  const T* src = table + size_t(id) * H;
  float* dst = out + size_t(row) * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = to_f32(src[i]) * scale;
}

// residual += sum of fp32 planes [n_planes][M][H] + sum of the row's slots [M][n_slots][H];
// out = RMSNorm(residual) * weight.  A row is split over the CTAs of a cluster (gridDim.x), each thread keeps its
// columns in registers between the sum and the norm; VEC consecutive columns per access (4 when H % 4 == 0).
constexpr int kRowThreads = 256;
constexpr int kRowRegs = 8;          // accesses per thread: H <= 8 * VEC * 256 * cluster

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

template <typename T, typename S, int VEC>
__global__ void __launch_bounds__(kRowThreads)
add_norm_kernel(float* __restrict__ residual, const float* __restrict__ planes, int n_planes,
                const S* __restrict__ slots, int n_slots, const T* __restrict__ weight, T* __restrict__ out, int M,
                int H, float eps) {
  __shared__ float red[32];
  __shared__ float cluster_ss;
  pdl_launch_dependents();
  const int row = blockIdx.y, cs = gridDim.x;
  const int nv = (H / VEC + cs - 1) / cs;                  // accesses of this CTA
  const int v0 = blockIdx.x * nv, v1 = min(H / VEC, v0 + nv);
  const size_t base = size_t(row) * H, plane = size_t(M) * H;
  pdl_wait();
  F32Vec<VEC> x[kRowRegs];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i < v1) {
      const size_t at = base + size_t(i) * VEC;
      x[j] = load_vec<VEC>(residual + at);
#pragma unroll 4
      for (int p = 0; p < n_planes; ++p) {
        const F32Vec<VEC> y = load_vec<VEC>(planes + p * plane + at);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[j].v[e] += y.v[e];
      }
#pragma unroll 4
      for (int k = 0; k < n_slots; ++k) {
        const F32Vec<VEC> y = load_vec<VEC>(slots + (size_t(row) * n_slots + k) * H + size_t(i) * VEC);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[j].v[e] += y.v[e];
      }
      if (n_planes + n_slots > 0) store_vec<VEC>(residual + at, x[j]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x[j].v[e] * x[j].v[e];
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = warp_sum((threadIdx.x & 31) < (kRowThreads >> 5) ? red[threadIdx.x & 31] : 0.f);
  if (cs > 1) {
    if (threadIdx.x == 0) cluster_ss = total;
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    total = 0.f;
    const uint32_t local = smem_u32(&cluster_ss);
    for (int r = 0; r < cs; ++r) {                         // same order in every CTA: identical sums
      uint32_t remote;
      float t;
      asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(r));
      asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(t) : "r"(remote) : "memory");
      total += t;
    }
    // nobody exits while its value may still be read
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
  }
  const float inv = 1.f / sqrtf(total / float(H) + eps);
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i < v1) {
      F32Vec<VEC> w = load_vec<VEC>(weight + size_t(i) * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) w.v[e] *= x[j].v[e] * inv;
      store_vec<VEC>(out + base + size_t(i) * VEC, w);
    }
  }
}

template <typename T, typename S>
int launch_add_norm(void* residual, const void* planes, int n_planes, const void* slots, int n_slots,
                    const void* weight, void* out, int M, int H, float eps, cudaStream_t st) {
  const bool vec = H % 4 == 0 && !((reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(out) |
                                    reinterpret_cast<uintptr_t>(residual)) & 15);
  const int n = vec ? H / 4 : H;
  int cs = 1;
  while (cs < 8 && ((M * cs < 256 && n / (cs * 2) >= 64) || (n + cs - 1) / cs > kRowThreads * kRowRegs)) cs *= 2;
  if ((n + cs - 1) / cs > kRowThreads * kRowRegs) return ZSE_ERR_SHAPE;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(cs, M);
  cfg.blockDim = dim3(kRowThreads);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cs;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  auto kern = vec ? add_norm_kernel<T, S, 4> : add_norm_kernel<T, S, 1>;
  return cudaLaunchKernelEx(&cfg, kern, reinterpret_cast<float*>(residual), reinterpret_cast<const float*>(planes),
                            n_planes, reinterpret_cast<const S*>(slots), n_slots, reinterpret_cast<const T*>(weight),
                            reinterpret_cast<T*>(out), M, H, eps) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

__global__ void logits_finish_kernel(float* __restrict__ x, int ld, int V, float scale, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  float* row = x + size_t(blockIdx.y) * ld;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < V; i += gridDim.x * blockDim.x) {
    const float z = row[i] * scale;
    row[i] = cap > 0.f ? cap * tanhf(z / cap) : z;
  }
}

// lowest index of the row maximum
__global__ void __launch_bounds__(1024) argmax_f32_kernel(const float* __restrict__ x, int ld, int* __restrict__ out,
                                                          int V) {
  __shared__ unsigned long long red[32];
  pdl_launch_dependents();
  pdl_wait();
  const float* row = x + size_t(blockIdx.x) * ld;
  unsigned long long best = 0ull;
  for (int i = threadIdx.x; i < V; i += blockDim.x) {
    const uint32_t b = __float_as_uint(row[i]);
    const uint32_t key = (b & 0x80000000u) ? ~b : (b | 0x80000000u);
    const unsigned long long cand = ((unsigned long long)key << 32) | (0xFFFFFFFFu - (unsigned)i);
    best = cand > best ? cand : best;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const unsigned long long other = __shfl_xor_sync(0xffffffffu, best, o);
    best = other > best ? other : best;
  }
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = best;
  __syncthreads();
  if (threadIdx.x < 32) {
    best = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0ull;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const unsigned long long other = __shfl_xor_sync(0xffffffffu, best, o);
      best = other > best ? other : best;
    }
    if (threadIdx.x == 0) out[blockIdx.x] = int(0xFFFFFFFFu - unsigned(best & 0xFFFFFFFFull));
  }
}

}  // namespace
}  // namespace zse

using namespace zse;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int zse_embedding_typed(int dtype, const void* table, const void* ids, void* out, int M, int H, int vocab,
                                   float scale, void* status, void* stream) {
  if (M <= 0) return 0;
  cudaError_t e;
  if (dtype == kBF16)
    e = launch_pdl(embedding_typed_kernel<bf16>, dim3(M), dim3(128), 0, ST(stream), reinterpret_cast<const bf16*>(table),
                   reinterpret_cast<const int*>(ids), reinterpret_cast<float*>(out), H, vocab, scale,
                   reinterpret_cast<Status*>(status));
  else
    e = launch_pdl(embedding_typed_kernel<float>, dim3(M), dim3(128), 0, ST(stream),
                   reinterpret_cast<const float*>(table), reinterpret_cast<const int*>(ids),
                   reinterpret_cast<float*>(out), H, vocab, scale, reinterpret_cast<Status*>(status));
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_add_norm(int dtype, int slot_dtype, void* residual, const void* planes, int n_planes,
                            const void* slots, int n_slots, const void* weight, void* out, int M, int H, float eps,
                            void* stream) {
  if (M <= 0) return 0;
  if (dtype == kF32)
    return launch_add_norm<float, float>(residual, planes, n_planes, slots, n_slots, weight, out, M, H, eps, ST(stream));
  if (slot_dtype == kF32)
    return launch_add_norm<bf16, float>(residual, planes, n_planes, slots, n_slots, weight, out, M, H, eps, ST(stream));
  return launch_add_norm<bf16, bf16>(residual, planes, n_planes, slots, n_slots, weight, out, M, H, eps, ST(stream));
}

extern "C" int zse_logits_finish(void* logits, int ld, int M, int V, float scale, float cap, void* stream) {
  if (M <= 0 || V <= 0) return 0;
  return launch_pdl(logits_finish_kernel, dim3(min((V + 255) / 256, 64), M), dim3(256), 0, ST(stream),
                    reinterpret_cast<float*>(logits), ld, V, scale, cap) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_argmax_f32(const void* logits, int ld, void* out, int M, int V, void* stream) {
  if (M <= 0) return 0;
  return launch_pdl(argmax_f32_kernel, dim3(M), dim3(1024), 0, ST(stream), reinterpret_cast<const float*>(logits), ld,
                    reinterpret_cast<int*>(out), V) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}
