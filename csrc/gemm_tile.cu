// General matrix product on the CUDA cores, fp32 arithmetic throughout: any sizes, strides and alignments, batched over
// heads or grouped by expert.
//
//   out[m, n] = epilogue( scale[m] * sum_k A[m, k] * B[n, k] )          A, B bfloat16 or float
//
// It is the path of models that run in float, and of bfloat16 shapes whose rows are no multiple of 16 bytes (which TMA
// cannot address).  Epilogues: 0 store in the activation type, 1 store fp32, 2 gelu, 3 times sigmoid(gate[m, n]), 4 the
// square of relu.
#include "api.h"
#include "moe.cuh"
#include "typed.cuh"

namespace zse {
namespace {

constexpr int kBM = 64, kBN = 64, kBK = 16;

template <typename T>
__global__ void __launch_bounds__(256) gemm_tile_kernel(const ZseTileGemm a) {
  __shared__ float sa[kBK][kBM + 4];
  __shared__ float sb[kBK][kBN + 4];
  pdl_launch_dependents();
  pdl_wait();
  const int n0 = blockIdx.x * kBN, z = blockIdx.z;
  int m0 = blockIdx.y * kBM, m_end = a.M;
  const T* B = reinterpret_cast<const T*>(a.b) + z * a.b_batch;
  if (a.tiles != nullptr) {                          // grouped: the tile table says which expert and rows
    if (int(blockIdx.y) >= *a.n_tiles) return;
    const MoeTile t = reinterpret_cast<const MoeTile*>(a.tiles)[blockIdx.y];
    m0 = t.row0;
    m_end = t.row0 + t.rows;
    B += t.group * a.b_group;
  }
  const T* A = reinterpret_cast<const T*>(a.a) + z * a.a_batch;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += kBK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int idx = threadIdx.x + j * 256;
      const int m = idx / kBK, k = idx % kBK;        // A rows are contiguous in k
      sa[k][m] = (m0 + m < m_end && k0 + k < a.K) ? to_f32(A[size_t(m0 + m) * a.lda + k0 + k]) : 0.f;
      int n, kb;
      if (a.ldb_k == 1) {
        n = idx / kBK;
        kb = idx % kBK;
      } else {
        n = idx % kBN;
        kb = idx / kBN;
      }
      sb[kb][n] = (n0 + n < a.N && k0 + kb < a.K) ? to_f32(B[size_t(n0 + n) * a.ldb_n + size_t(k0 + kb) * a.ldb_k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kBK; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        x[i] = sa[k][ty * 4 + i];
        y[i] = sb[k][tx + 16 * i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= m_end) continue;
    const size_t om = a.out_rows != nullptr ? a.out_rows[m] : size_t(m) * a.out_row_mul + a.out_row_add;
    const float sc = a.row_scale != nullptr ? a.row_scale[m] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n >= a.N) continue;
      float v = acc[i][j] * sc;
      const size_t at = om * a.ldo + z * a.o_batch + n;
      if (a.epilogue == 1) {
        reinterpret_cast<float*>(a.out)[at] = v;
        continue;
      }
      if (a.epilogue == 2) v = gelu_exact(v);
      if (a.epilogue == 4) v = relu2(v);
      if (a.epilogue == 3)
        v *= sigmoid_exact(to_f32(reinterpret_cast<const T*>(a.gate)[size_t(m) * a.ldg + z * a.gate_batch + n]));
      reinterpret_cast<T*>(a.out)[at] = from_f32<T>(v);
    }
  }
}

// in [rows, 2 * ff] (gate, up) -> out [rows, ff]
template <typename T>
__global__ void __launch_bounds__(256)
glu_kernel(const T* __restrict__ in, T* __restrict__ out, int ldo, long long n, int ff, int kind, float limit) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) {
    const T* g = in + i / ff * 2 * ff + i % ff;
    out[i / ff * ldo + i % ff] = from_f32<T>(glu<false>(kind, to_f32(g[0]), to_f32(g[ff]), limit));
  }
}

}  // namespace
}  // namespace zse

using namespace zse;

extern "C" int zse_glu(int dtype, const void* in, void* out, int ldo, int rows, int ff, int kind, float limit, void* stream) {
  const long long n = (long long)(rows) * ff;
  if (n <= 0) return 0;
  const dim3 grid(unsigned(n + 255 < 4096ll * 256 ? (n + 255) / 256 : 4096));
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (dtype == kBF16)
    e = launch_pdl(glu_kernel<bf16>, grid, dim3(256), 0, st, reinterpret_cast<const bf16*>(in),
                   reinterpret_cast<bf16*>(out), ldo, n, ff, kind, limit);
  else
    e = launch_pdl(glu_kernel<float>, grid, dim3(256), 0, st, reinterpret_cast<const float*>(in),
                   reinterpret_cast<float*>(out), ldo, n, ff, kind, limit);
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_gemm_tile(int dtype, const ZseTileGemm* a, int batch, int max_tiles, void* stream) {
  const int my = a->tiles != nullptr ? max_tiles : (a->M + kBM - 1) / kBM;
  if (my <= 0 || a->N <= 0 || batch <= 0) return 0;
  if (my > 65535 || batch > 65535) return ZSE_ERR_LIMIT;
  dim3 grid((a->N + kBN - 1) / kBN, my, batch);
  auto kern = dtype == kBF16 ? gemm_tile_kernel<bf16> : gemm_tile_kernel<float>;
  return launch_pdl(kern, grid, dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), *a) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}
