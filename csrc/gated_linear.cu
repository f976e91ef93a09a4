// Gated linear attention: per head S [dim, vdim] in fp32, whose rows (key channels) decay each at its own rate,
//
//   S' = diag(alpha) S + k v^T;  o = S'^T q dim^(-1/2);  y = o / rms(o) * norm * silu(g)
//
// with alpha = sigmoid(z)^(1 / tau), z = W_a2 u + bias from an inner vector u of low rank.
// (S. Yang, B. Wang, Y. Shen, R. Panda, Y. Kim: Gated Linear Attention Transformers with Hardware-Efficient Training.)
//
//   gl_prep     second half of the fused input projection [q | k | v | g | u]: split-K sum, logarithms of the decays
//   gl_tokens   token by token (decode, short portions, any shape, any type): a cluster per head and sequence makes one pass over
//               S for update and read-out; the head norm's sum crosses the cluster; a decode step sums the split-K planes and
//               makes the decays here as well
//   gl_chunk    chunks of 64 tokens (bfloat16): a CTA per (64 columns of S, head, sequence) keeps its part of S in accumulators
//               and walks through the sequence; gl_out norms and gates what it read
//
// Inside a chunk, with b_t the sum of log alpha up to t (per channel), the read-out is
//   o_t = (q_t exp(b_t))^T S_start + sum_{s <= t} A_ts v_s,   A_ts = sum_d q_t[d] k_s[d] exp(b_t[d] - b_s[d])
//   S_end = exp(b_end) S_start + sum_s (k_s exp(b_end - b_s)) v_s^T
// A is made in blocks of 16 tokens: with r the b before the first token of t's block, the product of q_t exp(b_t - r) and
// k_s exp(r - b_s).  Only keys of t's own block have positive exponents; where a channel decays so fast that those could leave
// fp32, the blocks on the diagonal are summed element by element instead, whose exponents b_t - b_s are never positive.
// All that a decay has touched - S, A, weighted queries and keys - enters the tensor-core products as two bfloat16 terms, value
// and remainder (of the product of two such factors the remainders' own is left out).
//
// State rows come in pairs: a pass reads one row (-1: zero) and writes another, see cache/state_slots.py.
#include "api.h"
#include "typed.cuh"

namespace zse {
namespace {

struct Gl {
  int heads, dim, vdim, rank, q_col, k_col, v_col, gate_col, rank_col;
  float* states;
  long long row_floats;
  const int* state_rows;
  int state_ld;
  float tau, eps, out_scale;
  const float *decay_w, *decay_b;
};

// log(sigmoid(z)) = min(z, 0) - log(1 + e), e = exp(-|z|) in (0, 1].  log(1 + e) = 2 artanh(s) with s = e / (2 + e) <= 1/3, by
// the series of artanh, whose first terms left out are below 2^-27 of it.
__device__ __forceinline__ float log_sigmoid(float z) {
  const float e = ex2(fabsf(z) * -kLog2E), s = e * rcp(2.f + e), q = s * s;
  float p = 1.f / 15.f;
  p = fmaf(p, q, 1.f / 13.f);
  p = fmaf(p, q, 1.f / 11.f);
  p = fmaf(p, q, 1.f / 9.f);
  p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 1.f / 5.f);
  p = fmaf(p, q, 1.f / 3.f);
  p = fmaf(p, q, 1.f);
  return fminf(z, 0.f) - 2.f * s * p;
}

// ---- prep -----------------------------------------------------------------------------------------------------------
constexpr int kGpThreads = 256, kGpGroup = 16, kGpCols = kGpThreads * 4;      // rows that share a reading of the weights

// grid (blocks of rows, pieces of channels + pieces of columns); u rows in shared memory, padded to 4 floats
template <typename T>
__global__ void __launch_bounds__(kGpThreads)
gl_prep_kernel(T* __restrict__ inp, int ld, const float* __restrict__ planes, int n_planes, const float* __restrict__ side,
               int side_ld, const Gl m, float* __restrict__ decays, int M, int channel_pieces, int rows) {
  extern __shared__ __align__(16) float us[];
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * rows, n = min(M - t0, rows);
  const size_t plane = size_t(M) * ld;
  if (blockIdx.y >= channel_pieces) {            // with planes: the columns before the inner vectors
    const int c = m.q_col + (blockIdx.y - channel_pieces) * kGpCols + threadIdx.x * 4;
    if (c >= m.rank_col) return;
#pragma unroll 2
    for (int j = 0; j < n; ++j) {
      const size_t at = size_t(t0 + j) * ld + c;
      F32Vec<4> x{};
#pragma unroll 4
      for (int p = 0; p < n_planes; ++p) {
        const F32Vec<4> y = load_vec<4>(planes + p * plane + at);
#pragma unroll
        for (int e = 0; e < 4; ++e) x.v[e] += y.v[e];
      }
      store_vec<4>(inp + at, x);
    }
    return;
  }
  const int rp = (m.rank + 3) / 4 * 4, width = m.heads * m.dim;
  for (int i = threadIdx.x; i < n * rp; i += kGpThreads) {
    const int j = i / rp, r = i % rp, t = t0 + j;
    float x = 0.f;
    if (r < m.rank) {
      if (n_planes > 0) {
        for (int p = 0; p < n_planes; ++p) x += planes[p * plane + size_t(t) * ld + m.rank_col + r];
      } else {
        x = side != nullptr ? side[size_t(t) * side_ld + r] : to_f32(inp[size_t(t) * ld + m.rank_col + r]);
      }
    }
    us[i] = x;
  }
  __syncthreads();
  const int c = blockIdx.y * kGpThreads + threadIdx.x;
  if (c >= width) return;
  const float bias = m.decay_b[c], inv = 1.f / m.tau;
  auto weights = [&](int r, float (&w)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) w[e] = r + e < m.rank ? m.decay_w[size_t(c) * m.rank + r + e] : 0.f;
  };
  auto add = [&](float z, const float (&w)[4], const float* at) {
    const float4 u = *reinterpret_cast<const float4*>(at);
    return fmaf(w[0], u.x, fmaf(w[1], u.y, fmaf(w[2], u.z, fmaf(w[3], u.w, z))));
  };
  float* dst = decays + size_t(t0) * width + c;
  if (rp == 16) {                                // the weights stay in registers
    float w[4][4];
#pragma unroll
    for (int r = 0; r < 4; ++r) weights(r * 4, w[r]);
#pragma unroll 4
    for (int j = 0; j < n; ++j) {
      float z = bias;
#pragma unroll
      for (int r = 0; r < 4; ++r) z = add(z, w[r], us + j * 16 + r * 4);
      dst[size_t(j) * width] = log_sigmoid(z) * inv;
    }
    return;
  }
  for (int j0 = 0; j0 < n; j0 += kGpGroup) {
    float z[kGpGroup];
#pragma unroll
    for (int j = 0; j < kGpGroup; ++j) z[j] = bias;
    for (int r = 0; r < rp; r += 4) {
      float w[4];
      weights(r, w);
#pragma unroll
      for (int j = 0; j < kGpGroup; ++j) z[j] = add(z[j], w, us + min(j0 + j, n - 1) * rp + r);
    }
#pragma unroll
    for (int j = 0; j < kGpGroup; ++j)
      if (j0 + j < n) dst[size_t(j0 + j) * width] = log_sigmoid(z[j]) * inv;
  }
}

// ---- token by token ----------------------------------------------------------------------------------------------------
constexpr int kGtThreads = 256, kGtBatch = 8;

__device__ __forceinline__ float gt_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int w = 0; w < kGtThreads / 32; ++w) s += red[w];
  return s;
}

// grid (cluster, heads, sequences)
template <typename T, int VEC>
__global__ void __launch_bounds__(kGtThreads, 3)
gl_tokens_kernel(const T* __restrict__ inp, int ld, const float* __restrict__ planes, int n_planes, int M,
                 const float* __restrict__ decays, const Gl m, const int* __restrict__ cu_q, const T* __restrict__ head_norm,
                 T* __restrict__ out, int ldo) {
  extern __shared__ __align__(16) float sm[];    // q, k, alpha [dim] each; u [rank]; v, o [columns of this CTA]
  __shared__ float red[kGtThreads / 32];
  __shared__ float part[kGtThreads * VEC];
  __shared__ float cluster_ss;
  pdl_launch_dependents();
  pdl_wait();
  const int cs = gridDim.x, head = blockIdx.y, s = blockIdx.z;
  const int nvec = m.vdim / VEC, share = (nvec + cs - 1) / cs;
  const int c0 = blockIdx.x * share, nc = max(0, min(nvec, c0 + share) - c0);      // column vectors of this CTA
  float *q = sm, *k = q + m.dim, *alpha = k + m.dim, *u = alpha + m.dim, *v = u + m.rank, *o = v + share * VEC;
  const int first = cu_q != nullptr ? cu_q[s] : s, last = cu_q != nullptr ? cu_q[s + 1] : s + 1;
  const int read = m.state_rows[s], write = m.state_rows[m.state_ld + s];
  const size_t mem_at = size_t(head) * m.dim * m.vdim + size_t(c0) * VEC;
  float* dst = m.states + size_t(max(write, 0)) * m.row_floats + mem_at;
  const float* from = read >= 0 ? m.states + size_t(read) * m.row_floats + mem_at : nullptr;
  int cw = 1;                                    // column vectors side by side
  while (cw * 2 <= nc && cw < 64) cw *= 2;
  const int tc = threadIdx.x % cw, tr = threadIdx.x / cw, rows = kGtThreads / cw;
  const float q_scale = 1.f / sqrtf(float(m.dim)), inv_tau = 1.f / m.tau;
  const size_t plane = size_t(M) * ld;
  const bool summed = n_planes == 0 || decays != nullptr;          // inp holds the projection
  for (int t = first; t < last; ++t) {
    auto value = [&](int c) {
      if (summed) return to_f32(inp[size_t(t) * ld + c]);
      float x = 0.f;
#pragma unroll 4
      for (int p = 0; p < n_planes; ++p) x += planes[p * plane + size_t(t) * ld + c];
      return x;
    };
    F32Vec<VEC> x[kGtBatch];
    auto fetch = [&](int cb, int d0) {
#pragma unroll
      for (int i = 0; i < kGtBatch; ++i) {
        const int d = d0 + i * rows;
        x[i] = F32Vec<VEC>{};
        if (from != nullptr && d < m.dim && cb + tc < nc) x[i] = load_vec<VEC>(from + size_t(d) * m.vdim + (cb + tc) * VEC);
      }
    };
    fetch(0, tr);                                // under way while the row is taken in
    if (decays == nullptr)
      for (int i = threadIdx.x; i < m.rank; i += kGtThreads) u[i] = value(m.rank_col + i);
    for (int i = threadIdx.x; i < m.dim; i += kGtThreads) {
      q[i] = value(m.q_col + head * m.dim + i) * q_scale;
      k[i] = value(m.k_col + head * m.dim + i);
      if (decays != nullptr) alpha[i] = expf(decays[size_t(t) * m.heads * m.dim + head * m.dim + i]);
    }
    for (int i = threadIdx.x; i < nc * VEC; i += kGtThreads) v[i] = value(m.v_col + head * m.vdim + c0 * VEC + i);
    __syncthreads();
    if (decays == nullptr) {
      for (int i = threadIdx.x; i < m.dim; i += kGtThreads) {
        const float* w = m.decay_w + size_t(head * m.dim + i) * m.rank;
        float z = m.decay_b[head * m.dim + i];
#pragma unroll 4
        for (int r = 0; r < m.rank; ++r) z = fmaf(w[r], u[r], z);
        alpha[i] = expf(log_sigmoid(z) * inv_tau);
      }
      __syncthreads();
    }
    float ss = 0.f;
    for (int cb = 0; cb < nc; cb += cw) {
      F32Vec<VEC> acc{};
      const int col = (cb + tc) * VEC;
      F32Vec<VEC> vv{};
      if (cb + tc < nc) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) vv.v[e] = v[col + e];
      }
      // a batch of loads is under way before the first store (which might alias the next loads)
      for (int d0 = tr; d0 < m.dim; d0 += rows * kGtBatch) {
        if (cb > 0 || d0 != tr) fetch(cb, d0);
        if (cb + tc >= nc) continue;
#pragma unroll
        for (int i = 0; i < kGtBatch; ++i) {
          const int d = d0 + i * rows;
          if (d >= m.dim) break;
          const float kd = k[d], qd = q[d], ad = alpha[d];
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            x[i].v[e] = fmaf(ad, x[i].v[e], kd * vv.v[e]);
            acc.v[e] = fmaf(qd, x[i].v[e], acc.v[e]);
          }
          if (write >= 0) store_vec<VEC>(dst + size_t(d) * m.vdim + col, x[i]);
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) part[threadIdx.x * VEC + e] = acc.v[e];
      __syncthreads();
      for (int i = threadIdx.x; i < cw * VEC && cb * VEC + i < nc * VEC; i += kGtThreads) {
        float y = 0.f;
        for (int r = 0; r < rows; ++r) y += part[r * cw * VEC + i];
        o[cb * VEC + i] = y;
        ss += y * y;
      }
      __syncthreads();
    }
    ss = gt_sum(ss, red);
    if (cs > 1) {
      if (threadIdx.x == 0) cluster_ss = ss;
      asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
      ss = 0.f;
      const uint32_t local = smem_u32(&cluster_ss);
      for (int r = 0; r < cs; ++r) {             // same order in every CTA: identical sums
        uint32_t remote;
        float y;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(r));
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(y) : "r"(remote) : "memory");
        ss += y;
      }
      // nobody overwrites its value, or exits, while it may still be read
      asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    }
    const float inv = m.out_scale / sqrtf(ss / float(m.vdim) + m.eps);
    for (int i = threadIdx.x; i < nc * VEC; i += kGtThreads) {
      const int c = c0 * VEC + i;
      const float y = o[i] * inv * to_f32(head_norm[c]) * silu_exact(value(m.gate_col + head * m.vdim + c));
      out[size_t(t) * ldo + head * m.vdim + c] = from_f32<T>(y);
    }
    from = dst;                                  // the next token starts from what this thread has written
    __syncthreads();
  }
}

// ---- chunks of 64 tokens -----------------------------------------------------------------------------------------------
constexpr int kGcT = 64, kGcC = 64, kGcThreads = 256;    // tokens, columns of S per CTA
constexpr int kGcPitch = (kGcC / 8 + 1) * 16;            // bytes of a row of 64 columns
constexpr float kGcFar = 100.f;                          // decay of a channel within 16 tokens, in powers of two

__host__ __device__ inline int gl_steps(int dim) { return (dim + 15) / 16; }
__host__ __device__ inline int gl_pitch(int dim) { return (gl_steps(dim) * 2 + 1) * 16; }       // bytes of a row of q or k
__host__ __device__ inline int gl_bpitch(int dim) { return gl_steps(dim) * 16 + 8; }            // floats of a row of b
__host__ __device__ inline int gl_overlay(int dim) {     // S in two terms, later A in two terms
  const int rows = gl_steps(dim) * 16;
  return 2 * kGcPitch * (rows > kGcT ? rows : kGcT);
}
inline size_t gl_chunk_smem(int dim) {
  return size_t(2) * kGcT * gl_pitch(dim) + size_t(kGcT) * kGcPitch + gl_overlay(dim) + size_t(kGcT) * gl_bpitch(dim) * 4;
}

__device__ __forceinline__ float2 unpack_bf16(uint32_t x) {
  return make_float2(__uint_as_float(x << 16), __uint_as_float(x & 0xFFFF0000u));
}

// value and remainder of two numbers
__device__ __forceinline__ void two_terms(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  const float2 v = unpack_bf16(hi);
  lo = pack_bf16(x - v.x, y - v.y);
}

// MT: 16-row tiles of S per warp (8 warps: dim <= 128 * MT).  grid (column blocks, heads, sequences)
template <int MT>
__global__ void __launch_bounds__(kGcThreads, MT == 1 ? 2 : 1)
gl_chunk_kernel(const bf16* __restrict__ inp, int ld, const float* __restrict__ decays, const Gl m,
                const int* __restrict__ cu_q, int first, float* __restrict__ o_out) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int cb = blockIdx.x * kGcC, head = blockIdx.y, s = first + blockIdx.z, N = m.dim;
  const int nc = min(kGcC, m.vdim - cb);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qp = gl_pitch(N), ksteps = gl_steps(N), dch = N / 8, bp = gl_bpitch(N);
  uint8_t* sq = smem;
  uint8_t* sk = sq + kGcT * qp;
  uint8_t* sv = sk + kGcT * qp;
  uint8_t* ssh = sv + kGcT * kGcPitch;           // S at the chunk's start, two terms
  uint8_t* ssl = ssh + ksteps * 16 * kGcPitch;
  uint8_t* sph = ssh;                            // in the same place: A, two terms
  uint8_t* spl = sph + kGcT * kGcPitch;
  float* sb = reinterpret_cast<float*>(ssh + gl_overlay(N));       // b, in units of ln 2

  const int begin = cu_q[s], end = cu_q[s + 1];
  const int read = m.state_rows[s], write = m.state_rows[m.state_ld + s];
  const float* src = m.states + size_t(max(read, 0)) * m.row_floats + size_t(head) * N * m.vdim + cb;
  const int r4 = lane >> 2, c2 = (lane & 3) * 2;
  const float q_scale = 1.f / sqrtf(float(N));
  const int HD = m.heads * N, ldo = m.heads * m.vdim;

  // this warp's part of S: tiles of 16 rows warp * MT + i, 8 blocks of 8 columns
  float S[MT][8][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = (warp * MT + i) * 16 + r4 + h * 8, c = n * 8 + c2;
        float2 x = make_float2(0.f, 0.f);
        if (read >= 0 && d < N && c < nc) x = *reinterpret_cast<const float2*>(src + size_t(d) * m.vdim + c);
        S[i][n][h * 2] = x.x;
        S[i][n][h * 2 + 1] = x.y;
      }
  for (int i = threadIdx.x; i < kGcT; i += kGcThreads) {           // what no copy writes
    if (dch < ksteps * 2) {
      *reinterpret_cast<uint4*>(sq + i * qp + dch * 16) = make_uint4(0, 0, 0, 0);
      *reinterpret_cast<uint4*>(sk + i * qp + dch * 16) = make_uint4(0, 0, 0, 0);
    }
    for (int c = N; c < bp; ++c) sb[i * bp + c] = 0.f;
  }

  // 16 tokens and half of the columns in the read-out; later tokens have more work, so a scheduler's two warps share it
  const int pc = warp >> 2, pr = pc ? 3 - (warp & 3) : warp & 3;
  for (int t0 = begin; t0 < end; t0 += kGcT) {
    const int len = min(kGcT, end - t0);
    for (int i = threadIdx.x; i < kGcT * dch; i += kGcThreads) {
      const int r = i / dch, c = i % dch;
      uint8_t *qd = sq + r * qp + c * 16, *kd = sk + r * qp + c * 16;
      float* bd = sb + r * bp + c * 8;
      if (r < len) {
        const bf16* row = inp + size_t(t0 + r) * ld + head * N + c * 8;
        const float* g = decays + size_t(t0 + r) * HD + head * N + c * 8;
        cpa16(qd, row + m.q_col);
        cpa16(kd, row + m.k_col);
        cpa16(bd, g);
        cpa16(bd + 4, g + 4);
      } else {                                   // tokens past the end neither decay nor add
        *reinterpret_cast<uint4*>(qd) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(kd) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(bd) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(bd + 4) = make_uint4(0, 0, 0, 0);
      }
    }
    for (int i = threadIdx.x; i < kGcT * (kGcC / 8); i += kGcThreads) {
      const int r = i / (kGcC / 8), c = i % (kGcC / 8);
      uint8_t* vd = sv + r * kGcPitch + c * 16;
      if (r < len && c * 8 < nc)
        cpa16(vd, inp + size_t(t0 + r) * ld + m.v_col + head * m.vdim + cb + c * 8);
      else
        *reinterpret_cast<uint4*>(vd) = make_uint4(0, 0, 0, 0);
    }
    cpa_commit();
    // S in two terms
#pragma unroll
    for (int i = 0; i < MT; ++i)
      if ((warp * MT + i) * 16 < N) {
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int at = ((warp * MT + i) * 16 + r4 + h * 8) * kGcPitch + (n * 8 + c2) * 2;
            two_terms(S[i][n][h * 2], S[i][n][h * 2 + 1], *reinterpret_cast<uint32_t*>(ssh + at),
                      *reinterpret_cast<uint32_t*>(ssl + at));
          }
      }
    cpa_wait<0>();
    __syncthreads();
    // sums of the logarithms: two lanes per channel, 32 tokens each
    bool far = false;
    for (int d0 = 0; d0 < N; d0 += kGcThreads / 2) {
      const int d = d0 + (threadIdx.x >> 1), half = threadIdx.x & 1;
      float* col = sb + (half * 32) * bp + min(d, N - 1);
      float b[32];
      float run = 0.f;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        run = fmaf(col[i * bp], kLog2E, run);
        b[i] = run;
      }
      const float other = __shfl_xor_sync(0xffffffffu, run, 1);
      far |= d < N && (-b[15] > kGcFar || b[15] - b[31] > kGcFar);
      const float base = half ? other : 0.f;
      __syncwarp();
      if (d < N) {
#pragma unroll
        for (int i = 0; i < 32; ++i) col[i * bp] = b[i] + base;
      }
    }
    const bool slow = __syncthreads_or(far) != 0;
    // A of this warp's 16 tokens against the chunk's keys 32 pc .. 32 pc + 31, and q S
    float sc[4][4] = {}, acc[4][4] = {};
    const int blocks = min(2, pr + 1 - pc * 2);  // blocks of 16 keys up to the tokens' own
    const uint32_t q_addr = smem_u32(sq) + (pr * 16 + (lane & 15)) * qp + (lane >> 4) * 16;
    const uint32_t k_addr = smem_u32(sk) + (pc * 32 + (lane >> 4) * 8 + (lane & 7)) * qp + (lane >> 3 & 1) * 16;
    const uint32_t s_row = ((lane >> 3 & 1) * 8 + (lane & 7)) * kGcPitch + (lane >> 4) * 16 + pc * 64;
    const uint32_t sh_addr = smem_u32(ssh) + s_row, sl_addr = smem_u32(ssl) + s_row;
    const float* b_q = sb + (pr * 16 + r4) * bp + c2;
    const float* b_ref = sb + (pr * 16 - 1) * bp + c2;             // not read for pr 0
    const float* b_k = sb + (pc * 32 + r4) * bp + c2;
    for (int kk = 0; kk < ksteps; ++kk) {
      uint32_t b[4], qh[4], ql[4], sh[4], sl[4];   // queries towards their block's start, and towards the chunk's
      ldm_x4(q_addr + kk * 32, qh);
      float2 ref[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
      if (pr > 0) {
        ref[0] = *reinterpret_cast<const float2*>(b_ref + kk * 16);
        ref[1] = *reinterpret_cast<const float2*>(b_ref + kk * 16 + 8);
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {              // columns c2 and c2 + 8 of the step
        const float ex = ex2(ref[x].x), ey = ex2(ref[x].y);
#pragma unroll
        for (int h = 0; h < 2; ++h) {            // rows r4 and r4 + 8
          const float2 bt = *reinterpret_cast<const float2*>(b_q + h * 8 * bp + kk * 16 + x * 8);
          const float2 q = unpack_bf16(qh[x * 2 + h]);
          const float qx = q.x * q_scale * ex2(bt.x - ref[x].x), qy = q.y * q_scale * ex2(bt.y - ref[x].y);
          two_terms(qx, qy, qh[x * 2 + h], ql[x * 2 + h]);
          two_terms(qx * ex, qy * ey, sh[x * 2 + h], sl[x * 2 + h]);
        }
      }
#pragma unroll
      for (int n = 0; n < 4; n += 2) {
        ldm_x4_t(sh_addr + kk * 16 * kGcPitch + n * 16, b);
        mma_bf16(acc[n], sh, b[0], b[1]);
        mma_bf16(acc[n + 1], sh, b[2], b[3]);
        mma_bf16(acc[n], sl, b[0], b[1]);
        mma_bf16(acc[n + 1], sl, b[2], b[3]);
        ldm_x4_t(sl_addr + kk * 16 * kGcPitch + n * 16, b);
        mma_bf16(acc[n], sh, b[0], b[1]);
        mma_bf16(acc[n + 1], sh, b[2], b[3]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        if (j >= blocks || (slow && pc * 2 + j == pr)) continue;
        uint32_t bl[4];
        ldm_x4(k_addr + j * 16 * qp + kk * 32, b);
#pragma unroll
        for (int h = 0; h < 2; ++h)              // keys r4 and r4 + 8 of the block
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const float2 bs = *reinterpret_cast<const float2*>(b_k + (j * 16 + h * 8) * bp + kk * 16 + x * 8);
            const float2 key = unpack_bf16(b[h * 2 + x]);
            two_terms(key.x * ex2(ref[x].x - bs.x), key.y * ex2(ref[x].y - bs.y), b[h * 2 + x], bl[h * 2 + x]);
          }
        mma_bf16(sc[j * 2], qh, b[0], b[1]);
        mma_bf16(sc[j * 2 + 1], qh, b[2], b[3]);
        mma_bf16(sc[j * 2], ql, b[0], b[1]);
        mma_bf16(sc[j * 2 + 1], ql, b[2], b[3]);
        mma_bf16(sc[j * 2], qh, bl[0], bl[1]);
        mma_bf16(sc[j * 2 + 1], qh, bl[2], bl[3]);
      }
    }
    if (slow && (pr >> 1) == pc) {               // the block on the diagonal, element by element
      float x[2][4] = {};                        // as sc of that block: rows r4, r4 + 8, keys c2, c2 + 1 and eight on
      for (int d = 0; d < N; ++d)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = pr * 16 + r4 + h * 8;
          const float q = to_f32(reinterpret_cast<const bf16*>(sq + t * qp)[d]) * q_scale, bt = sb[t * bp + d];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int c = pr * 16 + (e >> 1) * 8 + c2 + (e & 1);
            const float key = to_f32(reinterpret_cast<const bf16*>(sk + c * qp)[d]);
            if (c <= t) x[e >> 1][h * 2 + (e & 1)] = fmaf(q * key, ex2(bt - sb[c * bp + d]), x[e >> 1][h * 2 + (e & 1)]);
          }
        }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (pr & 1)
            sc[2 + n][e] = x[n][e];
          else
            sc[n][e] = x[n][e];
        }
    }
    __syncthreads();                             // S has been read: A takes its place
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = pr * 16 + r4 + h * 8;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int c = pc * 32 + n * 8 + c2;
        const float x = c <= t ? sc[n][h * 2] : 0.f, y = c + 1 <= t ? sc[n][h * 2 + 1] : 0.f;
        two_terms(x, y, *reinterpret_cast<uint32_t*>(sph + t * kGcPitch + c * 2),
                  *reinterpret_cast<uint32_t*>(spl + t * kGcPitch + c * 2));
      }
    }
    __syncthreads();
    // A times v
    const uint32_t p_row = (pr * 16 + (lane & 15)) * kGcPitch + (lane >> 4) * 16;
    const uint32_t v_row = ((lane >> 3 & 1) * 8 + (lane & 7)) * kGcPitch + (lane >> 4) * 16;
    const uint32_t v_addr = smem_u32(sv) + v_row + pc * 64;
#pragma unroll
    for (int kk = 0; kk < kGcT / 16; ++kk) {
      if (kk <= pr) {
        uint32_t ph[4], pl[4], b[4];
        ldm_x4(smem_u32(sph) + p_row + kk * 32, ph);
        ldm_x4(smem_u32(spl) + p_row + kk * 32, pl);
#pragma unroll
        for (int n = 0; n < 4; n += 2) {
          ldm_x4_t(v_addr + kk * 16 * kGcPitch + n * 16, b);
          mma_bf16(acc[n], ph, b[0], b[1]);
          mma_bf16(acc[n], pl, b[0], b[1]);
          mma_bf16(acc[n + 1], ph, b[2], b[3]);
          mma_bf16(acc[n + 1], pl, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = pr * 16 + r4 + h * 8;
      if (t >= len) continue;
      float* o = o_out + size_t(t0 + t) * ldo + head * m.vdim + cb;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int c = pc * 32 + n * 8 + c2;
        if (c < nc) *reinterpret_cast<float2*>(o + c) = make_float2(acc[n][h * 2], acc[n][h * 2 + 1]);
      }
    }
    // next state
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int mt = warp * MT + i;
      if (mt * 16 >= N) continue;
      float b_end[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        b_end[h] = sb[(kGcT - 1) * bp + mt * 16 + r4 + h * 8];
        const float keep = ex2(b_end[h]);
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          S[i][n][h * 2] *= keep;
          S[i][n][h * 2 + 1] *= keep;
        }
      }
      const uint32_t kt = smem_u32(sk) + ((lane >> 4) * 8 + (lane & 7)) * qp + (mt * 16 + (lane >> 3 & 1) * 8) * 2;
      const float* b_s = sb + c2 * bp + mt * 16 + r4;
#pragma unroll
      for (int kk = 0; kk < kGcT / 16; ++kk) {
        uint32_t a[4], al[4], b[4];
        ldm_x4_t(kt + kk * 16 * qp, a);
#pragma unroll
        for (int x = 0; x < 2; ++x)              // tokens c2, c2 + 1 and eight on
#pragma unroll
          for (int h = 0; h < 2; ++h) {          // channels r4 and r4 + 8
            const float* at = b_s + (kk * 16 + x * 8) * bp + h * 8;
            const float2 key = unpack_bf16(a[x * 2 + h]);
            const float k0 = key.x * ex2(b_end[h] - at[0]), k1 = key.y * ex2(b_end[h] - at[bp]);
            two_terms(k0, k1, a[x * 2 + h], al[x * 2 + h]);
          }
        const uint32_t w = smem_u32(sv) + v_row + kk * 16 * kGcPitch;
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
          ldm_x4_t(w + n * 16, b);
          mma_bf16(S[i][n], a, b[0], b[1]);
          mma_bf16(S[i][n + 1], a, b[2], b[3]);
          mma_bf16(S[i][n], al, b[0], b[1]);
          mma_bf16(S[i][n + 1], al, b[2], b[3]);
        }
      }
    }
    __syncthreads();                             // everyone is done with the chunk's tiles
  }
  if (write < 0) return;
  float* dst = m.states + size_t(write) * m.row_floats + size_t(head) * N * m.vdim + cb;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = (warp * MT + i) * 16 + r4 + h * 8, c = n * 8 + c2;
        if (d < N && c < nc)
          *reinterpret_cast<float2*>(dst + size_t(d) * m.vdim + c) = make_float2(S[i][n][h * 2], S[i][n][h * 2 + 1]);
      }
}

// A warp per (row, head): y = o / rms(o) * norm * silu(g) * out_scale.
__global__ void __launch_bounds__(256)
gl_out_kernel(const float* __restrict__ o, const bf16* __restrict__ inp, int ld, const Gl m, const bf16* __restrict__ head_norm,
              bf16* __restrict__ out, int ldo, int row0, int rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long id = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (id >= (long long)(rows) * m.heads) return;
  const int t = row0 + int(id / m.heads), head = int(id % m.heads), c0 = head * m.vdim;
  const float* src = o + size_t(t) * m.heads * m.vdim + c0;
  float ss = 0.f;
#pragma unroll 4
  for (int i = lane * 4; i < m.vdim; i += 128) {
    const F32Vec<4> x = load_vec<4>(src + i);
#pragma unroll
    for (int e = 0; e < 4; ++e) ss += x.v[e] * x.v[e];
  }
  const float inv = m.out_scale / sqrtf(warp_sum(ss) / float(m.vdim) + m.eps);
#pragma unroll 4
  for (int i = lane * 4; i < m.vdim; i += 128) {
    F32Vec<4> x = load_vec<4>(src + i);
    const F32Vec<4> w = load_vec<4>(head_norm + i), g = load_vec<4>(inp + size_t(t) * ld + m.gate_col + c0 + i);
#pragma unroll
    for (int e = 0; e < 4; ++e) x.v[e] *= inv * w.v[e] * (g.v[e] * sigmoid_fast(g.v[e]));
    store_vec<4>(out + size_t(t) * ldo + c0 + i, x);
  }
}

template <typename K>
int raise_smem(K kern, size_t bytes, size_t* done) {      // `done`: per device, the size already granted
  const int slot = current_device_slot();
  if (bytes > done[slot]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(bytes)) != cudaSuccess)
      return ZSE_ERR_LAUNCH;
    done[slot] = bytes;
  }
  return 0;
}

Gl gl_of(const ZseGatedLinear* z) {
  return Gl{z->heads, z->dim, z->vdim, z->rank, z->q_col, z->k_col, z->v_col, z->gate_col, z->rank_col,
            reinterpret_cast<float*>(z->states), (long long)(z->row_floats), reinterpret_cast<const int*>(z->state_rows),
            z->state_ld, z->tau, z->eps, z->out_scale, reinterpret_cast<const float*>(z->decay_w),
            reinterpret_cast<const float*>(z->decay_b)};
}

bool gl_shape_ok(const ZseGatedLinear* z) {
  return z->heads > 0 && z->heads <= 65535 && z->dim > 0 && z->vdim > 0 && z->rank > 0 && z->tau > 0.f;
}

template <typename T>
int launch_gl_prep(void* inp, int ld, const void* planes, int n_planes, const void* side, int side_ld, const ZseGatedLinear* z,
                   void* decays, int M, cudaStream_t st) {
  const Gl m = gl_of(z);
  const int pieces = (m.heads * m.dim + kGpThreads - 1) / kGpThreads;
  const int copies = n_planes > 0 ? (m.rank_col - m.q_col + kGpCols - 1) / kGpCols : 0;
  const int rp = (m.rank + 3) / 4 * 4;
  int rows = M >= 4096 ? 64 : 16;
  while (rows > 1 && size_t(rows) * rp * sizeof(float) > 48 * 1024) rows /= 2;
  const size_t smem = size_t(rows) * rp * sizeof(float);
  if (smem > 48 * 1024) return ZSE_ERR_LIMIT;
  return launch_pdl(gl_prep_kernel<T>, dim3((M + rows - 1) / rows, pieces + copies), dim3(kGpThreads), smem, st,
                    reinterpret_cast<T*>(inp), ld, reinterpret_cast<const float*>(planes), n_planes,
                    reinterpret_cast<const float*>(side), side_ld, m, reinterpret_cast<float*>(decays), M, pieces,
                    rows) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

template <typename T, int VEC>
int launch_gl_tokens(const ZseGatedLinear* z, const void* inp, int ld, const void* planes, int n_planes, int M,
                     const void* decays, const void* cu_q, int S, void* out, int ldo, cudaStream_t st) {
  static size_t done[kMaxDevices] = {};
  const Gl m = gl_of(z);
  auto kern = gl_tokens_kernel<T, VEC>;
  // CTAs of a cluster share a head's columns: enough of them to fill the GPU, at least 32 columns each
  int cs = 1;
  while (cs < 8 && S * m.heads * cs < 2 * 148 && m.vdim / (cs * 2) >= 32) cs *= 2;
  const int share = (m.vdim / VEC + cs - 1) / cs * VEC;
  const size_t smem = (size_t(3) * m.dim + m.rank + 2 * share) * sizeof(float);
  if (smem > 200 * 1024) return ZSE_ERR_LIMIT;
  if (smem > 40 * 1024)
    if (int r = raise_smem(kern, smem, done)) return r;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(cs, m.heads, S);
  cfg.blockDim = dim3(kGtThreads);
  cfg.dynamicSmemBytes = smem;
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
  return cudaLaunchKernelEx(&cfg, kern, reinterpret_cast<const T*>(inp), ld, reinterpret_cast<const float*>(planes), n_planes,
                            M, reinterpret_cast<const float*>(decays), m, reinterpret_cast<const int*>(cu_q),
                            reinterpret_cast<const T*>(z->head_norm), reinterpret_cast<T*>(out), ldo) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

template <int MT>
int launch_gl_chunks(const ZseGatedLinear* z, const void* inp, int ld, const void* decays, const void* cu_q, int first, int last,
                     void* o, cudaStream_t st) {
  static size_t done[kMaxDevices] = {};
  const Gl m = gl_of(z);
  auto kern = gl_chunk_kernel<MT>;
  const size_t smem = gl_chunk_smem(m.dim);
  if (int r = raise_smem(kern, smem, done)) return r;
  return launch_pdl(kern, dim3((m.vdim + kGcC - 1) / kGcC, m.heads, last - first), dim3(kGcThreads), smem, st,
                    reinterpret_cast<const bf16*>(inp), ld, reinterpret_cast<const float*>(decays), m,
                    reinterpret_cast<const int*>(cu_q), first, reinterpret_cast<float*>(o)) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

}  // namespace
}  // namespace zse

using namespace zse;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int zse_gated_linear_chunk_ok(int dim, int vdim) {
  return dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 256 && gl_chunk_smem(dim) <= 227 * 1024;
}

extern "C" int zse_gated_linear_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, const void* side,
                                     int side_ld, const ZseGatedLinear* z, void* decays, int M, void* stream) {
  if (M <= 0) return 0;
  if (!gl_shape_ok(z) || ld % 4 || z->q_col % 4 || z->rank_col % 4 || z->rank_col + z->rank > ld) return ZSE_ERR_SHAPE;
  auto run = dtype == kBF16 ? launch_gl_prep<bf16> : launch_gl_prep<float>;
  return run(inp, ld, planes, n_planes, side, side_ld, z, decays, M, ST(stream));
}

extern "C" int zse_gated_linear_tokens(int dtype, const void* inp, int ld, const void* planes, int n_planes, int M,
                                       const void* decays, const ZseGatedLinear* z, const void* cu_q, int S, void* out, int ldo,
                                       void* stream) {
  if (S <= 0) return 0;
  if (!gl_shape_ok(z) || S > 65535 || (decays == nullptr && n_planes <= 0)) return ZSE_ERR_SHAPE;
  const bool vec = z->vdim % 4 == 0 && z->row_floats % 4 == 0 && !(reinterpret_cast<uintptr_t>(z->states) & 15);
  auto run = dtype == kBF16 ? (vec ? launch_gl_tokens<bf16, 4> : launch_gl_tokens<bf16, 1>)
                            : (vec ? launch_gl_tokens<float, 4> : launch_gl_tokens<float, 1>);
  return run(z, inp, ld, planes, n_planes, M, decays, cu_q, S, out, ldo, ST(stream));
}

extern "C" int zse_gated_linear_chunks(const void* inp, int ld, const void* decays, const ZseGatedLinear* z, const void* cu_q,
                                       int first, int last, void* o, int M, int row0, void* out, int ldo, void* stream) {
  if (last <= first) return 0;
  if (!gl_shape_ok(z) || !zse_gated_linear_chunk_ok(z->dim, z->vdim) || ld % 8 || z->q_col % 8 || z->k_col % 8 ||
      z->v_col % 8 || z->gate_col % 8 || z->row_floats % 2 || ldo % 4 || last - first > 65535)
    return ZSE_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(inp) | reinterpret_cast<uintptr_t>(decays) | reinterpret_cast<uintptr_t>(o)) & 15)
    return ZSE_ERR_ALIGN;
  const int rc = z->dim <= 128 ? launch_gl_chunks<1>(z, inp, ld, decays, cu_q, first, last, o, ST(stream))
                               : launch_gl_chunks<2>(z, inp, ld, decays, cu_q, first, last, o, ST(stream));
  if (rc) return rc;
  const Gl m = gl_of(z);
  const long long units = (long long)(M - row0) * m.heads;
  return launch_pdl(gl_out_kernel, dim3(unsigned((units + 7) / 8)), dim3(256), 0, ST(stream), reinterpret_cast<const float*>(o),
                    reinterpret_cast<const bf16*>(inp), ld, m, reinterpret_cast<const bf16*>(z->head_norm),
                    reinterpret_cast<bf16*>(out), ldo, row0, M - row0) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}
