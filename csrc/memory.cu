// Matrix memory (mLSTM): per head S [dim, vdim], key sum n [dim] and running maximum m of the log gates, all fp32.
//
//   m' = max(f + m, i);  S' = exp(f + m - m') S + exp(i - m') k v^T;  n' likewise with k alone
//   o  = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6);  q is projected / sqrt(dim)
//   y  = o / rms(o) * norm * sigmoid(g)
//
//   memory_prep    second half of the fused input projection: split-K sum, logarithms of the gates
//   memory_tokens  token by token (decode, short portions, any shape, any type): a cluster per (head, sequence) whose CTAs
//                  take shares of the columns of S; update, read-out, head norm and output gate in one pass over the state
//   memory_chunks  chunks of 64 tokens (bfloat16): a CTA per (64 columns of S, head, sequence) keeps its part of S in
//                  accumulators and walks through the sequence
//   memory_out     head norm and output gate after memory_chunks
//
// Inside a chunk, with b_t the sum of the f up to t, a_s = i_s - b_s and M_t = max(m_start, max_{s <= t} a_s), the recursion
// gives m_t = b_t + M_t and
//   S_t = exp(m_start - M_t) S_start + sum_{s <= t} exp(a_s - M_t) k_s v_s^T
// so that a chunk is three products: scores q k^T weighted by exp(a_s - M_t) times v, q S_start, and k^T (weighted v) for the
// next state.  Their fp32 factors (weighted scores, S, weighted v) enter as two bfloat16 terms, value and remainder.
//
// State rows come in pairs: a pass reads one row (-1: zero) and writes another, see cache/state_slots.py.
#include "api.h"
#include "typed.cuh"

namespace zse {
namespace {

struct Memory {
  int heads, dim, vdim, k_col, v_col, gate_col, if_col;
  float* states;
  long long row_floats;
  int sum_at, max_at;
  const int* state_rows;
  int state_ld;
  float gate_cap, eps;
};

// ---- prep -----------------------------------------------------------------------------------------------------------
constexpr int kPrepCols = 1024;

__device__ __forceinline__ float log_gate(float z, float cap, bool forget) {
  const float g = cap * tanhf(z / cap);
  return forget ? fminf(g, 0.f) - log1pf(expf(-fabsf(g))) : g;
}

// grid (rows, 1 + pieces): piece 0 takes the gates, the others sum kPrepCols columns each.  Without planes: grid (blocks)
// over all gates.
template <typename T>
__global__ void __launch_bounds__(256)
memory_prep_kernel(T* __restrict__ inp, int ld, const float* __restrict__ planes, int n_planes,
                   const float* __restrict__ gate_planes, int n_gate_planes, const float* __restrict__ bias,
                   float* __restrict__ gates, Memory m, int M) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, g = 2 * m.heads;
  if (n_planes == 0) {
    const int id = blockIdx.x * blockDim.x + threadIdx.x;
    if (id >= M * g) return;
    const int i = id % g;
    float z = bias[i];
    for (int p = 0; p < n_gate_planes; ++p) z += gate_planes[size_t(p) * M * g + id];
    gates[id] = log_gate(z, m.gate_cap, i >= m.heads);
    return;
  }
  if (blockIdx.y == 0) {
    for (int i = threadIdx.x; i < g; i += blockDim.x) {
      float z = bias[i];
      for (int p = 0; p < n_planes; ++p) z += planes[(size_t(p) * M + t) * ld + m.if_col + i];
      gates[size_t(t) * g + i] = log_gate(z, m.gate_cap, i >= m.heads);
    }
    return;
  }
  const int c = (blockIdx.y - 1) * kPrepCols + threadIdx.x * 4;    // ld and if_col are multiples of 8
  if (c >= m.if_col) return;
  F32Vec<4> x{};
#pragma unroll 4
  for (int p = 0; p < n_planes; ++p) {
    const F32Vec<4> y = load_vec<4>(planes + (size_t(p) * M + t) * ld + c);
#pragma unroll
    for (int e = 0; e < 4; ++e) x.v[e] += y.v[e];
  }
  store_vec<4>(inp + size_t(t) * ld + c, x);
}

// ---- token by token ----------------------------------------------------------------------------------------------------
constexpr int kTokThreads = 256, kTokBatch = 8;

__device__ __forceinline__ float tok_sum(float v, float* red) {    // over the CTA; two barriers
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = warp_sum((threadIdx.x & 31) < kTokThreads / 32 ? red[threadIdx.x & 31] : 0.f);
  __syncthreads();
  return v;
}

// grid (cluster, heads, sequences)
template <typename T, int VEC>
__global__ void __launch_bounds__(kTokThreads)
memory_tokens_kernel(const T* __restrict__ inp, int ld, const float* __restrict__ gates, Memory m,
                     const int* __restrict__ cu_q, const T* __restrict__ head_norm, T* __restrict__ out, int ldo) {
  extern __shared__ float sm[];                  // q, k, n [dim] each; v, o [columns of this CTA]
  __shared__ float red[kTokThreads / 32];
  __shared__ float part[kTokThreads * VEC];
  __shared__ float cluster_ss;
  pdl_launch_dependents();
  pdl_wait();
  const int cs = gridDim.x, head = blockIdx.y, s = blockIdx.z;
  const int nvec = m.vdim / VEC, share = (nvec + cs - 1) / cs;
  const int c0 = blockIdx.x * share, nc = max(0, min(nvec, c0 + share) - c0);      // column vectors of this CTA
  float* q = sm;
  float* k = q + m.dim;
  float* n = k + m.dim;
  float* v = n + m.dim;
  float* o = v + share * VEC;
  const int first = cu_q != nullptr ? cu_q[s] : s, last = cu_q != nullptr ? cu_q[s + 1] : s + 1;
  const int read = m.state_rows[s], write = m.state_rows[m.state_ld + s];
  const size_t mem_at = size_t(head) * m.dim * m.vdim + size_t(c0) * VEC;
  const float* src = m.states + size_t(max(read, 0)) * m.row_floats;
  float* dst = m.states + size_t(max(write, 0)) * m.row_floats;
  float mx = read >= 0 ? src[m.max_at + head] : 0.f;
  for (int i = threadIdx.x; i < m.dim; i += kTokThreads) n[i] = read >= 0 ? src[m.sum_at + head * m.dim + i] : 0.f;
  int cw = 1;                                    // column vectors side by side
  while (cw * 2 <= nc && cw < 64) cw *= 2;
  const int tc = threadIdx.x % cw, tr = threadIdx.x / cw, rows = kTokThreads / cw;
  const float q_scale = 1.f / sqrtf(float(m.dim));
  const float* from = read >= 0 ? src + mem_at : nullptr;
  for (int t = first; t < last; ++t) {
    const T* in = inp + size_t(t) * ld;
    const float lf = gates[size_t(t) * 2 * m.heads + m.heads + head], li = gates[size_t(t) * 2 * m.heads + head];
    const float mn = fmaxf(lf + mx, li), keep = expf(lf + mx - mn), add = expf(li - mn);
    mx = mn;
    for (int i = threadIdx.x; i < m.dim; i += kTokThreads) {
      q[i] = to_f32(in[head * m.dim + i]) * q_scale;
      k[i] = add * to_f32(in[m.k_col + head * m.dim + i]);
    }
    for (int i = threadIdx.x; i < nc * VEC; i += kTokThreads) v[i] = to_f32(in[m.v_col + head * m.vdim + c0 * VEC + i]);
    float nq = 0.f;
    for (int i = threadIdx.x; i < m.dim; i += kTokThreads) {       // a thread's own entries of q, k and n
      n[i] = keep * n[i] + k[i];
      nq += n[i] * q[i];
    }
    nq = tok_sum(nq, red);                       // q, k, v are in place after its barriers
    const float inv_den = 1.f / (fmaxf(fabsf(nq), expf(-mx)) + 1e-6f);
    float ss = 0.f;
    for (int cb = 0; cb < nc; cb += cw) {
      F32Vec<VEC> acc{};
      if (cb + tc < nc) {
        const int col = (cb + tc) * VEC;
        F32Vec<VEC> vv;
#pragma unroll
        for (int e = 0; e < VEC; ++e) vv.v[e] = v[col + e];
        // a batch of loads is under way before the first store (which might alias the next loads)
        for (int d0 = tr; d0 < m.dim; d0 += rows * kTokBatch) {
          F32Vec<VEC> x[kTokBatch];
#pragma unroll
          for (int u = 0; u < kTokBatch; ++u) {
            const int d = d0 + u * rows;
            x[u] = F32Vec<VEC>{};
            if (from != nullptr && d < m.dim) x[u] = load_vec<VEC>(from + size_t(d) * m.vdim + col);
          }
#pragma unroll
          for (int u = 0; u < kTokBatch; ++u) {
            const int d = d0 + u * rows;
            if (d >= m.dim) break;
            const float kd = k[d], qd = q[d];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
              x[u].v[e] = fmaf(keep, x[u].v[e], kd * vv.v[e]);
              acc.v[e] = fmaf(qd, x[u].v[e], acc.v[e]);
            }
            if (write >= 0) store_vec<VEC>(dst + mem_at + size_t(d) * m.vdim + col, x[u]);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) part[threadIdx.x * VEC + e] = acc.v[e];
      __syncthreads();
      for (int i = threadIdx.x; i < cw * VEC && cb * VEC + i < nc * VEC; i += kTokThreads) {
        float y = 0.f;
        for (int r = 0; r < rows; ++r) y += part[r * cw * VEC + i];
        y *= inv_den;
        o[cb * VEC + i] = y;
        ss += y * y;
      }
      __syncthreads();
    }
    ss = tok_sum(ss, red);
    if (cs > 1) {
      if (threadIdx.x == 0) cluster_ss = ss;
      asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
      ss = 0.f;
      const uint32_t local = smem_u32(&cluster_ss);
      for (int r = 0; r < cs; ++r) {             // same order in every CTA: identical sums
        uint32_t remote;
        float x;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(r));
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(x) : "r"(remote) : "memory");
        ss += x;
      }
      // nobody overwrites its value, or exits, while it may still be read
      asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    }
    const float inv = 1.f / sqrtf(ss / float(m.vdim) + m.eps);
    for (int i = threadIdx.x; i < nc * VEC; i += kTokThreads) {
      const int c = head * m.vdim + c0 * VEC + i;
      const float y = o[i] * inv * to_f32(head_norm[c]) * sigmoid_exact(to_f32(in[m.gate_col + c]));
      out[size_t(t) * ldo + c] = from_f32<T>(y);
    }
    from = dst + mem_at;                         // the next token starts from what this thread has written
    __syncthreads();
  }
  if (write >= 0 && blockIdx.x == 0) {
    for (int i = threadIdx.x; i < m.dim; i += kTokThreads) dst[m.sum_at + head * m.dim + i] = n[i];
    if (threadIdx.x == 0) dst[m.max_at + head] = mx;
  }
}

// ---- chunks of 64 tokens -----------------------------------------------------------------------------------------------
constexpr int kChT = 64;                         // tokens of a chunk
constexpr int kChC = 64;                         // columns of S per CTA
constexpr int kChThreads = 256;
constexpr int kVPitch = (kChC / 8 + 1) * 16;     // bytes of a row of v, and of the weighted scores
constexpr int kSPitch = (kChC / 8 + 3) * 16;     // of a row of S and of the weighted v: 64 columns, the key sum's 8, 8 unused

__host__ __device__ inline int pitch_of(int n) { return ((n + 15) / 16 * 2 + 1) * 16; }
inline size_t memory_chunk_smem(int dim) {
  const int rows = (dim + 15) / 16 * 16;
  return size_t(2) * kChT * pitch_of(dim) + size_t(kChT) * kVPitch * 3 + size_t(2) * kChT * kSPitch +
         size_t(2) * rows * kSPitch + (6 * kChT + 2 * kChT) * 4 + 16;
}

// MT: 16-row tiles of S per warp (8 warps: dim <= 128 * MT).  grid (column blocks, heads, sequences)
template <int MT>
__global__ void __launch_bounds__(kChThreads)
memory_chunk_kernel(const bf16* __restrict__ inp, int ld, const float* __restrict__ gates, Memory m,
                    const int* __restrict__ cu_q, int first, float* __restrict__ o_out, int ldo) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int cb = blockIdx.x * kChC, head = blockIdx.y, s = first + blockIdx.z;
  const int nc = min(kChC, m.vdim - cb);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qp = pitch_of(m.dim), ksteps = (m.dim + 15) / 16, dch = m.dim / 8;
  uint8_t* sq = smem;
  uint8_t* sk = sq + kChT * qp;
  uint8_t* sv = sk + kChT * qp;                  // v
  uint8_t* sph = sv + kChT * kVPitch;            // weighted scores, two terms
  uint8_t* spl = sph + kChT * kVPitch;
  uint8_t* swh = spl + kChT * kVPitch;           // weighted v (and the weights alone in column 64), two terms
  uint8_t* swl = swh + kChT * kSPitch;
  uint8_t* ssh = swl + kChT * kSPitch;           // S at the chunk's start (and the key sum in column 64), two terms
  uint8_t* ssl = ssh + ksteps * 16 * kSPitch;
  float* ga = reinterpret_cast<float*>(ssl + ksteps * 16 * kSPitch);     // a_s
  float* gm = ga + kChT;                         // M_t
  float* gi = gm + kChT;                         // exp(m_start - M_t): weight of the start state
  float* gf = gi + kChT;                         // exp(-m_t): floor of the denominator
  float* gw = gf + kChT;                         // exp(a_s - M_end): weight in the next state
  float* gd = gw + kChT;                         // 1 / denominator
  float* rs = gd + kChT;                         // sums of the weighted scores, two halves of the columns
  float* misc = rs + 2 * kChT;                   // exp(m_start - M_end), new m

  const int begin = cu_q[s], end = cu_q[s + 1];
  const int read = m.state_rows[s], write = m.state_rows[m.state_ld + s];
  const float* src = m.states + size_t(max(read, 0)) * m.row_floats;
  const int r4 = lane >> 2, c2 = (lane & 3) * 2;

  // this warp's part of S: tiles of 16 rows warp * MT + i, 8 blocks of 8 columns, and a block whose column 0 is the key sum
  float S[MT][9][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int n = 0; n < 9; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (warp * MT + i) * 16 + r4 + (e >> 1) * 8, c = n * 8 + c2 + (e & 1);
        float x = 0.f;
        if (read >= 0 && d < m.dim) {
          if (n < 8 && c < nc) x = src[(size_t(head) * m.dim + d) * m.vdim + cb + c];
          if (n == 8 && c == kChC) x = src[m.sum_at + head * m.dim + d];
        }
        S[i][n][e] = x;
      }
  float mx = read >= 0 ? src[m.max_at + head] : 0.f;

  for (int i = threadIdx.x; i < kChT; i += kChThreads) {           // halves of a step that no copy writes
    if (dch < ksteps * 2) {
      *reinterpret_cast<uint4*>(sq + i * qp + dch * 16) = make_uint4(0, 0, 0, 0);
      *reinterpret_cast<uint4*>(sk + i * qp + dch * 16) = make_uint4(0, 0, 0, 0);
    }
    for (int c = 8; c < 11; ++c) {
      *reinterpret_cast<uint4*>(swh + i * kSPitch + c * 16) = make_uint4(0, 0, 0, 0);
      *reinterpret_cast<uint4*>(swl + i * kSPitch + c * 16) = make_uint4(0, 0, 0, 0);
    }
  }
  for (int i = threadIdx.x; i < ksteps * 16; i += kChThreads)
    for (int c = 8; c < 11; ++c) {
      *reinterpret_cast<uint4*>(ssh + i * kSPitch + c * 16) = make_uint4(0, 0, 0, 0);
      *reinterpret_cast<uint4*>(ssl + i * kSPitch + c * 16) = make_uint4(0, 0, 0, 0);
    }

  const int pr = warp & 3, pc = warp >> 2;       // 16 tokens and half of the columns in the read-out
  const float q_scale = 1.f / sqrtf(float(m.dim));
  for (int t0 = begin; t0 < end; t0 += kChT) {
    const int len = min(kChT, end - t0);
    for (int i = threadIdx.x; i < kChT * dch; i += kChThreads) {
      const int r = i / dch, c = i % dch;
      uint8_t *qd = sq + r * qp + c * 16, *kd = sk + r * qp + c * 16;
      if (r < len) {
        const bf16* row = inp + size_t(t0 + r) * ld + head * m.dim + c * 8;
        cpa16(qd, row);
        cpa16(kd, row + m.k_col);
      } else {
        *reinterpret_cast<uint4*>(qd) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(kd) = make_uint4(0, 0, 0, 0);
      }
    }
    for (int i = threadIdx.x; i < kChT * (kChC / 8); i += kChThreads) {
      const int r = i / (kChC / 8), c = i % (kChC / 8);
      uint8_t* vd = sv + r * kVPitch + c * 16;
      if (r < len && c * 8 < nc)
        cpa16(vd, inp + size_t(t0 + r) * ld + m.v_col + head * m.vdim + cb + c * 8);
      else
        *reinterpret_cast<uint4*>(vd) = make_uint4(0, 0, 0, 0);
    }
    cpa_commit();
    if (warp == 0) {                             // two tokens a lane; tokens past the end neither decay nor add
      float f[2], a[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = lane * 2 + j;
        const float* g = gates + size_t(t0 + min(t, len - 1)) * 2 * m.heads + head;
        f[j] = t < len ? g[m.heads] : 0.f;
        a[j] = t < len ? g[0] : -INFINITY;
      }
      float b = f[0] + f[1];
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, b, d);
        if (lane >= d) b += x;
      }
      const float b1 = b, b0 = b - f[1];
      a[0] -= b0;
      a[1] -= b1;
      float top = fmaxf(a[0], a[1]);
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, top, d);
        if (lane >= d) top = fmaxf(top, x);
      }
      float before = __shfl_up_sync(0xffffffffu, top, 1);
      if (lane == 0) before = -INFINITY;
      const float M1 = fmaxf(mx, top), M0 = fmaxf(mx, fmaxf(before, a[0]));
      const float Mend = __shfl_sync(0xffffffffu, M1, 31), bend = __shfl_sync(0xffffffffu, b1, 31);
      const float Mt[2] = {M0, M1}, bt[2] = {b0, b1};
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = lane * 2 + j;
        ga[t] = a[j];
        gm[t] = Mt[j];
        gi[t] = expf(mx - Mt[j]);
        gf[t] = expf(-(bt[j] + Mt[j]));
        gw[t] = expf(a[j] - Mend);
      }
      if (lane == 0) {
        misc[0] = expf(mx - Mend);
        misc[1] = bend + Mend;
      }
    }
    // S in two terms
#pragma unroll
    for (int i = 0; i < MT; ++i)
      if ((warp * MT + i) * 16 < m.dim) {
#pragma unroll
        for (int n = 0; n < 9; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int at = ((warp * MT + i) * 16 + r4 + h * 8) * kSPitch + (n * 8 + c2) * 2;
            *reinterpret_cast<uint32_t*>(ssh + at) = pack_bf16(S[i][n][h * 2], S[i][n][h * 2 + 1]);
            *reinterpret_cast<uint32_t*>(ssl + at) = pack_bf16_rest(S[i][n][h * 2], S[i][n][h * 2 + 1]);
          }
      }
    cpa_wait<0>();
    __syncthreads();
    const float keep = misc[0], m_next = misc[1];
    // weighted v in two terms
    for (int i = threadIdx.x; i < kChT * (kChC / 2); i += kChThreads) {
      const int r = i / (kChC / 2), c = i % (kChC / 2);
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + r * kVPitch + c * 4));
      const float w = gw[r];
      *reinterpret_cast<uint32_t*>(swh + r * kSPitch + c * 4) = pack_bf16(w * x.x, w * x.y);
      *reinterpret_cast<uint32_t*>(swl + r * kSPitch + c * 4) = pack_bf16_rest(w * x.x, w * x.y);
    }
    if (threadIdx.x < kChT) {
      *reinterpret_cast<uint32_t*>(swh + threadIdx.x * kSPitch + kChC * 2) = pack_bf16(gw[threadIdx.x], 0.f);
      *reinterpret_cast<uint32_t*>(swl + threadIdx.x * kSPitch + kChC * 2) = pack_bf16_rest(gw[threadIdx.x], 0.f);
    }
    // scores of this warp's 16 tokens against 32 of the chunk's, and q S
    float sc[4][4] = {}, acc[5][4] = {};         // acc[4]: the key sum (pc == 0 only)
    const bool causal = pc * 32 <= pr * 16 + 15;
    const uint32_t q_addr = smem_u32(sq) + (pr * 16 + (lane & 15)) * qp + (lane >> 4) * 16;
    const uint32_t k_addr = smem_u32(sk) + (pc * 32 + (lane >> 4) * 8 + (lane & 7)) * qp + (lane >> 3 & 1) * 16;
    const uint32_t s_row = ((lane >> 3 & 1) * 8 + (lane & 7)) * kSPitch + (lane >> 4) * 16 + pc * 64;
    const uint32_t sh_addr = smem_u32(ssh) + s_row, sl_addr = smem_u32(ssl) + s_row;
    for (int kk = 0; kk < ksteps; ++kk) {
      uint32_t a[4], b[4];
      ldm_x4(q_addr + kk * 32, a);
      if (causal) {
#pragma unroll
        for (int n = 0; n < 4; n += 2) {
          ldm_x4(k_addr + n * 8 * qp + kk * 32, b);
          mma_bf16(sc[n], a, b[0], b[1]);
          mma_bf16(sc[n + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int n = 0; n < 4; n += 2) {
        ldm_x4_t(sh_addr + kk * 16 * kSPitch + n * 16, b);
        mma_bf16(acc[n], a, b[0], b[1]);
        mma_bf16(acc[n + 1], a, b[2], b[3]);
        ldm_x4_t(sl_addr + kk * 16 * kSPitch + n * 16, b);
        mma_bf16(acc[n], a, b[0], b[1]);
        mma_bf16(acc[n + 1], a, b[2], b[3]);
      }
      if (pc == 0) {                             // columns 64..71 (72..79 are zero)
        ldm_x4_t(sh_addr + kk * 16 * kSPitch + 128, b);
        mma_bf16(acc[4], a, b[0], b[1]);
        ldm_x4_t(sl_addr + kk * 16 * kSPitch + 128, b);
        mma_bf16(acc[4], a, b[0], b[1]);
      }
    }
    float sums[2] = {0.f, 0.f};
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = pr * 16 + r4 + h * 8;
      const float Mt = gm[t], wi = gi[t] * q_scale;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int c = pc * 32 + n * 8 + c2;
        const float x = c <= t ? sc[n][h * 2] * q_scale * expf(ga[c] - Mt) : 0.f;
        const float y = c + 1 <= t ? sc[n][h * 2 + 1] * q_scale * expf(ga[c + 1] - Mt) : 0.f;
        sums[h] += x + y;
        *reinterpret_cast<uint32_t*>(sph + t * kVPitch + c * 2) = pack_bf16(x, y);
        *reinterpret_cast<uint32_t*>(spl + t * kVPitch + c * 2) = pack_bf16_rest(x, y);
      }
#pragma unroll
      for (int n = 0; n < 5; ++n) {
        acc[n][h * 2] *= wi;
        acc[n][h * 2 + 1] *= wi;
      }
      sums[h] += __shfl_xor_sync(0xffffffffu, sums[h], 1);
      sums[h] += __shfl_xor_sync(0xffffffffu, sums[h], 2);
      if ((lane & 3) == 0) rs[pc * kChT + t] = sums[h] + (pc == 0 ? acc[4][h * 2] : 0.f);
    }
    __syncthreads();
    if (threadIdx.x < kChT) {
      const float nq = rs[threadIdx.x] + rs[kChT + threadIdx.x];
      gd[threadIdx.x] = 1.f / (fmaxf(fabsf(nq), gf[threadIdx.x]) + 1e-6f);
    }
    // weighted scores times v
    const uint32_t p_row = (pr * 16 + (lane & 15)) * kVPitch + (lane >> 4) * 16;
    const uint32_t v_addr = smem_u32(sv) + ((lane >> 3 & 1) * 8 + (lane & 7)) * kVPitch + (lane >> 4) * 16 + pc * 64;
#pragma unroll
    for (int kk = 0; kk < kChT / 16; ++kk) {
      if (kk <= pr) {
        uint32_t ph[4], pl[4], b[4];
        ldm_x4(smem_u32(sph) + p_row + kk * 32, ph);
        ldm_x4(smem_u32(spl) + p_row + kk * 32, pl);
#pragma unroll
        for (int n = 0; n < 4; n += 2) {
          ldm_x4_t(v_addr + kk * 16 * kVPitch + n * 16, b);
          mma_bf16(acc[n], ph, b[0], b[1]);
          mma_bf16(acc[n], pl, b[0], b[1]);
          mma_bf16(acc[n + 1], ph, b[2], b[3]);
          mma_bf16(acc[n + 1], pl, b[2], b[3]);
        }
      }
    }
    // next state
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int mt = warp * MT + i;
      if (mt * 16 >= m.dim) continue;
#pragma unroll
      for (int n = 0; n < 9; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][n][e] *= keep;
      const uint32_t kt = smem_u32(sk) + ((lane >> 4) * 8 + (lane & 7)) * qp + (mt * 16 + (lane >> 3 & 1) * 8) * 2;
      const uint32_t w_row = ((lane >> 3 & 1) * 8 + (lane & 7)) * kSPitch + (lane >> 4) * 16;
#pragma unroll
      for (int kk = 0; kk < kChT / 16; ++kk) {
        uint32_t a[4], b[4];
        ldm_x4_t(kt + kk * 16 * qp, a);
#pragma unroll
        for (int term = 0; term < 2; ++term) {
          const uint32_t w = smem_u32(term == 0 ? swh : swl) + w_row + kk * 16 * kSPitch;
#pragma unroll
          for (int n = 0; n < 8; n += 2) {
            ldm_x4_t(w + n * 16, b);
            mma_bf16(S[i][n], a, b[0], b[1]);
            mma_bf16(S[i][n + 1], a, b[2], b[3]);
          }
          ldm_x4_t(w + 128, b);
          mma_bf16(S[i][8], a, b[0], b[1]);
        }
      }
    }
    mx = m_next;
    __syncthreads();                             // denominators are there; everyone is done with the chunk's tiles
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = pr * 16 + r4 + h * 8;
      if (t >= len) continue;
      const float inv = gd[t];
      float* o = o_out + size_t(t0 + t) * ldo + head * m.vdim + cb;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int c = pc * 32 + n * 8 + c2;
        if (c < nc) *reinterpret_cast<float2*>(o + c) = make_float2(acc[n][h * 2] * inv, acc[n][h * 2 + 1] * inv);
      }
    }
    __syncthreads();                             // gd is written again by the next chunk
  }
  if (write < 0) return;
  float* dst = m.states + size_t(write) * m.row_floats;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int n = 0; n < 9; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = (warp * MT + i) * 16 + r4 + h * 8, c = n * 8 + c2;
        if (d >= m.dim) continue;
        if (n < 8 && c < nc)
          *reinterpret_cast<float2*>(dst + (size_t(head) * m.dim + d) * m.vdim + cb + c) =
              make_float2(S[i][n][h * 2], S[i][n][h * 2 + 1]);
        if (n == 8 && c == kChC && blockIdx.x == 0) dst[m.sum_at + head * m.dim + d] = S[i][n][h * 2];
      }
  if (blockIdx.x == 0 && threadIdx.x == 0) dst[m.max_at + head] = mx;
}

// A warp per (row, head): y = o / rms(o) * norm * sigmoid(g).
template <int VEC>
__global__ void __launch_bounds__(256)
memory_out_kernel(const float* __restrict__ o, const bf16* __restrict__ inp, int ld, Memory m,
                  const bf16* __restrict__ head_norm, bf16* __restrict__ out, int ldo, int row0, int rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long id = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (id >= (long long)(rows) * m.heads) return;
  const int t = row0 + int(id / m.heads), head = int(id % m.heads), c0 = head * m.vdim;
  const float* src = o + size_t(t) * m.heads * m.vdim + c0;
  float ss = 0.f;
#pragma unroll 4
  for (int i = lane * VEC; i < m.vdim; i += 32 * VEC) {
    const F32Vec<VEC> x = load_vec<VEC>(src + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += x.v[e] * x.v[e];
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / float(m.vdim) + m.eps);
#pragma unroll 4
  for (int i = lane * VEC; i < m.vdim; i += 32 * VEC) {
    F32Vec<VEC> x = load_vec<VEC>(src + i);
    const F32Vec<VEC> w = load_vec<VEC>(head_norm + c0 + i), g = load_vec<VEC>(inp + size_t(t) * ld + m.gate_col + c0 + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x.v[e] *= inv * w.v[e] * sigmoid_exact(g.v[e]);
    store_vec<VEC>(out + size_t(t) * ldo + c0 + i, x);
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

Memory memory_of(const ZseMemory* z) {
  return Memory{z->heads, z->dim, z->vdim, z->k_col, z->v_col, z->gate_col, z->if_col, reinterpret_cast<float*>(z->states),
                (long long)(z->row_floats), z->sum_at, z->max_at, reinterpret_cast<const int*>(z->state_rows), z->state_ld,
                z->gate_cap, z->eps};
}

template <typename T, int VEC>
int launch_tokens(const ZseMemory* z, const void* inp, int ld, const void* gates, const void* cu_q, int S, void* out, int ldo,
                  cudaStream_t st) {
  static size_t done[kMaxDevices] = {};
  const Memory m = memory_of(z);
  auto kern = memory_tokens_kernel<T, VEC>;
  // CTAs of a cluster share a head's columns: enough of them to fill the GPU, at least 32 columns each
  int cs = 1;
  while (cs < 8 && S * m.heads * cs < 2 * 148 && m.vdim / (cs * 2) >= 32) cs *= 2;
  const int share = (m.vdim / VEC + cs - 1) / cs * VEC;
  const size_t smem = (size_t(3) * m.dim + 2 * share) * sizeof(float);
  if (smem > 200 * 1024) return ZSE_ERR_LIMIT;
  if (smem > 40 * 1024)
    if (int r = raise_smem(kern, smem, done)) return r;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(cs, m.heads, S);
  cfg.blockDim = dim3(kTokThreads);
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
  return cudaLaunchKernelEx(&cfg, kern, reinterpret_cast<const T*>(inp), ld, reinterpret_cast<const float*>(gates), m,
                            reinterpret_cast<const int*>(cu_q), reinterpret_cast<const T*>(z->head_norm),
                            reinterpret_cast<T*>(out), ldo) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

template <int MT>
int launch_memory_chunks(const ZseMemory* z, const void* inp, int ld, const void* gates, const void* cu_q, int first, int last,
                         void* o, cudaStream_t st) {
  static size_t done[kMaxDevices] = {};
  const Memory m = memory_of(z);
  auto kern = memory_chunk_kernel<MT>;
  const size_t smem = memory_chunk_smem(m.dim);
  if (int r = raise_smem(kern, smem, done)) return r;
  return launch_pdl(kern, dim3((m.vdim + kChC - 1) / kChC, m.heads, last - first), dim3(kChThreads), smem, st,
                    reinterpret_cast<const bf16*>(inp), ld, reinterpret_cast<const float*>(gates), m,
                    reinterpret_cast<const int*>(cu_q), first, reinterpret_cast<float*>(o), m.heads * m.vdim) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

}  // namespace
}  // namespace zse

using namespace zse;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int zse_memory_chunk_ok(int dim, int vdim) { return dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 256; }

extern "C" int zse_memory_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, const void* gate_planes,
                               int n_gate_planes, const void* if_bias, void* gates, const ZseMemory* z, int M,
                               void* stream) {
  if (M <= 0) return 0;
  if (ld % 8 || z->if_col % 8) return ZSE_ERR_SHAPE;
  const Memory m = memory_of(z);
  const dim3 grid = n_planes > 0 ? dim3(M, 1 + (m.if_col + kPrepCols - 1) / kPrepCols)
                                 : dim3((M * 2 * m.heads + 255) / 256);
  cudaError_t e;
  if (dtype == kBF16)
    e = launch_pdl(memory_prep_kernel<bf16>, grid, dim3(256), 0, ST(stream), reinterpret_cast<bf16*>(inp), ld,
                   reinterpret_cast<const float*>(planes), n_planes, reinterpret_cast<const float*>(gate_planes),
                   n_gate_planes, reinterpret_cast<const float*>(if_bias), reinterpret_cast<float*>(gates), m, M);
  else
    e = launch_pdl(memory_prep_kernel<float>, grid, dim3(256), 0, ST(stream), reinterpret_cast<float*>(inp), ld,
                   reinterpret_cast<const float*>(planes), n_planes, reinterpret_cast<const float*>(gate_planes),
                   n_gate_planes, reinterpret_cast<const float*>(if_bias), reinterpret_cast<float*>(gates), m, M);
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_memory_tokens(int dtype, const void* inp, int ld, const void* gates, const ZseMemory* m, const void* cu_q,
                                 int S, void* out, int ldo, void* stream) {
  if (S <= 0) return 0;
  if (S > 65535 || m->heads > 65535 || m->dim <= 0 || m->vdim <= 0) return ZSE_ERR_SHAPE;
  const bool vec = m->vdim % 4 == 0 && m->row_floats % 4 == 0 && !(reinterpret_cast<uintptr_t>(m->states) & 15);
  auto run = dtype == kBF16 ? (vec ? launch_tokens<bf16, 4> : launch_tokens<bf16, 1>)
                            : (vec ? launch_tokens<float, 4> : launch_tokens<float, 1>);
  return run(m, inp, ld, gates, cu_q, S, out, ldo, ST(stream));
}

extern "C" int zse_memory_chunks(const void* inp, int ld, const void* gates, const ZseMemory* z, const void* cu_q, int first,
                                 int last, void* o, int M, int row0, void* out, int ldo, void* stream) {
  if (last <= first) return 0;
  if (!zse_memory_chunk_ok(z->dim, z->vdim) || ld % 8 || z->row_floats % 2 || ldo % 4 || z->heads > 65535 ||
      last - first > 65535)
    return ZSE_ERR_SHAPE;
  const int rc = z->dim <= 128 ? launch_memory_chunks<1>(z, inp, ld, gates, cu_q, first, last, o, ST(stream))
                               : launch_memory_chunks<2>(z, inp, ld, gates, cu_q, first, last, o, ST(stream));
  if (rc) return rc;
  const Memory m = memory_of(z);
  const long long units = (long long)(M - row0) * m.heads;
  return launch_pdl(memory_out_kernel<4>, dim3(unsigned((units + 7) / 8)), dim3(256), 0, ST(stream),
                    reinterpret_cast<const float*>(o), reinterpret_cast<const bf16*>(inp), ld, m,
                    reinterpret_cast<const bf16*>(z->head_norm), reinterpret_cast<bf16*>(out), ldo, row0, M - row0) ==
                 cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}
