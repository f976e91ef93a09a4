// State space (Mamba-2): per head S [state, vdim] in fp32,
//
//   S' = exp(neg_a dt) S + dt B x^T;  y = S'^T C + D x;  y *= silu(z)
//
// with x, B and C out of a causal convolution per channel and silu, dt = softplus(projected + bias) and neg_a = -exp(A_log) per
// head; heads of a group share B and C.  The gated result is RMS-normed in equal parts (group_norm).
//
//   ss_prep     second half of the fused input projection [z | x | B | C | dt]: split-K sum, convolution, step sizes
//   ss_tokens   token by token (decode, short portions, any shape, any type): a CTA per (columns of S, head, sequence) keeps
//               its part of S in registers
//   ss_chunk    chunks of 64 tokens (bfloat16): a CTA per (64 columns of S, head, sequence) keeps its part of S in accumulators
//               and walks through the sequence
//   group_norm  norm in parts and weight, in place
//
// Inside a chunk, with b_t the sum of neg_a dt up to t,
//   y_t = exp(b_t) S_start^T C_t + sum_{s <= t} exp(b_t - b_s) dt_s (C_t . B_s) x_s
//   S_end = exp(b_end) S_start + sum_s exp(b_end - b_s) dt_s B_s x_s^T
// are four products, and no exponent is positive.  Their fp32 factors (S, the weighted scores, the weighted x) enter as two
// bfloat16 terms, value and remainder.
//
// State rows come in pairs: a pass reads one row (-1: zero) and writes another, see cache/state_slots.py.  A row holds S and,
// from conv_at on, the last taps - 1 inputs of the convolution, the oldest first.
#include "api.h"
#include "typed.cuh"

namespace zse {
namespace {

struct Space {
  int heads, vdim, state, groups, taps, x_col, b_at, c_at, conv_width, dt_col;
  float* states;
  long long row_floats;
  int conv_at;
  const int* state_rows;
  int state_ld;
};

// ---- prep -----------------------------------------------------------------------------------------------------------
constexpr int kSpPrepThreads = 256, kSpPrepCols = kSpPrepThreads * 4;

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

struct SpPrep {
  int ld, n_planes, M, rows;            // rows: of a thread
  const float *planes, *side;           // side: fp32 step sizes [M][side_ld], or null: those of inp
  int side_ld, z_pieces, conv_pieces;
  const int *row_seq, *cu_q;
  const float *conv_w, *conv_b, *dt_bias;
  float* dt;
};

// grid (blocks of rows, pieces of columns): z (with planes only), the channels, the step sizes.  TAPS 0: any number of taps.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kSpPrepThreads)
ss_prep_kernel(T* __restrict__ inp, T* __restrict__ xbc, const Space m, const SpPrep a) {
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * a.rows, t1 = min(a.M, t0 + a.rows);
  const size_t plane = size_t(a.M) * a.ld;
  auto raw = [&](int t, int c) {
    if (a.n_planes == 0) return load_vec<4>(inp + size_t(t) * a.ld + c);
    F32Vec<4> x{};
#pragma unroll 4
    for (int p = 0; p < a.n_planes; ++p) {
      const F32Vec<4> y = load_vec<4>(a.planes + p * plane + size_t(t) * a.ld + c);
#pragma unroll
      for (int e = 0; e < 4; ++e) x.v[e] += y.v[e];
    }
    return x;
  };
  int piece = blockIdx.y;
  if (piece < a.z_pieces) {
    const int c = piece * kSpPrepCols + threadIdx.x * 4;
    if (c < m.x_col)
      for (int t = t0; t < t1; ++t) store_vec<4>(inp + size_t(t) * a.ld + c, raw(t, c));
    return;
  }
  piece -= a.z_pieces;
  if (piece == a.conv_pieces) {                  // step sizes
    for (int i = threadIdx.x; i < (t1 - t0) * m.heads; i += kSpPrepThreads) {
      const int t = t0 + i / m.heads, h = i % m.heads;
      float z = a.dt_bias[h];
      if (a.n_planes > 0) {
        for (int p = 0; p < a.n_planes; ++p) z += a.planes[p * plane + size_t(t) * a.ld + m.dt_col + h];
      } else {
        z += a.side != nullptr ? a.side[size_t(t) * a.side_ld + h] : to_f32(inp[size_t(t) * a.ld + m.dt_col + h]);
      }
      a.dt[size_t(t) * m.heads + h] = softplus(z);
    }
    return;
  }
  const int c = piece * kSpPrepCols + threadIdx.x * 4;
  if (c >= m.conv_width) return;
  const int taps = TAPS > 0 ? TAPS : m.taps, col = m.x_col + c;
  constexpr int kWin = TAPS > 1 ? TAPS - 1 : 1;
  F32Vec<4> w[TAPS > 0 ? TAPS : 1], win[kWin];
  const F32Vec<4> bias = load_vec<4>(a.conv_b + c);
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = load_vec<4>(a.conv_w + size_t(j) * m.conv_width + c);
  }
  int s = 0, begin = 0, end = -1, read = -1, write = -1;
  // the input `back` rows before row t (back < taps): of this pass, of the state, or zero
  auto before = [&](int t, int back) {
    if (t - back >= begin) return raw(t - back, col);
    if (read < 0) return F32Vec<4>{};
    return load_vec<4>(m.states + size_t(read) * m.row_floats + m.conv_at +
                       size_t(taps - 1 + t - back - begin) * m.conv_width + c);
  };
  constexpr int kAhead = 4;                      // rows whose loads are under way together
  for (int tb = t0; tb < t1; tb += kAhead) {
    F32Vec<4> rows_in[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (tb + j < t1) rows_in[j] = raw(tb + j, col);
#pragma unroll
    for (int jr = 0; jr < kAhead; ++jr) {
      const int t = tb + jr;
      if (t >= t1) break;
      if (t >= end) {                              // the block's first row, or a sequence's
        s = a.row_seq != nullptr ? a.row_seq[t] : t;
        begin = a.cu_q != nullptr ? a.cu_q[s] : t;
        end = a.cu_q != nullptr ? a.cu_q[s + 1] : t + 1;
        read = m.state_rows[s];
        write = m.state_rows[m.state_ld + s];
        if constexpr (TAPS > 1) {
#pragma unroll
          for (int j = 0; j < TAPS - 1; ++j) win[j] = before(t, TAPS - 1 - j);
        }
      }
      float* last = write >= 0 ? m.states + size_t(write) * m.row_floats + m.conv_at + c : nullptr;
      if (last != nullptr && t == begin && end - begin < taps - 1)   // what stays of the inputs before a short portion
        for (int j = 0; j + end - begin < taps - 1; ++j)
          store_vec<4>(last + size_t(j) * m.conv_width, before(t, taps - 1 - j - (end - begin)));
      const F32Vec<4> x = rows_in[jr];
      F32Vec<4> y = bias;
      if constexpr (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) y.v[e] = fmaf(w[j].v[e], win[j].v[e], y.v[e]);
#pragma unroll
        for (int e = 0; e < 4; ++e) y.v[e] = fmaf(w[TAPS - 1].v[e], x.v[e], y.v[e]);
        if constexpr (TAPS > 1) {
#pragma unroll
          for (int j = 0; j + 1 < TAPS - 1; ++j) win[j] = win[j + 1];
          win[TAPS - 2] = x;
        }
      } else {
        for (int j = 0; j < taps; ++j) {
          const F32Vec<4> f = load_vec<4>(a.conv_w + size_t(j) * m.conv_width + c);
          const F32Vec<4> v = j + 1 == taps ? x : before(t, taps - 1 - j);
#pragma unroll
          for (int e = 0; e < 4; ++e) y.v[e] = fmaf(f.v[e], v.v[e], y.v[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) y.v[e] = sizeof(T) == 2 ? y.v[e] * sigmoid_fast(y.v[e]) : silu_exact(y.v[e]);
      store_vec<4>(xbc + size_t(t) * m.conv_width + c, y);
      const int place = t - (end - (taps - 1));
      if (last != nullptr && place >= 0) store_vec<4>(last + size_t(place) * m.conv_width, x);
    }
  }
}

// ---- token by token ----------------------------------------------------------------------------------------------------
constexpr int kSpTokThreads = 256, kSpTokRows = 8;       // rows of S that a thread keeps

// grid (columns / (cw * VEC), heads, sequences); cw: column vectors side by side, a power of two up to 32
template <typename T, int VEC>
__global__ void __launch_bounds__(kSpTokThreads, 3)
ss_tokens_kernel(const T* __restrict__ inp, int ld, const T* __restrict__ xbc, const float* __restrict__ dt,
                 const Space m, const float* __restrict__ neg_a, const float* __restrict__ skip, const int* __restrict__ cu_q,
                 T* __restrict__ out, int ldo, int cw) {
  extern __shared__ float sm[];                  // B, C [state] each
  __shared__ float part[kSpTokThreads / 32][32 * VEC];
  __shared__ float sx[32 * VEC];
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.y, s = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = blockIdx.x * cw * VEC, nc = min(cw * VEC, m.vdim - c0);
  const int tc = threadIdx.x % cw, tr = threadIdx.x / cw, rows = kSpTokThreads / cw, col = tc * VEC;
  const int g = head / (m.heads / m.groups);
  float *B = sm, *C = sm + m.state;
  const int first = cu_q != nullptr ? cu_q[s] : s, last = cu_q != nullptr ? cu_q[s + 1] : s + 1;
  const int read = m.state_rows[s], write = m.state_rows[m.state_ld + s];
  const size_t at = size_t(head) * m.state * m.vdim + c0 + col;
  F32Vec<VEC> S[kSpTokRows];
#pragma unroll
  for (int u = 0; u < kSpTokRows; ++u) {
    const int d = tr + u * rows;
    S[u] = F32Vec<VEC>{};
    if (read >= 0 && d < m.state && col < nc)
      S[u] = load_vec<VEC>(m.states + size_t(read) * m.row_floats + at + size_t(d) * m.vdim);
  }
  const float na = neg_a[head], D = skip[head];
  for (int t = first; t < last; ++t) {
    const T* row = xbc + size_t(t) * m.conv_width;
    const float step = dt[size_t(t) * m.heads + head], keep = expf(na * step);
    for (int i = threadIdx.x; i < m.state; i += kSpTokThreads) {
      B[i] = step * to_f32(row[m.b_at + g * m.state + i]);
      C[i] = to_f32(row[m.c_at + g * m.state + i]);
    }
    for (int i = threadIdx.x; i < cw * VEC; i += kSpTokThreads)
      sx[i] = i < nc ? to_f32(row[head * m.vdim + c0 + i]) : 0.f;
    __syncthreads();
    F32Vec<VEC> acc{}, x;
#pragma unroll
    for (int e = 0; e < VEC; ++e) x.v[e] = sx[col + e];
#pragma unroll
    for (int u = 0; u < kSpTokRows; ++u) {
      const int d = tr + u * rows;
      if (d >= m.state) break;
      const float b = B[d], c = C[d];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        S[u].v[e] = fmaf(keep, S[u].v[e], b * x.v[e]);
        acc.v[e] = fmaf(c, S[u].v[e], acc.v[e]);
      }
    }
    for (int o = cw; o < 32; o <<= 1)
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc.v[e] += __shfl_xor_sync(0xffffffffu, acc.v[e], o);
    if (lane < cw)
#pragma unroll
      for (int e = 0; e < VEC; ++e) part[warp][col + e] = acc.v[e];
    __syncthreads();
    for (int i = threadIdx.x; i < nc; i += kSpTokThreads) {
      float y = D * sx[i];
#pragma unroll
      for (int w = 0; w < kSpTokThreads / 32; ++w) y += part[w][i];
      const int c = head * m.vdim + c0 + i;
      out[size_t(t) * ldo + c] = from_f32<T>(y * silu_exact(to_f32(inp[size_t(t) * ld + c])));
    }
    if (t + 1 < last) __syncthreads();           // x of this token has been read
  }
  if (write < 0 || col >= nc) return;
#pragma unroll
  for (int u = 0; u < kSpTokRows; ++u) {
    const int d = tr + u * rows;
    if (d < m.state) store_vec<VEC>(m.states + size_t(write) * m.row_floats + at + size_t(d) * m.vdim, S[u]);
  }
}

// ---- chunks of 64 tokens -----------------------------------------------------------------------------------------------
constexpr int kCkT = 64, kCkC = 64, kCkThreads = 256;    // tokens, columns of S per CTA
constexpr int kCkPitch = (kCkC / 8 + 1) * 16;            // bytes of a row of 64 columns

__host__ __device__ inline int pitch_of(int n) { return ((n + 15) / 16 * 2 + 1) * 16; }
__host__ __device__ inline int overlay_bytes(int state) {        // S in two terms, later the weighted scores in two terms
  const int rows = (state + 15) / 16 * 16;
  return 2 * kCkPitch * (rows > kCkT ? rows : kCkT);
}
inline size_t ss_chunk_smem(int state) {
  return size_t(2) * kCkT * pitch_of(state) + size_t(4) * kCkT * kCkPitch + overlay_bytes(state) + (4 * kCkT + 4) * 4;
}

// MT: 16-row tiles of S per warp (8 warps: state <= 128 * MT).  grid (column blocks, heads, sequences)
template <int MT>
__global__ void __launch_bounds__(kCkThreads, MT == 1 ? 2 : 1)
ss_chunk_kernel(const bf16* __restrict__ inp, int ld, const bf16* __restrict__ xbc, const float* __restrict__ dt, const Space m,
                const float* __restrict__ neg_a, const float* __restrict__ skip, const int* __restrict__ cu_q, int first,
                bf16* __restrict__ out, int ldo) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int cb = blockIdx.x * kCkC, head = blockIdx.y, s = first + blockIdx.z, N = m.state;
  const int nc = min(kCkC, m.vdim - cb), g = head / (m.heads / m.groups);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qp = pitch_of(N), ksteps = (N + 15) / 16, dch = N / 8;
  uint8_t* sc_ = smem;                           // C
  uint8_t* sb = sc_ + kCkT * qp;                 // B
  uint8_t* sx = sb + kCkT * qp;                  // x
  uint8_t* sz = sx + kCkT * kCkPitch;            // z
  uint8_t* swh = sz + kCkT * kCkPitch;           // weighted x, two terms
  uint8_t* swl = swh + kCkT * kCkPitch;
  uint8_t* ssh = swl + kCkT * kCkPitch;          // S at the chunk's start, two terms
  uint8_t* ssl = ssh + ksteps * 16 * kCkPitch;
  uint8_t* sph = ssh;                            // in the same place: weighted scores, two terms
  uint8_t* spl = sph + kCkT * kCkPitch;
  float* gb = reinterpret_cast<float*>(ssh + overlay_bytes(N));    // b_t, in units of ln 2
  float* gd = gb + kCkT;                         // dt_t
  float* ge = gd + kCkT;                         // exp(b_t)
  float* gw = ge + kCkT;                         // exp(b_end - b_t) dt_t
  float* misc = gw + kCkT;                       // exp(b_end)

  const int begin = cu_q[s], end = cu_q[s + 1];
  const int read = m.state_rows[s], write = m.state_rows[m.state_ld + s];
  const float* src = m.states + size_t(max(read, 0)) * m.row_floats + size_t(head) * N * m.vdim + cb;
  const int r4 = lane >> 2, c2 = (lane & 3) * 2;
  const float na = neg_a[head], D = skip[head];

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
  if (dch < ksteps * 2)                          // halves of a step that no copy writes
    for (int i = threadIdx.x; i < 2 * kCkT; i += kCkThreads)
      *reinterpret_cast<uint4*>(sc_ + i * qp + dch * 16) = make_uint4(0, 0, 0, 0);

  const int pr = warp & 3, pc = warp >> 2;       // 16 tokens and half of the columns in the read-out
  for (int t0 = begin; t0 < end; t0 += kCkT) {
    const int len = min(kCkT, end - t0);
    for (int i = threadIdx.x; i < kCkT * dch; i += kCkThreads) {
      const int r = i / dch, c = i % dch;
      uint8_t *cd = sc_ + r * qp + c * 16, *bd = sb + r * qp + c * 16;
      if (r < len) {
        const bf16* row = xbc + size_t(t0 + r) * m.conv_width + g * N + c * 8;
        cpa16(cd, row + m.c_at);
        cpa16(bd, row + m.b_at);
      } else {
        *reinterpret_cast<uint4*>(cd) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(bd) = make_uint4(0, 0, 0, 0);
      }
    }
    for (int i = threadIdx.x; i < kCkT * (kCkC / 8); i += kCkThreads) {
      const int r = i / (kCkC / 8), c = i % (kCkC / 8);
      uint8_t *xd = sx + r * kCkPitch + c * 16, *zd = sz + r * kCkPitch + c * 16;
      if (r < len && c * 8 < nc) {
        cpa16(xd, xbc + size_t(t0 + r) * m.conv_width + head * m.vdim + cb + c * 8);
        cpa16(zd, inp + size_t(t0 + r) * ld + head * m.vdim + cb + c * 8);
      } else {
        *reinterpret_cast<uint4*>(xd) = make_uint4(0, 0, 0, 0);
      }
    }
    cpa_commit();
    if (warp == 0) {                             // two tokens a lane; tokens past the end neither decay nor add
      float d[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = lane * 2 + j;
        d[j] = t < len ? dt[size_t(t0 + t) * m.heads + head] : 0.f;
      }
      float b = na * d[0] + na * d[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, b, o);
        if (lane >= o) b += x;
      }
      const float bend = __shfl_sync(0xffffffffu, b, 31), bt[2] = {b - na * d[1], b};
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = lane * 2 + j;
        gb[t] = bt[j] * kLog2E;
        gd[t] = d[j];
        ge[t] = expf(bt[j]);
        gw[t] = expf(bend - bt[j]) * d[j];
      }
      if (lane == 0) misc[0] = expf(bend);
    }
    // S in two terms
#pragma unroll
    for (int i = 0; i < MT; ++i)
      if ((warp * MT + i) * 16 < N) {
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int at = ((warp * MT + i) * 16 + r4 + h * 8) * kCkPitch + (n * 8 + c2) * 2;
            *reinterpret_cast<uint32_t*>(ssh + at) = pack_bf16(S[i][n][h * 2], S[i][n][h * 2 + 1]);
            *reinterpret_cast<uint32_t*>(ssl + at) = pack_bf16_rest(S[i][n][h * 2], S[i][n][h * 2 + 1]);
          }
      }
    cpa_wait<0>();
    __syncthreads();
    // weighted x in two terms
    for (int i = threadIdx.x; i < kCkT * (kCkC / 2); i += kCkThreads) {
      const int r = i / (kCkC / 2), c = i % (kCkC / 2);
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sx + r * kCkPitch + c * 4));
      const float w = gw[r];
      *reinterpret_cast<uint32_t*>(swh + r * kCkPitch + c * 4) = pack_bf16(w * x.x, w * x.y);
      *reinterpret_cast<uint32_t*>(swl + r * kCkPitch + c * 4) = pack_bf16_rest(w * x.x, w * x.y);
    }
    // scores of this warp's 16 tokens against 32 of the chunk's, and C S
    float sc[4][4] = {}, acc[4][4] = {};
    const bool causal = pc * 32 <= pr * 16 + 15;
    const uint32_t q_addr = smem_u32(sc_) + (pr * 16 + (lane & 15)) * qp + (lane >> 4) * 16;
    const uint32_t k_addr = smem_u32(sb) + (pc * 32 + (lane >> 4) * 8 + (lane & 7)) * qp + (lane >> 3 & 1) * 16;
    const uint32_t s_row = ((lane >> 3 & 1) * 8 + (lane & 7)) * kCkPitch + (lane >> 4) * 16 + pc * 64;
    const uint32_t sh_addr = smem_u32(ssh) + s_row, sl_addr = smem_u32(ssl) + s_row;
#pragma unroll 2
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
        ldm_x4_t(sh_addr + kk * 16 * kCkPitch + n * 16, b);
        mma_bf16(acc[n], a, b[0], b[1]);
        mma_bf16(acc[n + 1], a, b[2], b[3]);
        ldm_x4_t(sl_addr + kk * 16 * kCkPitch + n * 16, b);
        mma_bf16(acc[n], a, b[0], b[1]);
        mma_bf16(acc[n + 1], a, b[2], b[3]);
      }
    }
    const float keep = misc[0];
    __syncthreads();                             // S has been read: the weighted scores take its place
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = pr * 16 + r4 + h * 8;
      const float bt = gb[t], wi = ge[t];
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int c = pc * 32 + n * 8 + c2;
        const float x = c <= t ? sc[n][h * 2] * gd[c] * ex2(bt - gb[c]) : 0.f;
        const float y = c + 1 <= t ? sc[n][h * 2 + 1] * gd[c + 1] * ex2(bt - gb[c + 1]) : 0.f;
        *reinterpret_cast<uint32_t*>(sph + t * kCkPitch + c * 2) = pack_bf16(x, y);
        *reinterpret_cast<uint32_t*>(spl + t * kCkPitch + c * 2) = pack_bf16_rest(x, y);
        acc[n][h * 2] *= wi;
        acc[n][h * 2 + 1] *= wi;
      }
    }
    __syncthreads();
    // weighted scores times x
    const uint32_t p_row = (pr * 16 + (lane & 15)) * kCkPitch + (lane >> 4) * 16;
    const uint32_t v_addr = smem_u32(sx) + ((lane >> 3 & 1) * 8 + (lane & 7)) * kCkPitch + (lane >> 4) * 16 + pc * 64;
#pragma unroll
    for (int kk = 0; kk < kCkT / 16; ++kk) {
      if (kk <= pr) {
        uint32_t ph[4], pl[4], b[4];
        ldm_x4(smem_u32(sph) + p_row + kk * 32, ph);
        ldm_x4(smem_u32(spl) + p_row + kk * 32, pl);
#pragma unroll
        for (int n = 0; n < 4; n += 2) {
          ldm_x4_t(v_addr + kk * 16 * kCkPitch + n * 16, b);
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
      if (mt * 16 >= N) continue;
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][n][e] *= keep;
      const uint32_t kt = smem_u32(sb) + ((lane >> 4) * 8 + (lane & 7)) * qp + (mt * 16 + (lane >> 3 & 1) * 8) * 2;
      const uint32_t w_row = ((lane >> 3 & 1) * 8 + (lane & 7)) * kCkPitch + (lane >> 4) * 16;
#pragma unroll
      for (int kk = 0; kk < kCkT / 16; ++kk) {
        uint32_t a[4], b[4];
        ldm_x4_t(kt + kk * 16 * qp, a);
#pragma unroll
        for (int term = 0; term < 2; ++term) {
          const uint32_t w = smem_u32(term == 0 ? swh : swl) + w_row + kk * 16 * kCkPitch;
#pragma unroll
          for (int n = 0; n < 8; n += 2) {
            ldm_x4_t(w + n * 16, b);
            mma_bf16(S[i][n], a, b[0], b[1]);
            mma_bf16(S[i][n + 1], a, b[2], b[3]);
          }
        }
      }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = pr * 16 + r4 + h * 8;
      if (t >= len) continue;
      bf16* o = out + size_t(t0 + t) * ldo + head * m.vdim + cb;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int c = pc * 32 + n * 8 + c2;
        if (c >= nc) continue;
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sx + t * kCkPitch + c * 2));
        const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sz + t * kCkPitch + c * 2));
        *reinterpret_cast<uint32_t*>(o + c) = pack_bf16(fmaf(D, x.x, acc[n][h * 2]) * (z.x * sigmoid_fast(z.x)),
                                                        fmaf(D, x.y, acc[n][h * 2 + 1]) * (z.y * sigmoid_fast(z.y)));
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

// ---- norm in parts -----------------------------------------------------------------------------------------------------
constexpr int kGnRegs = 8;

// grid (parts, rows)
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
group_norm_kernel(T* __restrict__ x, int ld, int width, const T* __restrict__ weight, float eps) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  T* row = x + size_t(blockIdx.y) * ld + size_t(blockIdx.x) * width;
  const T* w = weight + size_t(blockIdx.x) * width;
  const int step = blockDim.x * VEC, far = kGnRegs * step;
  F32Vec<VEC> v[kGnRegs];
  float ss = 0.f;
  auto add = [&](const F32Vec<VEC>& y) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += y.v[e] * y.v[e];
  };
#pragma unroll
  for (int j = 0; j < kGnRegs; ++j) {
    const int i = threadIdx.x * VEC + j * step;
    if (i < width) add(v[j] = load_vec<VEC>(row + i));
  }
  for (int i = far + threadIdx.x * VEC; i < width; i += step) add(load_vec<VEC>(row + i));
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = warp_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f);
  const float inv = 1.f / sqrtf(ss / float(width) + eps);
  auto put = [&](int i, const F32Vec<VEC>& y) {
    F32Vec<VEC> f = load_vec<VEC>(w + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) f.v[e] *= y.v[e] * inv;
    store_vec<VEC>(row + i, f);
  };
#pragma unroll
  for (int j = 0; j < kGnRegs; ++j) {
    const int i = threadIdx.x * VEC + j * step;
    if (i < width) put(i, v[j]);
  }
  for (int i = far + threadIdx.x * VEC; i < width; i += step) put(i, load_vec<VEC>(row + i));
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

Space space_of(const ZseSpace* z) {
  return Space{z->heads, z->vdim, z->state, z->groups, z->taps, z->x_col, z->b_at, z->c_at, z->conv_width, z->dt_col,
               reinterpret_cast<float*>(z->states), (long long)(z->row_floats), z->conv_at,
               reinterpret_cast<const int*>(z->state_rows), z->state_ld};
}

template <typename T, int TAPS>
int launch_space_prep(void* inp, void* xbc, const Space& m, const SpPrep& a, cudaStream_t st) {
  const dim3 grid((a.M + a.rows - 1) / a.rows, a.z_pieces + a.conv_pieces + 1);
  return launch_pdl(ss_prep_kernel<T, TAPS>, grid, dim3(kSpPrepThreads), 0, st, reinterpret_cast<T*>(inp),
                    reinterpret_cast<T*>(xbc), m, a) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}
template <typename T>
int launch_space_prep_t(void* inp, void* xbc, const Space& m, const SpPrep& a, cudaStream_t st) {
  auto run = m.taps == 2   ? launch_space_prep<T, 2>
             : m.taps == 3 ? launch_space_prep<T, 3>
             : m.taps == 4 ? launch_space_prep<T, 4>
                           : launch_space_prep<T, 0>;
  return run(inp, xbc, m, a, st);
}

template <typename T, int VEC>
int launch_space_tokens(const ZseSpace* z, const void* inp, int ld, const void* xbc, const void* dt, const void* cu_q, int S,
                        void* out, int ldo, cudaStream_t st) {
  const Space m = space_of(z);
  const int nvec = (m.vdim + VEC - 1) / VEC;
  int cw = 1;
  while (cw < 32 && cw < nvec && m.state * cw * 2 <= kSpTokRows * kSpTokThreads) cw *= 2;
  while (cw > 4 && S * m.heads * ((nvec + cw - 1) / cw) < 2 * 148) cw /= 2;
  const size_t smem = size_t(2) * m.state * sizeof(float);
  return launch_pdl(ss_tokens_kernel<T, VEC>, dim3((nvec + cw - 1) / cw, m.heads, S), dim3(kSpTokThreads), smem, st,
                    reinterpret_cast<const T*>(inp), ld, reinterpret_cast<const T*>(xbc), reinterpret_cast<const float*>(dt),
                    m, reinterpret_cast<const float*>(z->neg_a), reinterpret_cast<const float*>(z->skip),
                    reinterpret_cast<const int*>(cu_q), reinterpret_cast<T*>(out), ldo, cw) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

template <int MT>
int launch_space_chunks(const ZseSpace* z, const void* inp, int ld, const void* xbc, const void* dt, const void* cu_q,
                        int first, int last, void* out, int ldo, cudaStream_t st) {
  static size_t done[kMaxDevices] = {};
  const Space m = space_of(z);
  auto kern = ss_chunk_kernel<MT>;
  const size_t smem = ss_chunk_smem(m.state);
  if (int r = raise_smem(kern, smem, done)) return r;
  return launch_pdl(kern, dim3((m.vdim + kCkC - 1) / kCkC, m.heads, last - first), dim3(kCkThreads), smem, st,
                    reinterpret_cast<const bf16*>(inp), ld, reinterpret_cast<const bf16*>(xbc),
                    reinterpret_cast<const float*>(dt), m, reinterpret_cast<const float*>(z->neg_a),
                    reinterpret_cast<const float*>(z->skip), reinterpret_cast<const int*>(cu_q), first,
                    reinterpret_cast<bf16*>(out), ldo) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

template <typename T>
cudaError_t launch_group_norm(void* x, int ld, int M, int parts, int width, const void* weight, float eps, cudaStream_t st) {
  const bool vec = width % 4 == 0 && ld % 4 == 0 &&
                   !((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(weight)) & 15);
  const int n = vec ? width / 4 : width;
  const dim3 block(min(256, (n + 31) / 32 * 32));
  return launch_pdl(vec ? group_norm_kernel<T, 4> : group_norm_kernel<T, 1>, dim3(parts, M), block, 0, st,
                    reinterpret_cast<T*>(x), ld, width, reinterpret_cast<const T*>(weight), eps);
}

bool space_shape_ok(const ZseSpace* z) {
  return z->heads > 0 && z->heads <= 65535 && z->groups > 0 && z->heads % z->groups == 0 && z->vdim > 0 && z->state > 0 &&
         z->taps > 0 && z->x_col % 4 == 0 && z->conv_width % 4 == 0 && z->conv_at % 4 == 0 && z->row_floats % 4 == 0;
}

}  // namespace
}  // namespace zse

using namespace zse;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int zse_space_chunk_ok(int state, int vdim) {
  return state > 0 && vdim > 0 && state % 8 == 0 && vdim % 8 == 0 && state <= 256 && ss_chunk_smem(state) <= 227 * 1024;
}

extern "C" int zse_space_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, const void* side, int side_ld,
                              const ZseSpace* z, const void* row_seq, const void* cu_q, void* xbc, void* dt, int M,
                              void* stream) {
  if (M <= 0) return 0;
  if (!space_shape_ok(z) || ld % 4 || z->dt_col + z->heads > ld) return ZSE_ERR_SHAPE;
  const Space m = space_of(z);
  const int rows = M >= 4096 ? 16 : M >= 512 ? 4 : 1;
  const int pieces = (m.conv_width + kSpPrepCols - 1) / kSpPrepCols;
  const SpPrep a{ld, n_planes, M, rows, reinterpret_cast<const float*>(planes), reinterpret_cast<const float*>(side), side_ld,
                 n_planes > 0 ? (m.x_col + kSpPrepCols - 1) / kSpPrepCols : 0, pieces, reinterpret_cast<const int*>(row_seq),
                 reinterpret_cast<const int*>(cu_q), reinterpret_cast<const float*>(z->conv_w),
                 reinterpret_cast<const float*>(z->conv_b), reinterpret_cast<const float*>(z->dt_bias),
                 reinterpret_cast<float*>(dt)};
  return dtype == kBF16 ? launch_space_prep_t<bf16>(inp, xbc, m, a, ST(stream))
                        : launch_space_prep_t<float>(inp, xbc, m, a, ST(stream));
}

extern "C" int zse_space_tokens(int dtype, const void* inp, int ld, const void* xbc, const void* dt, const ZseSpace* z,
                                const void* cu_q, int S, void* out, int ldo, void* stream) {
  if (S <= 0) return 0;
  if (!space_shape_ok(z) || S > 65535) return ZSE_ERR_SHAPE;
  if (z->state > kSpTokRows * kSpTokThreads) return ZSE_ERR_LIMIT;
  const bool vec = z->vdim % 4 == 0 && !(reinterpret_cast<uintptr_t>(z->states) & 15);
  auto run = dtype == kBF16 ? (vec ? launch_space_tokens<bf16, 4> : launch_space_tokens<bf16, 1>)
                            : (vec ? launch_space_tokens<float, 4> : launch_space_tokens<float, 1>);
  return run(z, inp, ld, xbc, dt, cu_q, S, out, ldo, ST(stream));
}

extern "C" int zse_space_chunks(const void* inp, int ld, const void* xbc, const void* dt, const ZseSpace* z, const void* cu_q,
                                int first, int last, void* out, int ldo, void* stream) {
  if (last <= first) return 0;
  if (!space_shape_ok(z) || !zse_space_chunk_ok(z->state, z->vdim) || ld % 8 || z->conv_width % 8 || z->b_at % 8 ||
      z->c_at % 8 || ldo % 2 || last - first > 65535)
    return ZSE_ERR_SHAPE;
  return z->state <= 128 ? launch_space_chunks<1>(z, inp, ld, xbc, dt, cu_q, first, last, out, ldo, ST(stream))
                         : launch_space_chunks<2>(z, inp, ld, xbc, dt, cu_q, first, last, out, ldo, ST(stream));
}

extern "C" int zse_group_norm(int dtype, void* x, int ld, int M, int parts, int width, const void* weight, float eps,
                              void* stream) {
  if (M <= 0) return 0;
  if (parts <= 0 || width <= 0 || M > 65535) return ZSE_ERR_SHAPE;
  const cudaError_t e = dtype == kBF16 ? launch_group_norm<bf16>(x, ld, M, parts, width, weight, eps, ST(stream))
                                       : launch_group_norm<float>(x, ld, M, parts, width, weight, eps, ST(stream));
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}
