// Attention over heads whose keys and values have their own widths, grouped-query, with chunk or window masks.
//
//   heads_prep      second half of the fused input projection: split-K sum, bias, rotation, query and key norm, temperature
//                   of the queries, cache write
//   heads_prep_whole  the same where one norm covers all query (key) heads and comes before the rotation
//   heads_simple    a row's heads against the cached keys it sees; any shape, bfloat16 or float
//   heads_rows      the same on bfloat16 tensor cores: the query heads of a kv head are one 16-row tile, each warp streams
//                   its own tiles of 16 keys; keys may be split over CTAs (heads_combine merges)
//   heads_chunk     tiles of 64 queries of a sequence against tiles of 64 keys, flash-attention style (widths up to 128 take
//                   the tcgen05 form, heads_tc.cu)
//
// Cached tiles: [block][kv head][token][dim], then the same for values, dims padded to 8 (the padding is zero).  Scores and
// softmax are fp32; softmax weights enter the product with the values as two bfloat16 terms (value and remainder).  A row
// sees the positions from first_seen(position) to its own, and the first `keep` ones; block -1 of a table is a hole whose
// tokens do not exist.  With `pool` > 0 the means of blocks of tokens come before the window's tokens as further keys and values:
// rows of cache blocks of their own, which heads_prep_whole (decode) or heads_pool leave there.
#include "api.h"
#include "heads.cuh"

namespace zse {
namespace {

// ---- prep -----------------------------------------------------------------------------------------------------------
struct HeadsPrepArgs {
  int ld, k_col, v_col, gate_col, gate_w, own_kv;
  float eps;
  const float* turns;
  const int* positions;
  int rot_dims;
  float temp_coef;
  int temp_every;
};
constexpr int kPrepGates = 256;                  // gates of a warp
constexpr int kPrepPairs = 128;                  // pairs whose sine and cosine a CTA keeps in shared memory

// Sine and cosine of p * (turns per position, as two floats): the reduced angle keeps fp32 accuracy at any position.
__device__ __forceinline__ float2 pair_turn(const float* turns, int i, float p) {
  const float f = turns[2 * i], lo = turns[2 * i + 1];
  const float hi = p * f;
  const float r = (hi - rintf(hi)) + fmaf(p, lo, fmaf(p, f, -hi));
  float2 cs;
  sincospif(2.f * r, &cs.y, &cs.x);
  return cs;
}

// A warp per (row, section): query heads, then key heads, value heads and - with planes - the gates.  grid (rows, sections / 8)
// MORE: with bias, rotation or temperature.
template <typename T, int VEC, bool MORE>
__global__ void __launch_bounds__(256)
heads_prep_kernel(T* __restrict__ inp, const float* __restrict__ planes, int n_planes, int M, T* __restrict__ kc,
                  T* __restrict__ vc, Heads h, const long long* __restrict__ slots, const T* __restrict__ q_norm,
                  const T* __restrict__ k_norm, const T* __restrict__ bias, HeadsPrepArgs a, int units) {
  constexpr int kKeep = VEC == 4 ? 2 : 8;        // accesses of a head that stay in registers (up to 256 dimensions)
  __shared__ float2 turned[MORE ? kPrepPairs : 1];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x, u = blockIdx.y * 8 + (threadIdx.x >> 5);
  const float pos = MORE && a.positions != nullptr ? float(a.positions[t]) : 0.f;
  if (MORE && a.rot_dims > 0) {
    for (int i = threadIdx.x; i < min(kPrepPairs, a.rot_dims / 2); i += blockDim.x) turned[i] = pair_turn(a.turns, i, pos);
    __syncthreads();
  }
  if (u >= units) return;
  T* in = inp + size_t(t) * a.ld;
  const float* pl = planes + size_t(t) * a.ld;
  const size_t plane = size_t(M) * a.ld;
  auto value = [&](int c) {
    F32Vec<VEC> v{};
    if (n_planes == 0 && !MORE) return load_vec<VEC>(in + c);
    if (MORE && bias != nullptr) v = load_vec<VEC>(bias + c);
    if (n_planes == 0) {
      const F32Vec<VEC> x = load_vec<VEC>(in + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += x.v[e];
      return v;
    }
#pragma unroll 4
    for (int p = 0; p < n_planes; ++p) {
      const F32Vec<VEC> x = load_vec<VEC>(pl + p * plane + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += x.v[e];
    }
    return v;
  };
  const int G = a.own_kv ? h.kv_heads : 0;
  if (u >= h.heads + 2 * G) {                    // gates; their section is padded to 8 columns
    const int g0 = (u - h.heads - 2 * G) * kPrepGates, g1 = min(a.gate_w, g0 + kPrepGates);
#pragma unroll 2
    for (int i = g0 + lane * VEC; i < g1; i += 32 * VEC) store_vec<VEC>(in + a.gate_col + i, value(a.gate_col + i));
    return;
  }
  T* dst = nullptr;
  if (u >= h.heads) {
    const long long slot = slots[t];
    if (slot < 0) return;
    const int g = u - h.heads - (u >= h.heads + G ? G : 0), block = h.block_of(int(slot)), token = h.in_block(int(slot));
    if (u >= h.heads + G) {                      // values: copied
      dst = vc + h.at(block, g, token, h.vp);
      const int c0 = a.v_col + g * h.vdim;       // with v_col = k_col vdim is dim
      for (int i = lane * VEC; i < h.vdim; i += 32 * VEC) store_vec<VEC>(dst + i, value(c0 + i));
      return;
    }
    dst = kc + h.at(block, g, token, h.dp);
  }
  const int c0 = u < h.heads ? u * h.dim : a.k_col + (u - h.heads) * h.dim;
  const T* w = u < h.heads ? q_norm : k_norm;
  if (u < h.heads) dst = in + c0;
  auto turn = [&](int i, float& x, float& y) {   // the pair of dimensions i, i + 1
    const float2 cs = i / 2 < kPrepPairs ? turned[i / 2] : pair_turn(a.turns, i / 2, pos);
    const float u0 = x;
    x = u0 * cs.x - y * cs.y;
    y = y * cs.x + u0 * cs.y;
  };
  auto rotated = [&](int i) {                    // dimensions from i on
    F32Vec<VEC> v = value(c0 + i);
    if constexpr (!MORE) return v;
    if constexpr (VEC == 4) {
      if (i < a.rot_dims) turn(i, v.v[0], v.v[1]);
      if (i + 2 < a.rot_dims) turn(i + 2, v.v[2], v.v[3]);
    } else if (i < a.rot_dims) {
      float other = value(c0 + (i ^ 1)).v[0];
      if (i & 1)
        turn(i - 1, other, v.v[0]);
      else
        turn(i, v.v[0], other);
    }
    return v;
  };
  F32Vec<VEC> x[kKeep];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int i = (lane + j * 32) * VEC;
    if (i < h.dim) {
      x[j] = rotated(i);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x[j].v[e] * x[j].v[e];
    }
  }
  for (int i = (lane + kKeep * 32) * VEC; i < h.dim; i += 32 * VEC) {
    const F32Vec<VEC> v = value(c0 + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v.v[e] * v.v[e];
  }
  float inv = 1.f / sqrtf(warp_sum(ss) / float(h.dim) + a.eps);
  if (MORE && u < h.heads && a.temp_coef != 0.f)
    inv *= 1.f + a.temp_coef * logf(float((a.positions[t] + 1) / a.temp_every + 1));
  auto put = [&](int i, const F32Vec<VEC>& v) {
    F32Vec<VEC> y;
#pragma unroll
    for (int e = 0; e < VEC; ++e) y.v[e] = 1.f;
    if (w != nullptr) y = load_vec<VEC>(w + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) y.v[e] *= v.v[e] * inv;
    store_vec<VEC>(dst + i, y);
  };
  for (int i = (lane + kKeep * 32) * VEC; i < h.dim; i += 32 * VEC) put(i, rotated(i));
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int i = (lane + j * 32) * VEC;
    if (i < h.dim) put(i, x[j]);
  }
}

// The sum of a value over the block; `red`: one place per warp.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  return warp_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f);
}

// Pieces of VEC columns of a cached token, keys first, then values.
template <int VEC>
__device__ __forceinline__ int cached_pieces(const Heads& h) { return h.kv_heads * (h.dim / VEC + h.vdim / VEC); }

// Piece i of a cached token: a place in its row of `kc` or `vc`.
template <typename T, int VEC>
__device__ __forceinline__ T* cached_piece(T* kc, T* vc, const Heads& h, int block, int token, int i) {
  const int kv = h.dim / VEC, n = h.kv_heads * kv;
  if (i < n) return kc + h.at(block, i / kv, token, h.dp) + i % kv * VEC;
  const int vv = h.vdim / VEC;
  return vc + h.at(block, (i - n) / vv, token, h.vp) + (i - n) % vv * VEC;
}

// Sum of piece i over the cached tokens [from, to) of a sequence; blocks that are gone count as zeros.
template <typename T, int VEC>
__device__ __forceinline__ F32Vec<VEC> pool_sum(T* kc, T* vc, const Heads& h, const int* table, int i, int from, int to) {
  constexpr int kAhead = 8;                      // tokens whose loads are under way together
  F32Vec<VEC> sum{};
  const T* base = cached_piece<T, VEC>(kc, vc, h, 0, 0, i);
  const int width = i < h.kv_heads * (h.dim / VEC) ? h.dp : h.vp;
  for (int p0 = from; p0 < to; p0 += kAhead) {
    int block[kAhead];
    F32Vec<VEC> x[kAhead];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) block[u] = p0 + u < to ? table[h.block_of(p0 + u)] : -1;
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      x[u] = F32Vec<VEC>{};
      if (block[u] >= 0) x[u] = load_vec<VEC>(base + size_t(block[u]) * h.block_stride + size_t(h.in_block(p0 + u)) * width);
    }
#pragma unroll
    for (int u = 0; u < kAhead; ++u)
#pragma unroll
      for (int e = 0; e < VEC; ++e) sum.v[e] += x[u].v[e];
  }
  return sum;
}

// Stores a sum over a block of tokens as the mean of the sequence's block b.
template <typename T, int VEC>
__device__ __forceinline__ void put_mean(T* kc, T* vc, const Heads& h, const int* table, int i, int b, F32Vec<VEC> sum) {
  const int to = table[h.means_at + h.block_of(b)];
  if (to < 0) return;
  const float inv = 1.f / float(h.pool);
#pragma unroll
  for (int e = 0; e < VEC; ++e) sum.v[e] *= inv;
  store_vec<VEC>(cached_piece<T, VEC>(kc, vc, h, to, h.in_block(b), i), sum);
}

// grid (blocks of kPoolRows rows)
constexpr int kPoolRows = 16;
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
heads_pool_kernel(T* kc, T* vc, const Heads h, const int* __restrict__ row_seq, const int* __restrict__ positions, int M) {
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * kPoolRows;
  for (int t = t0; t < min(M, t0 + kPoolRows); ++t) {
    const int pos = positions[t];
    if ((pos + 1) % h.pool) continue;
    const int s = row_seq != nullptr ? row_seq[t] : t;
    const int* table = h.tables + size_t(s) * h.max_blocks;
    for (int i = threadIdx.x; i < cached_pieces<VEC>(h); i += 256)
      put_mean<T, VEC>(kc, vc, h, table, i, pos / h.pool, pool_sum<T, VEC>(kc, vc, h, table, i, pos + 1 - h.pool, pos + 1));
  }
}

// A CTA per row: split-K sum and bias of queries, keys, values and (with planes) gates; one norm over all queries and one over
// all keys, weights, rotation, factors of the heads' queries, cache write.  POOL: a row that completes a block of tokens leaves
// its mean in the cache as well; rows are sequences of their own.
template <typename T, int VEC, int THREADS>
__global__ void __launch_bounds__(THREADS)
heads_prep_whole_kernel(T* __restrict__ inp, const float* __restrict__ planes, int n_planes, int M, T* kc, T* vc, const Heads h,
                        const long long* __restrict__ slots, const T* __restrict__ q_norm, const T* __restrict__ k_norm,
                        const T* __restrict__ bias, const HeadsPrepArgs a, const float* __restrict__ head_temp, int pool_rows) {
  constexpr int kKeep = VEC == 4 ? 4 : 8;        // accesses of the queries that stay in registers
  __shared__ float2 turned[kPrepPairs];
  __shared__ float red[2][32];
  extern __shared__ float row[];                 // VEC 1: the queries with their bias (pairs lie in two threads)
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int pos_i = a.positions != nullptr ? a.positions[t] : 0;
  const float pos = float(pos_i);
  for (int i = threadIdx.x; i < min(kPrepPairs, a.rot_dims / 2); i += THREADS) turned[i] = pair_turn(a.turns, i, pos);
  T* in = inp + size_t(t) * a.ld;
  const float* pl = planes + size_t(t) * a.ld;
  const size_t plane = size_t(M) * a.ld;
  auto raw = [&](int c) {
    if (n_planes == 0) return load_vec<VEC>(in + c);
    F32Vec<VEC> v{};
#pragma unroll 4
    for (int p = 0; p < n_planes; ++p) {
      const F32Vec<VEC> x = load_vec<VEC>(pl + p * plane + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += x.v[e];
    }
    return v;
  };
  auto value = [&](int c) {
    F32Vec<VEC> v = raw(c);
    if (bias != nullptr) {
      const F32Vec<VEC> x = load_vec<VEC>(bias + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] += x.v[e];
    }
    return v;
  };
  const int nq = h.heads * h.dim, nk = a.own_kv ? h.kv_heads * h.dim : 0, nv = a.own_kv ? h.kv_heads * h.vdim : 0;
  const int step = THREADS * VEC, far = kKeep * step, i0 = threadIdx.x * VEC;
  constexpr bool kEarly = THREADS > 256;         // few rows: latency counts, not registers
  F32Vec<VEC> q[kKeep], qw[kEarly ? kKeep : 1], k0{}, kw{};
  float qs = 0.f, ks = 0.f;
  const long long slot = a.own_kv ? slots[t] : -1;
  // what does not depend on the row's values is under way before they are summed
  const int* table = h.tables + size_t(pool_rows ? t : 0) * h.max_blocks;
  const bool due = pool_rows && slot >= 0 && h.pool > 0 && (pos_i + 1) % h.pool == 0;
  const int pieces = cached_pieces<VEC>(h);
  F32Vec<VEC> before{};
  if (due && threadIdx.x < pieces) before = pool_sum<T, VEC>(kc, vc, h, table, threadIdx.x, pos_i + 1 - h.pool, pos_i);
  if (kEarly && i0 < nk) kw = load_vec<VEC>(k_norm + i0);
#pragma unroll
  for (int j = 0; j < kKeep; ++j)
    if (i0 + j * step < nq) {
      if constexpr (kEarly) qw[j] = load_vec<VEC>(q_norm + i0 + j * step);
      q[j] = value(i0 + j * step);
      if constexpr (VEC == 1) row[i0 + j * step] = q[j].v[0];
#pragma unroll
      for (int e = 0; e < VEC; ++e) qs += q[j].v[e] * q[j].v[e];
    }
  for (int i = far + i0; i < nq; i += step) {
    const F32Vec<VEC> x = value(i);
    if constexpr (VEC == 1) row[i] = x.v[0];
#pragma unroll
    for (int e = 0; e < VEC; ++e) qs += x.v[e] * x.v[e];
  }
  for (int i = i0; i < nk; i += step) {
    const F32Vec<VEC> x = value(a.k_col + i);
    if (i == i0) k0 = x;
#pragma unroll
    for (int e = 0; e < VEC; ++e) ks += x.v[e] * x.v[e];
  }
  const int block = slot >= 0 ? h.block_of(int(slot)) : 0, token = slot >= 0 ? h.in_block(int(slot)) : 0;
  if (slot >= 0) {
    for (int i = i0; i < nv; i += step)
      store_vec<VEC>(vc + h.at(block, i / h.vdim, token, h.vp) + i % h.vdim, value(a.v_col + i));
  }
  if (n_planes > 0)
    for (int i = i0; i < a.gate_w; i += step) store_vec<VEC>(in + a.gate_col + i, raw(a.gate_col + i));
  const float q_inv = 1.f / sqrtf(block_sum(qs, red[0]) / float(nq) + a.eps);
  const float k_inv = nk > 0 ? 1.f / sqrtf(block_sum(ks, red[1]) / float(nk) + a.eps) : 0.f;
  auto turn = [&](int i, float& x, float& y) {   // the pair of a head's dimensions i, i + 1
    const float2 cs = i / 2 < kPrepPairs ? turned[i / 2] : pair_turn(a.turns, i / 2, pos);
    const float u0 = x;
    x = u0 * cs.x - y * cs.y;
    y = y * cs.x + u0 * cs.y;
  };
  // columns i.. of the queries (or keys), normed, weighted and turned; `other_of`: one column of the same row, for VEC 1
  auto finished = [&](F32Vec<VEC> v, int i, float inv, const F32Vec<VEC>& f, const T* w, float factor, auto other_of) {
    const int d = i % h.dim;
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] *= inv * f.v[e];
    if constexpr (VEC == 4) {
      if (d < a.rot_dims) turn(d, v.v[0], v.v[1]);
      if (d + 2 < a.rot_dims) turn(d + 2, v.v[2], v.v[3]);
    } else if (d < a.rot_dims) {
      const int o = d & 1 ? i - 1 : i + 1;
      float other = other_of(o) * (inv * to_f32(w[o]));
      if (d & 1)
        turn(d - 1, other, v.v[0]);
      else
        turn(d, v.v[0], other);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] *= factor;
    return v;
  };
  auto put_q = [&](int i, const F32Vec<VEC>& x, const F32Vec<VEC>& w) {
    const float factor = head_temp != nullptr ? head_temp[i / h.dim] : 1.f;
    store_vec<VEC>(in + i, finished(x, i, q_inv, w, q_norm, factor, [&](int o) { return row[o]; }));
  };
#pragma unroll
  for (int j = 0; j < kKeep; ++j)
    if (i0 + j * step < nq) put_q(i0 + j * step, q[j], kEarly ? qw[kEarly ? j : 0] : load_vec<VEC>(q_norm + i0 + j * step));
  for (int i = far + i0; i < nq; i += step) {
    F32Vec<VEC> x;
    if constexpr (VEC == 1)
      x.v[0] = row[i];
    else
      x = value(i);
    put_q(i, x, load_vec<VEC>(q_norm + i));
  }
  if (slot < 0) return;                          // the same for the whole block
  for (int i = i0; i < nk; i += step) {
    const F32Vec<VEC> x = i == i0 ? k0 : value(a.k_col + i);
    store_vec<VEC>(kc + h.at(block, i / h.dim, token, h.dp) + i % h.dim,
                   finished(x, i, k_inv, kEarly && i == i0 ? kw : load_vec<VEC>(k_norm + i), k_norm, 1.f,
                            [&](int o) { return value(a.k_col + o).v[0]; }));
  }
  if (due) {
    __syncthreads();                             // this token's key and value are in the cache
    for (int i = threadIdx.x; i < pieces; i += THREADS) {
      F32Vec<VEC> sum = i == threadIdx.x ? before : pool_sum<T, VEC>(kc, vc, h, table, i, pos_i + 1 - h.pool, pos_i);
      const F32Vec<VEC> own = load_vec<VEC>(cached_piece<T, VEC>(kc, vc, h, block, token, i));
#pragma unroll
      for (int e = 0; e < VEC; ++e) sum.v[e] += own.v[e];
      put_mean<T, VEC>(kc, vc, h, table, i, pos_i / h.pool, sum);
    }
  }
}

// ---- any shape, any type -----------------------------------------------------------------------------------------------
// grid (heads, rows), 4 warps that take every fourth key.
template <typename T>
__global__ void __launch_bounds__(128)
heads_simple_kernel(const T* __restrict__ inp, int ld, const T* __restrict__ kc, const T* __restrict__ vc, Heads h,
                    const int* __restrict__ row_seq, const int* __restrict__ positions, T* __restrict__ out, int ldo,
                    const T* __restrict__ gate) {
  extern __shared__ float sm[];                  // q [dim], acc [4][vdim], m, l [4] each
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = head / (h.heads / h.kv_heads);
  float* q = sm;
  float* acc = sm + h.dim + warp * h.vdim;
  float* ml = sm + h.dim + 4 * h.vdim;
  const T* qp = inp + size_t(t) * ld + size_t(head) * h.dim;
  for (int i = threadIdx.x; i < h.dim; i += blockDim.x) q[i] = to_f32(qp[i]);
  for (int i = lane; i < h.vdim; i += 32) acc[i] = 0.f;
  __syncthreads();
  const int seq = row_seq != nullptr ? row_seq[t] : t, pos = positions[t];
  const int* table = h.tables + size_t(seq) * h.max_blocks;
  float m = -INFINITY, l = 0.f;
  const int lo = h.first_seen(pos), kept = h.pool > 0 ? h.means_seen(pos) : min(h.keep, lo);
  for (int n = warp; n < kept + pos + 1 - lo; n += 4) {
    const int j = n < kept ? n : lo + n - kept;
    const int block = table[(n < kept && h.pool > 0 ? h.means_at : 0) + h.block_of(j)];
    if (block < 0) continue;
    const T* k = kc + h.at(block, g, h.in_block(j), h.dp);
    const T* v = vc + h.at(block, g, h.in_block(j), h.vp);
    float s = 0.f;
    for (int i = lane; i < h.dim; i += 32) s = fmaf(q[i], to_f32(k[i]), s);
    s = warp_sum(s) * h.scale;
    if (h.cap > 0.f) s = h.cap * tanhf(s / h.cap);
    const float mn = fmaxf(m, s), corr = expf(m - mn), p = expf(s - mn);
    l = l * corr + p;
    m = mn;
    for (int i = lane; i < h.vdim; i += 32) acc[i] = acc[i] * corr + p * to_f32(v[i]);
  }
  if (lane == 0) {
    ml[warp] = m;
    ml[4 + warp] = l;
  }
  __syncthreads();
  float most = fmaxf(fmaxf(ml[0], ml[1]), fmaxf(ml[2], ml[3]));
  float f[4], L = 0.f;
  if (h.sink != nullptr) {
    most = fmaxf(most, h.sink[head]);
    L = expf(h.sink[head] - most);
  }
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    f[w] = ml[w] == -INFINITY ? 0.f : expf(ml[w] - most);
    L += ml[4 + w] * f[w];
  }
  const float inv = L > 0.f ? h.out_scale / L : 0.f;
  for (int i = threadIdx.x; i < h.vdim; i += blockDim.x) {
    float y = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) y += sm[h.dim + w * h.vdim + i] * f[w];
    if (gate != nullptr) y *= sigmoid_exact(to_f32(gate[size_t(t) * ld + h.gate_at(head, i)]));
    out[size_t(t) * ldo + size_t(head) * h.vdim + i] = from_f32<T>(y * inv);
  }
}

// What is special about a layer's scores: nothing, a soft cap, means of blocks as further keys.
enum ScoreKind { kPlainScores = 0, kCapped = 1, kPooled = 2 };

// ---- rows on tensor cores ----------------------------------------------------------------------------------------------
// An odd number of 16-byte pieces: consecutive rows start in different banks for ldmatrix.  Widths are whole steps of 16.
__host__ __device__ inline int pitch_of(int n) { return ((n + 15) / 16 * 2 + 1) * 16; }

constexpr int kRowWarps = 4, kRowStages = 3, kRowKeys = 16;
inline size_t rows_smem(int dim, int vdim) {
  const size_t ring = size_t(kRowWarps) * kRowStages * kRowKeys * (pitch_of(dim) + pitch_of(vdim));
  const size_t merge = size_t(kRowWarps) * 16 * (vdim + 2) * 4;
  return ring > merge ? ring : merge;
}

template <int DKS, int DVT, int KIND>  // steps of 16 key dimensions, blocks of 8 value dimensions (even)
__global__ void __launch_bounds__(kRowWarps * 32)
heads_rows_kernel(const bf16* __restrict__ inp, int ld, const bf16* __restrict__ kc, const bf16* __restrict__ vc, Heads h,
                  const int* __restrict__ row_seq, const int* __restrict__ positions, bf16* __restrict__ out, int ldo,
                  const bf16* __restrict__ gate, float* __restrict__ scratch, int num_splits, int groups) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int kvh = blockIdx.x / groups, t = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per = h.heads / h.kv_heads, head0 = kvh * per + blockIdx.x % groups * 16;
  const int G = min(16, (kvh + 1) * per - head0);                  // query heads of this CTA
  const int seq = row_seq != nullptr ? row_seq[t] : t, pos = positions[t];
  const int* table = h.tables + size_t(seq) * h.max_blocks;
  const int lo = h.first_seen(pos);
  const int tile0 = lo / kRowKeys;
  const int means = KIND == kPooled ? h.means_seen(pos) : 0;
  // tiles of kept tokens, or of means, before the first one of the window
  const int kept = KIND == kPooled ? (means + kRowKeys - 1) / kRowKeys : min(tile0, (h.keep + kRowKeys - 1) / kRowKeys);
  const int tiles = kept + pos / kRowKeys + 1 - tile0;
  const int per_split = (tiles + num_splits - 1) / num_splits;
  const int tb = split * per_split, te = min(tiles, tb + per_split);
  // first token of the i-th tile of this warp
  auto token_of = [&](int i) {
    const int n = tb + warp + i * kRowWarps;
    return (n < kept ? n : tile0 + n - kept) * kRowKeys;
  };
  auto of_means = [&](int i) { return KIND == kPooled && tb + warp + i * kRowWarps < kept; };
  auto block_at = [&](int i, int tok) { return table[(of_means(i) ? h.means_at : 0) + h.block_of(tok)]; };
  const int mine = te > tb + warp ? (te - tb - warp + kRowWarps - 1) / kRowWarps : 0;
  const int kp = pitch_of(h.dim), vp = pitch_of(h.vdim), ks = (h.dim + 15) / 16;
  const int kch = h.dp / 8, vch = h.vp / 8;
  uint8_t* ring = smem + warp * (kRowStages * kRowKeys * (kp + vp));

  uint32_t qa[DKS][4];
  {
    const int g0 = lane >> 2, g1 = g0 + 8, c0 = (lane & 3) * 2;
    const bf16* q0 = inp + size_t(t) * ld + size_t(head0 + g0) * h.dim;
    const bf16* q1 = q0 + size_t(8) * h.dim;
#pragma unroll
    for (int kk = 0; kk < DKS; ++kk) {
      const int c = kk * 16 + c0;
      qa[kk][0] = g0 < G && c < h.dim ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
      qa[kk][1] = g1 < G && c < h.dim ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
      qa[kk][2] = g0 < G && c + 8 < h.dim ? *reinterpret_cast<const uint32_t*>(q0 + c + 8) : 0u;
      qa[kk][3] = g1 < G && c + 8 < h.dim ? *reinterpret_cast<const uint32_t*>(q1 + c + 8) : 0u;
    }
  }
  if (kch < ks * 2 || (vch & 1)) {               // the halves of a step that no copy writes
    for (int r = lane; r < kRowStages * kRowKeys; r += 32) {
      uint8_t* st = ring + (r / kRowKeys) * kRowKeys * (kp + vp);
      if (kch < ks * 2) *reinterpret_cast<uint4*>(st + (r % kRowKeys) * kp + kch * 16) = make_uint4(0, 0, 0, 0);
      if (vch & 1)
        *reinterpret_cast<uint4*>(st + kRowKeys * kp + (r % kRowKeys) * vp + vch * 16) = make_uint4(0, 0, 0, 0);
    }
  }
  // a tile's rows are contiguous in the cache: piece j * 32 + lane of it goes to this place of the padded tile
  int k_to[DKS], v_to[DVT / 2];
#pragma unroll
  for (int j = 0; j < DKS; ++j) {
    const int idx = j * 32 + lane;
    k_to[j] = idx < kRowKeys * kch ? idx / kch * kp + idx % kch * 16 : -1;
  }
#pragma unroll
  for (int j = 0; j < DVT / 2; ++j) {
    const int idx = j * 32 + lane;
    v_to[j] = idx < kRowKeys * vch ? idx / vch * vp + idx % vch * 16 : -1;
  }
  auto issue = [&](int i) {                      // i-th tile of this warp; always commits a group
    if (i < mine) {
      const int tok = token_of(i), block = block_at(i, tok);
      if (block >= 0) {
        const bf16* ks_ = kc + h.at(block, kvh, h.in_block(tok), h.dp);
        const bf16* vs_ = vc + h.at(block, kvh, h.in_block(tok), h.vp);
        uint8_t* kd = ring + (i % kRowStages) * kRowKeys * (kp + vp);
        uint8_t* vd = kd + kRowKeys * kp;
#pragma unroll
        for (int j = 0; j < DKS; ++j)
          if (k_to[j] >= 0) cpa16(kd + k_to[j], ks_ + (j * 32 + lane) * 8);
#pragma unroll
        for (int j = 0; j < DVT / 2; ++j)
          if (v_to[j] >= 0) cpa16(vd + v_to[j], vs_ + (j * 32 + lane) * 8);
      }
    }
    cpa_commit();
  };
  float o[DVT][4];
#pragma unroll
  for (int n = 0; n < DVT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float scale_log2 = h.scale * kLog2E;
#pragma unroll
  for (int i = 0; i < kRowStages - 1; ++i) issue(i);
  for (int i = 0; i < mine; ++i) {
    cpa_wait<kRowStages - 2>();
    __syncwarp();
    issue(i + kRowStages - 1);
    const int tok = token_of(i);
    if (block_at(i, tok) < 0) continue;
    const bool mean = of_means(i);
    const uint32_t kb = smem_u32(ring + (i % kRowStages) * kRowKeys * (kp + vp)), vb = kb + kRowKeys * kp;
    float s[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < DKS; ++kk) {
      if (kk < ks) {
        uint32_t b[4];
        ldm_x4(kb + ((lane >> 4) * 8 + (lane & 7)) * kp + kk * 32 + (lane >> 3 & 1) * 16, b);
        mma_bf16(s[0], qa[kk], b[0], b[1]);
        mma_bf16(s[1], qa[kk], b[2], b[3]);
      }
    }
    float x[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int p = tok + j * 8 + (lane & 3) * 2 + (e & 1);
        const bool seen = KIND == kPooled ? (mean ? p < means : p <= pos && p >= lo) : h.sees(p, pos, lo);
        s[j][e] = seen ? (KIND == kCapped ? h.capped(s[j][e] * h.scale) * kLog2E : s[j][e] * scale_log2) : -INFINITY;
        x[e >> 1] = fmaxf(x[e >> 1], s[j][e]);
      }
    float base[2], corr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      x[r] = fmaxf(x[r], __shfl_xor_sync(0xffffffffu, x[r], 1));
      x[r] = fmaxf(x[r], __shfl_xor_sync(0xffffffffu, x[r], 2));
      const float mn = fmaxf(m[r], x[r]);
      base[r] = mn == -INFINITY ? 0.f : mn;
      corr[r] = ex2(m[r] - base[r]);
      m[r] = mn;
    }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
      l[0] *= corr[0];
      l[1] *= corr[1];
#pragma unroll
      for (int n = 0; n < DVT; ++n) {
        o[n][0] *= corr[0]; o[n][1] *= corr[0]; o[n][2] *= corr[1]; o[n][3] *= corr[1];
      }
    }
    float p[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        p[j][e] = ex2(s[j][e] - base[e >> 1]);
        l[e >> 1] += p[j][e];
      }
    const uint32_t ph[4] = {pack_bf16(p[0][0], p[0][1]), pack_bf16(p[0][2], p[0][3]), pack_bf16(p[1][0], p[1][1]),
                            pack_bf16(p[1][2], p[1][3])};
    const uint32_t pl[4] = {pack_bf16_rest(p[0][0], p[0][1]), pack_bf16_rest(p[0][2], p[0][3]),
                            pack_bf16_rest(p[1][0], p[1][1]), pack_bf16_rest(p[1][2], p[1][3])};
#pragma unroll
    for (int n = 0; n < DVT; n += 2) {
      if (n * 8 < h.vdim) {
        uint32_t v[4];
        ldm_x4_t(vb + ((lane >> 3 & 1) * 8 + (lane & 7)) * vp + (n + (lane >> 4)) * 16, v);
        mma_bf16(o[n], ph, v[0], v[1]);
        mma_bf16(o[n], pl, v[0], v[1]);
        mma_bf16(o[n + 1], ph, v[2], v[3]);
        mma_bf16(o[n + 1], pl, v[2], v[3]);
      }
    }
  }
  cpa_wait<0>();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  __syncthreads();                               // every warp is done with its ring
  float* mo = reinterpret_cast<float*>(smem);    // [warp][16][vdim], then maxima and sums [warp][16] each
  float* mm = mo + kRowWarps * 16 * h.vdim;
  float* ml = mm + kRowWarps * 16;
  {
    const int r0 = lane >> 2, c0 = (lane & 3) * 2;
    float* d = mo + warp * 16 * h.vdim;
#pragma unroll
    for (int n = 0; n < DVT; ++n) {
      const int c = n * 8 + c0;
      if (c < h.vdim) {
        *reinterpret_cast<float2*>(d + r0 * h.vdim + c) = make_float2(o[n][0], o[n][1]);
        *reinterpret_cast<float2*>(d + (r0 + 8) * h.vdim + c) = make_float2(o[n][2], o[n][3]);
      }
    }
    if ((lane & 3) == 0) {
      mm[warp * 16 + r0] = m[0];
      mm[warp * 16 + r0 + 8] = m[1];
      ml[warp * 16 + r0] = l[0];
      ml[warp * 16 + r0 + 8] = l[1];
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < G * h.vdim; idx += blockDim.x) {
    const int g = idx / h.vdim, d = idx % h.vdim;
    float most = -INFINITY;
#pragma unroll
    for (int w = 0; w < kRowWarps; ++w) most = fmaxf(most, mm[w * 16 + g]);
    float L = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < kRowWarps; ++w) {
      const float mw = mm[w * 16 + g], f = mw == -INFINITY ? 0.f : ex2(mw - most);
      L += ml[w * 16 + g] * f;
      acc += mo[(w * 16 + g) * h.vdim + d] * f;
    }
    const int head = head0 + g;
    if (num_splits == 1) {
      if (h.sink != nullptr) {
        const float sink = h.sink_log2(head), top = fmaxf(most, sink), f = ex2(most - top);
        L = L * f + ex2(sink - top);
        acc *= f;
      }
      float inv = L > 0.f ? h.out_scale / L : 0.f;
      if (gate != nullptr) inv *= sigmoid_exact(to_f32(gate[size_t(t) * ld + h.gate_at(head, d)]));
      out[size_t(t) * ldo + size_t(head) * h.vdim + d] = from_f32<bf16>(acc * inv);
    } else {
      float* dst = scratch + (size_t(t * h.heads + head) * num_splits + split) * (h.vdim + 2);
      dst[d] = acc;
      if (d == 0) {
        dst[h.vdim] = most;
        dst[h.vdim + 1] = L;
      }
    }
  }
}

// grid (heads, rows)
__global__ void __launch_bounds__(128)
heads_combine_kernel(const float* __restrict__ scratch, bf16* __restrict__ out, int ldo, const bf16* __restrict__ gate, int ld,
                     Heads h, int num_splits) {
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.x, t = blockIdx.y, heads = h.heads, vdim = h.vdim;
  const float* src = scratch + size_t(t * heads + head) * num_splits * (vdim + 2);
  float most = h.sink != nullptr ? h.sink_log2(head) : -INFINITY, L = 0.f;
  for (int s = 0; s < num_splits; ++s) most = fmaxf(most, src[s * (vdim + 2) + vdim]);
  if (h.sink != nullptr) L = ex2(h.sink_log2(head) - most);
  for (int s = 0; s < num_splits; ++s) {
    const float ms = src[s * (vdim + 2) + vdim];
    L += src[s * (vdim + 2) + vdim + 1] * (ms == -INFINITY ? 0.f : ex2(ms - most));
  }
  const float inv = L > 0.f ? h.out_scale / L : 0.f;
  for (int d = threadIdx.x; d < vdim; d += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < num_splits; ++s) {
      const float ms = src[s * (vdim + 2) + vdim];
      acc += src[s * (vdim + 2) + d] * (ms == -INFINITY ? 0.f : ex2(ms - most));
    }
    if (gate != nullptr) acc *= sigmoid_exact(to_f32(gate[size_t(t) * ld + h.gate_at(head, d)]));
    out[size_t(t) * ldo + size_t(head) * vdim + d] = from_f32<bf16>(acc * inv);
  }
}

// ---- tiles of queries --------------------------------------------------------------------------------------------------
constexpr int kChunkQ = 64, kChunkKeys = 64;
inline size_t chunk_smem(int dim, int vdim) {
  return size_t(kChunkQ + 2 * kChunkKeys) * pitch_of(dim) + size_t(2 * kChunkKeys) * pitch_of(vdim) + 2 * kChunkKeys * 4;
}

// CTA = (64 queries of a sequence, head), 4 warps of 16 queries; key tiles of 64 (aligned to 64) through a two-stage ring.
template <int DVT, int KIND>
__global__ void __launch_bounds__(128)
heads_chunk_kernel(const bf16* __restrict__ inp, int ld, const bf16* __restrict__ kc, const bf16* __restrict__ vc, Heads h,
                   const int* __restrict__ cu_q, const int* __restrict__ q_pos0, int first, bf16* __restrict__ out, int ldo,
                   const bf16* __restrict__ gate) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int s = first + blockIdx.z, head = blockIdx.y, kvh = head / (h.heads / h.kv_heads);
  const int q_begin = cu_q[s], q_len = cu_q[s + 1] - q_begin;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * kChunkQ;           // the longest key ranges first
  if (q0 >= q_len) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kp = pitch_of(h.dim), vp = pitch_of(h.vdim), ksteps = (h.dim + 15) / 16;
  const int kch = h.dp / 8, vch = h.vp / 8;
  uint8_t* sq = smem;
  uint8_t* sk = sq + kChunkQ * kp;
  uint8_t* sv = sk + 2 * kChunkKeys * kp;
  int* valid = reinterpret_cast<int*>(sv + 2 * kChunkKeys * vp);
  const int* table = h.tables + size_t(s) * h.max_blocks;
  const int p_first = q_pos0[s] + q0, p_last = q_pos0[s] + min(q_len, q0 + kChunkQ) - 1;
  const int see_all = h.first_seen(p_last);                        // from here on every query sees what is before it
  const int k_begin = h.first_seen(p_first) / kChunkKeys * kChunkKeys, k_end = p_last + 1;
  const int means = KIND == kPooled ? h.means_seen(p_last) : 0;
  // tiles of kept tokens or of means, then those from k_begin on
  const int kept = KIND == kPooled ? (means + kChunkKeys - 1) / kChunkKeys
                                   : min(k_begin / kChunkKeys, (h.keep + kChunkKeys - 1) / kChunkKeys);
  const int count = kept + (k_end - k_begin + kChunkKeys - 1) / kChunkKeys;
  auto key_of = [&](int i) { return i < kept ? i * kChunkKeys : k_begin + (i - kept) * kChunkKeys; };
  auto of_means = [&](int i) { return KIND == kPooled && i < kept; };

  for (int i = threadIdx.x; i < kChunkQ * ksteps * 2; i += 128) {
    const int r = i / (ksteps * 2), c = i % (ksteps * 2);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (q0 + r < q_len && c < h.dim / 8)
      v = *reinterpret_cast<const uint4*>(inp + size_t(q_begin + q0 + r) * ld + size_t(head) * h.dim + c * 8);
    *reinterpret_cast<uint4*>(sq + r * kp + c * 16) = v;
  }
  for (int r = threadIdx.x; r < 2 * kChunkKeys; r += 128) {        // halves of a step that no copy writes
    if (kch < ksteps * 2) *reinterpret_cast<uint4*>(sk + r * kp + kch * 16) = make_uint4(0, 0, 0, 0);
    if (vch & 1) *reinterpret_cast<uint4*>(sv + r * vp + vch * 16) = make_uint4(0, 0, 0, 0);
  }
  bool whole[2] = {true, true};                  // this thread's key of the stage exists
  auto issue = [&](int i) {
    if (i < count) {
      const int st = i & 1, key0 = key_of(i), end = of_means(i) ? means : k_end;
      const int* row = table + (of_means(i) ? h.means_at : 0);
      uint8_t *kd = sk + st * kChunkKeys * kp, *vd = sv + st * kChunkKeys * vp;
      if (threadIdx.x < kChunkKeys) {
        const int p = key0 + threadIdx.x;
        const bool v = p < end && row[h.block_of(p)] >= 0;
        valid[st * kChunkKeys + threadIdx.x] = v;
        if (st == 0) whole[0] = v; else whole[1] = v;
      }
      // runs of 16 keys are contiguous in a block; a warp takes one run
      const int tok = key0 + warp * 16, block = tok < end ? row[h.block_of(tok)] : -1;
      const size_t base_k = h.at(max(block, 0), kvh, h.in_block(tok), h.dp);
      const size_t base_v = h.at(max(block, 0), kvh, h.in_block(tok), h.vp);
      const int rows = block < 0 ? 0 : min(16, end - tok);
      for (int idx = lane; idx < 16 * kch; idx += 32) {
        const int r = idx / kch, c = idx % kch;
        uint8_t* d = kd + (warp * 16 + r) * kp + c * 16;
        if (r < rows) cpa16(d, kc + base_k + idx * 8); else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      }
      for (int idx = lane; idx < 16 * vch; idx += 32) {
        const int r = idx / vch, c = idx % vch;
        uint8_t* d = vd + (warp * 16 + r) * vp + c * 16;
        if (r < rows) cpa16(d, vc + base_v + idx * 8); else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      }
    }
    cpa_commit();
  };
  float o[DVT][4];
#pragma unroll
  for (int n = 0; n < DVT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int rq = lane >> 2, cq = (lane & 3) * 2;
  const int pr0 = p_first + warp * 16 + rq;                        // positions of this thread's two query rows
  const int lo[2] = {h.first_seen(pr0), h.first_seen(pr0 + 8)};
  const int seen_means[2] = {KIND == kPooled ? h.means_seen(pr0) : 0, KIND == kPooled ? h.means_seen(pr0 + 8) : 0};
  const uint32_t q_addr = smem_u32(sq) + (warp * 16 + (lane & 15)) * kp + (lane >> 4) * 16;
  const float scale_log2 = KIND == kCapped ? kLog2E : h.scale * kLog2E;

  issue(0);
  for (int i = 0; i < count; ++i) {
    issue(i + 1);
    cpa_wait<1>();
    const bool all_there = __syncthreads_and((i & 1) == 0 ? whole[0] : whole[1]) != 0;
    const uint32_t kb = smem_u32(sk + (i & 1) * kChunkKeys * kp), vb = smem_u32(sv + (i & 1) * kChunkKeys * vp);
    float sc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < ksteps; ++kk) {
      uint32_t a[4];
      ldm_x4(q_addr + kk * 32, a);
#pragma unroll
      for (int n = 0; n < 8; n += 2) {
        uint32_t b[4];
        ldm_x4(kb + ((n + (lane >> 4)) * 8 + (lane & 7)) * kp + kk * 32 + (lane >> 3 & 1) * 16, b);
        mma_bf16(sc[n], a, b[0], b[1]);
        mma_bf16(sc[n + 1], a, b[2], b[3]);
      }
    }
    const int key0 = key_of(i);
    float x[2] = {-INFINITY, -INFINITY};
    if constexpr (KIND == kCapped) {
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[n][e] = h.capped(sc[n][e] * h.scale);
    }
    const bool mean = of_means(i);
    const bool all_seen = mean ? key0 + kChunkKeys <= h.means_seen(p_first)
                               : key0 + kChunkKeys - 1 <= p_first && (key0 >= see_all || key0 + kChunkKeys <= h.keep);
    if (all_there && all_seen) {
#pragma unroll
      for (int n = 0; n < 8; ++n)                // every query sees every key
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          sc[n][e] *= scale_log2;
          x[e >> 1] = fmaxf(x[e >> 1], sc[n][e]);
        }
    } else {
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int c = n * 8 + cq + (e & 1), p = key0 + c;
          const bool in_reach = KIND == kPooled ? (mean ? p < seen_means[e >> 1] : p <= pr0 + (e >> 1) * 8 && p >= lo[e >> 1])
                                                : h.sees(p, pr0 + (e >> 1) * 8, lo[e >> 1]);
          const bool see = in_reach && valid[(i & 1) * kChunkKeys + c] != 0;
          sc[n][e] = see ? sc[n][e] * scale_log2 : -INFINITY;
          x[e >> 1] = fmaxf(x[e >> 1], sc[n][e]);
        }
    }
    float base[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      x[half] = fmaxf(x[half], __shfl_xor_sync(0xffffffffu, x[half], 1));
      x[half] = fmaxf(x[half], __shfl_xor_sync(0xffffffffu, x[half], 2));
      const float mn = fmaxf(m[half], x[half]);
      base[half] = mn == -INFINITY ? 0.f : mn;
      const float corr = ex2(m[half] - base[half]);
      m[half] = mn;
      l[half] *= corr;
#pragma unroll
      for (int n = 0; n < DVT; ++n) {
        o[n][half * 2] *= corr;
        o[n][half * 2 + 1] *= corr;
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      float p[2][4];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          p[j][e] = ex2(sc[2 * kk + j][e] - base[e >> 1]);
          l[e >> 1] += p[j][e];
        }
      const uint32_t ph[4] = {pack_bf16(p[0][0], p[0][1]), pack_bf16(p[0][2], p[0][3]), pack_bf16(p[1][0], p[1][1]),
                              pack_bf16(p[1][2], p[1][3])};
      const uint32_t pl[4] = {pack_bf16_rest(p[0][0], p[0][1]), pack_bf16_rest(p[0][2], p[0][3]),
                              pack_bf16_rest(p[1][0], p[1][1]), pack_bf16_rest(p[1][2], p[1][3])};
#pragma unroll
      for (int n = 0; n < DVT; n += 2) {
        if (n * 8 < h.vdim) {
          uint32_t v[4];
          ldm_x4_t(vb + (kk * 16 + (lane >> 3 & 1) * 8 + (lane & 7)) * vp + (n + (lane >> 4)) * 16, v);
          mma_bf16(o[n], ph, v[0], v[1]);
          mma_bf16(o[n], pl, v[0], v[1]);
          mma_bf16(o[n + 1], ph, v[2], v[3]);
          mma_bf16(o[n + 1], pl, v[2], v[3]);
        }
      }
    }
    __syncthreads();
  }
  cpa_wait<0>();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    float L = l[half];
    L += __shfl_xor_sync(0xffffffffu, L, 1);
    L += __shfl_xor_sync(0xffffffffu, L, 2);
    const int r = q0 + warp * 16 + rq + half * 8;
    if (r >= q_len) continue;
    const size_t t = size_t(q_begin + r);
    float inv;
    if (h.sink != nullptr) {
      const float sink = h.sink_log2(head), top = fmaxf(m[half], sink), f = ex2(m[half] - top);
      inv = h.out_scale * f / (L * f + ex2(sink - top));
    } else {
      inv = L > 0.f ? h.out_scale / L : 0.f;
    }
#pragma unroll
    for (int n = 0; n < DVT; ++n) {
      const int c = n * 8 + cq;
      if (c >= h.vdim) continue;
      float y0 = o[n][half * 2] * inv, y1 = o[n][half * 2 + 1] * inv;
      if (gate != nullptr) {
        y0 *= sigmoid_fast(to_f32(gate[t * ld + h.gate_at(head, c)]));
        y1 *= sigmoid_fast(to_f32(gate[t * ld + h.gate_at(head, c + 1)]));
      }
      *reinterpret_cast<uint32_t*>(out + t * ldo + size_t(head) * h.vdim + c) = pack_bf16(y0, y1);
    }
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

Heads heads_of(const ZseHeads* h) {
  int shift = -1;
  for (int i = 0; i < 30; ++i)
    if (h->block_size == 1 << i) shift = i;
  return Heads{(long long)(h->block_stride), h->block_size, h->dim_pad, h->vdim_pad, h->max_blocks, shift,
               reinterpret_cast<const int*>(h->tables), h->heads, h->kv_heads, h->dim, h->vdim, h->chunk, h->window,
               h->scale, h->keep_first, h->softcap, h->gate_each, h->pool, h->means_at,
               reinterpret_cast<const float*>(h->sink), h->out_scale};
}

struct RowsCall {
  const bf16* inp;
  int ld;
  const int *row_seq, *positions;
  bf16* out;
  int ldo;
  const bf16* gate;
  float* scratch;
  int M, splits;
  cudaStream_t st;
};

template <int DKS, int DVT, int KIND>
int launch_rows(const ZseHeads* z, const RowsCall& c) {
  static size_t done[kMaxDevices] = {};
  auto kern = heads_rows_kernel<DKS, DVT, KIND>;
  const Heads h = heads_of(z);
  const size_t smem = rows_smem(h.dim, h.vdim);
  if (int r = raise_smem(kern, smem, done)) return r;
  const int groups = (h.heads / h.kv_heads + 15) / 16;
  return launch_pdl(kern, dim3(h.kv_heads * groups, c.M, c.splits), dim3(kRowWarps * 32), smem, c.st, c.inp, c.ld,
                    reinterpret_cast<const bf16*>(z->k), reinterpret_cast<const bf16*>(z->v), h, c.row_seq, c.positions,
                    c.out, c.ldo, c.gate, c.scratch, c.splits, groups) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}
template <int DKS, int KIND>
int launch_rows_v(const ZseHeads* z, const RowsCall& c) {
  return z->vdim <= 64    ? launch_rows<DKS, 8, KIND>(z, c)
         : z->vdim <= 128 ? launch_rows<DKS, 16, KIND>(z, c)
                          : launch_rows<DKS, 32, KIND>(z, c);
}
template <int KIND>
int launch_rows_k(const ZseHeads* z, const RowsCall& c) {
  return z->dim <= 64    ? launch_rows_v<4, KIND>(z, c)
         : z->dim <= 128 ? launch_rows_v<8, KIND>(z, c)
                         : launch_rows_v<16, KIND>(z, c);
}

template <int DVT, int KIND>
int launch_chunks(const ZseHeads* z, const void* inp, int ld, const void* cu_q, const void* q_pos0, int first, int last,
                  int max_q, void* out, int ldo, const void* gate, cudaStream_t st) {
  static size_t done[kMaxDevices] = {};
  auto kern = heads_chunk_kernel<DVT, KIND>;
  const Heads h = heads_of(z);
  const size_t smem = chunk_smem(h.dim, h.vdim);
  if (int r = raise_smem(kern, smem, done)) return r;
  return launch_pdl(kern, dim3((max_q + kChunkQ - 1) / kChunkQ, h.heads, last - first), dim3(128), smem, st,
                    reinterpret_cast<const bf16*>(inp), ld, reinterpret_cast<const bf16*>(z->k),
                    reinterpret_cast<const bf16*>(z->v), h, reinterpret_cast<const int*>(cu_q),
                    reinterpret_cast<const int*>(q_pos0), first, reinterpret_cast<bf16*>(out), ldo,
                    reinterpret_cast<const bf16*>(gate)) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

template <typename T, int VEC>
cudaError_t launch_prep(void* inp, const void* planes, int n_planes, int M, const ZseHeads* z, const void* slots,
                        const ZseHeadsPrep* p, const HeadsPrepArgs& a, cudaStream_t st) {
  const Heads h = heads_of(z);
  const int units = h.heads + 2 * (a.own_kv ? h.kv_heads : 0) + (n_planes > 0 ? (a.gate_w + kPrepGates - 1) / kPrepGates : 0);
  const bool more = p->bias != nullptr || p->rot_dims > 0 || p->temp_coef != 0.f;
  return launch_pdl(more ? heads_prep_kernel<T, VEC, true> : heads_prep_kernel<T, VEC, false>, dim3(M, (units + 7) / 8),
                    dim3(256), 0, st,
                    reinterpret_cast<T*>(inp), reinterpret_cast<const float*>(planes), n_planes, M,
                    reinterpret_cast<T*>(z->k), reinterpret_cast<T*>(z->v), h, reinterpret_cast<const long long*>(slots),
                    reinterpret_cast<const T*>(p->q_norm), reinterpret_cast<const T*>(p->k_norm),
                    reinterpret_cast<const T*>(p->bias), a, units);
}

template <typename T, int VEC>
int launch_prep_whole(void* inp, const void* planes, int n_planes, int M, const ZseHeads* z, const void* slots,
                      const ZseHeadsPrep* p, const HeadsPrepArgs& a, cudaStream_t st) {
  static size_t done[2][kMaxDevices] = {};
  const Heads h = heads_of(z);
  const size_t smem = VEC == 1 ? size_t(h.heads) * h.dim * sizeof(float) : 0;
  const bool few = M < 4 * 148;                  // as many threads as a row has work for
  auto kern = few ? heads_prep_whole_kernel<T, VEC, 512> : heads_prep_whole_kernel<T, VEC, 256>;
  if (smem > 40 * 1024)
    if (int r = raise_smem(kern, smem, done[few])) return r;
  return launch_pdl(kern, dim3(M), dim3(few ? 512 : 256), smem, st, reinterpret_cast<T*>(inp),
                    reinterpret_cast<const float*>(planes), n_planes, M, reinterpret_cast<T*>(z->k),
                    reinterpret_cast<T*>(z->v), h, reinterpret_cast<const long long*>(slots),
                    reinterpret_cast<const T*>(p->q_norm), reinterpret_cast<const T*>(p->k_norm),
                    reinterpret_cast<const T*>(p->bias), a, reinterpret_cast<const float*>(p->head_temp),
                    p->pool_rows) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

// Vectors of four columns in every cached row.
bool cache_vec(const ZseHeads* h) {
  return h->dim % 4 == 0 && h->vdim % 4 == 0 && h->block_stride % 4 == 0 &&
         !((reinterpret_cast<uintptr_t>(h->k) | reinterpret_cast<uintptr_t>(h->v)) & 15);
}

bool pool_ok(const ZseHeads* h) {
  return h->pool >= 0 && (h->pool == 0 || (h->window > 0 && h->chunk == 0 && h->keep_first == 0 && h->softcap <= 0.f &&
                                           h->means_at > 0 && h->means_at <= h->max_blocks));
}

}  // namespace
}  // namespace zse

using namespace zse;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int zse_heads_mma_ok(int dim, int vdim, int block_size) {
  return dim % 8 == 0 && vdim % 8 == 0 && dim > 0 && vdim > 0 && dim <= 256 && vdim <= 256 && block_size % 16 == 0 &&
         rows_smem(dim, vdim) <= 227 * 1024 && chunk_smem(dim, vdim) <= 227 * 1024;
}

extern "C" int zse_heads_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, int M, const ZseHeads* h,
                              const void* slots, const ZseHeadsPrep* p, void* stream) {
  if (M <= 0) return 0;
  if (h->heads <= 0 || h->kv_heads <= 0 || h->heads % h->kv_heads || p->rot_dims % 2 || p->rot_dims > h->dim ||
      (p->temp_coef != 0.f && p->temp_every <= 0) || (p->own_kv && p->v_col == p->k_col && h->vdim != h->dim) ||
      ((p->rot_dims > 0 || p->temp_coef != 0.f) && p->positions == nullptr))
    return ZSE_ERR_SHAPE;
  const HeadsPrepArgs a{ld, p->k_col, p->v_col, p->gate_col, p->gate_w, p->own_kv, p->eps,
                        reinterpret_cast<const float*>(p->turns), reinterpret_cast<const int*>(p->positions), p->rot_dims,
                        p->temp_coef, p->temp_every};
  const bool vec = h->dim % 4 == 0 && h->vdim % 4 == 0 && ld % 4 == 0 && p->k_col % 4 == 0 && p->v_col % 4 == 0 &&
                   p->gate_col % 4 == 0 && p->gate_col + (p->gate_w + 3) / 4 * 4 <= ld &&
                   h->block_stride % 4 == 0 &&
                   !((reinterpret_cast<uintptr_t>(inp) | reinterpret_cast<uintptr_t>(planes) |
                      reinterpret_cast<uintptr_t>(h->k) | reinterpret_cast<uintptr_t>(h->v) |
                      reinterpret_cast<uintptr_t>(p->q_norm) | reinterpret_cast<uintptr_t>(p->k_norm) |
                      reinterpret_cast<uintptr_t>(p->bias)) & 15);
  if (p->whole) {
    if (p->temp_coef != 0.f || p->v_col == p->k_col || p->q_norm == nullptr || (p->own_kv && p->k_norm == nullptr) ||
        (p->pool_rows && (!pool_ok(h) || p->positions == nullptr)))
      return ZSE_ERR_SHAPE;
    auto whole = dtype == kBF16 ? (vec ? launch_prep_whole<bf16, 4> : launch_prep_whole<bf16, 1>)
                                : (vec ? launch_prep_whole<float, 4> : launch_prep_whole<float, 1>);
    return whole(inp, planes, n_planes, M, h, slots, p, a, ST(stream));
  }
  auto run = dtype == kBF16 ? (vec ? launch_prep<bf16, 4> : launch_prep<bf16, 1>)
                            : (vec ? launch_prep<float, 4> : launch_prep<float, 1>);
  return run(inp, planes, n_planes, M, h, slots, p, a, ST(stream)) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_heads_pool(int dtype, const ZseHeads* z, const void* row_seq, const void* positions, int M, void* stream) {
  if (M <= 0) return 0;
  if (!pool_ok(z) || z->pool <= 0) return ZSE_ERR_SHAPE;
  const Heads h = heads_of(z);
  const dim3 grid((M + kPoolRows - 1) / kPoolRows);
  const bool vec = cache_vec(z);
  const int* seq = reinterpret_cast<const int*>(row_seq);
  const int* pos = reinterpret_cast<const int*>(positions);
  const cudaError_t e =
      dtype == kBF16 ? launch_pdl(vec ? heads_pool_kernel<bf16, 4> : heads_pool_kernel<bf16, 1>, grid, dim3(256), 0, ST(stream),
                                  reinterpret_cast<bf16*>(z->k), reinterpret_cast<bf16*>(z->v), h, seq, pos, M)
                     : launch_pdl(vec ? heads_pool_kernel<float, 4> : heads_pool_kernel<float, 1>, grid, dim3(256), 0,
                                  ST(stream), reinterpret_cast<float*>(z->k), reinterpret_cast<float*>(z->v), h, seq, pos, M);
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_heads_attn(int dtype, const void* inp, int ld, const ZseHeads* z, const void* row_seq,
                              const void* positions, void* out, int ldo, const void* gate, void* scratch, int M,
                              int num_splits, int tensor_cores, void* stream) {
  if (M <= 0) return 0;
  if (z->heads <= 0 || z->kv_heads <= 0 || z->heads % z->kv_heads || M > 65535 || !pool_ok(z)) return ZSE_ERR_SHAPE;
  if (!tensor_cores || dtype != kBF16) {
    const Heads h = heads_of(z);
    const size_t smem = size_t(h.dim + 4 * h.vdim + 8) * sizeof(float);
    if (smem > 48 * 1024) return ZSE_ERR_LIMIT;
    const dim3 grid(h.heads, M);
    cudaError_t e;
    if (dtype == kBF16)
      e = launch_pdl(heads_simple_kernel<bf16>, grid, dim3(128), smem, ST(stream), reinterpret_cast<const bf16*>(inp), ld,
                     reinterpret_cast<const bf16*>(z->k), reinterpret_cast<const bf16*>(z->v), h,
                     reinterpret_cast<const int*>(row_seq), reinterpret_cast<const int*>(positions),
                     reinterpret_cast<bf16*>(out), ldo, reinterpret_cast<const bf16*>(gate));
    else
      e = launch_pdl(heads_simple_kernel<float>, grid, dim3(128), smem, ST(stream), reinterpret_cast<const float*>(inp), ld,
                     reinterpret_cast<const float*>(z->k), reinterpret_cast<const float*>(z->v), h,
                     reinterpret_cast<const int*>(row_seq), reinterpret_cast<const int*>(positions),
                     reinterpret_cast<float*>(out), ldo, reinterpret_cast<const float*>(gate));
    return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
  }
  if (!zse_heads_mma_ok(z->dim, z->vdim, z->block_size) || ld % 8 || z->block_stride % 8) return ZSE_ERR_SHAPE;
  if (num_splits > 1 && scratch == nullptr) num_splits = 1;
  const RowsCall c{reinterpret_cast<const bf16*>(inp), ld, reinterpret_cast<const int*>(row_seq),
                   reinterpret_cast<const int*>(positions), reinterpret_cast<bf16*>(out), ldo,
                   reinterpret_cast<const bf16*>(gate), reinterpret_cast<float*>(scratch), M, num_splits, ST(stream)};
  int rc = z->pool > 0        ? launch_rows_k<kPooled>(z, c)
           : z->softcap > 0.f ? launch_rows_k<kCapped>(z, c)
                              : launch_rows_k<kPlainScores>(z, c);
  if (rc == 0 && num_splits > 1 &&
      launch_pdl(heads_combine_kernel, dim3(z->heads, M), dim3(128), 0, ST(stream), reinterpret_cast<const float*>(scratch),
                 c.out, ldo, c.gate, ld, heads_of(z), num_splits) != cudaSuccess)
    rc = ZSE_ERR_LAUNCH;
  return rc;
}

extern "C" int zse_heads_attn_chunks(const void* inp, int ld, int rows, const ZseHeads* z, const void* cu_q,
                                     const void* q_pos0, int first, int last, int max_q, void* out, int ldo,
                                     const void* gate, int form, void* status, void* stream) {
  if (last <= first || max_q <= 0) return 0;
  if (!zse_heads_mma_ok(z->dim, z->vdim, z->block_size) || ld % 8 || ldo % 2 || z->block_stride % 8 ||
      z->heads % z->kv_heads || z->heads > 65535 || last - first > 65535 || !pool_ok(z))
    return ZSE_ERR_SHAPE;
  const Heads h = heads_of(z);
  if (form == 1 && heads_tc_ok(h, z->num_blocks, ld, ldo))
    return launch_heads_tc(reinterpret_cast<const bf16*>(inp), ld, rows, z->k, z->v, z->num_blocks, h,
                           reinterpret_cast<const int*>(cu_q), reinterpret_cast<const int*>(q_pos0), first, last, max_q,
                           reinterpret_cast<bf16*>(out), ldo, reinterpret_cast<const bf16*>(gate),
                           reinterpret_cast<Status*>(status), ST(stream));
  auto run = z->pool > 0
                 ? (z->vdim <= 64    ? launch_chunks<8, kPooled>
                    : z->vdim <= 128 ? launch_chunks<16, kPooled>
                                     : launch_chunks<32, kPooled>)
             : z->softcap > 0.f
                 ? (z->vdim <= 64    ? launch_chunks<8, kCapped>
                    : z->vdim <= 128 ? launch_chunks<16, kCapped>
                                     : launch_chunks<32, kCapped>)
                 : (z->vdim <= 64    ? launch_chunks<8, kPlainScores>
                    : z->vdim <= 128 ? launch_chunks<16, kPlainScores>
                                     : launch_chunks<32, kPlainScores>);
  return run(z, inp, ld, cu_q, q_pos0, first, last, max_q, out, ldo, gate, ST(stream));
}
