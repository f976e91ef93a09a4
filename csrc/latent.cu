// Latent attention: a token caches one row [latent (kv_rank) | rotated key part (rot)], shared by all heads.
//
//   latent_prep     second half of the fused input projection: latent norm, rotation, cache write
//   latent_attn     tokens against the cached rows themselves (queries already multiplied by W_uk): all heads of a group
//                   share each row, its leading part is the value as well (tcgen05 form: latent_tc.cu)
//   latent_combine  merges the key splits of a decode step
//   head_gemm       per-head products around latent_attn: q W_uk before it, o W_uv^T (times the gate) after it
//   latent_gather   cached rows a chunk's window reaches, in order, for the expansion GEMM
//   latent_chunk    a chunk's queries against the expanded per-head keys and values, flash-attention style
//
// Scores, softmax and rotation are fp32.  The bfloat16 kernels use mma.sync m16n8k16 tiles; softmax weights enter the
// product with the values as two bfloat16 terms (value and remainder), so that they keep 16 bits.  The *_simple kernels
// run any shape and float.  Cached rows are addressed through the block table; block -1 is a hole whose tokens do not exist.
#include "api.h"
#include "latent.cuh"

namespace zse {
namespace {

// ---- prep -----------------------------------------------------------------------------------------------------------
struct PrepArgs {
  int ld, heads, dim, rot, rot_dims, kv_rank, latent_col, gate_col, gate_w;
  float eps;
};

// With planes: grid (tokens, 1 + pieces): piece 0 does the latent, the others the queries and everything else that later
// kernels read, kPrepCols columns each.  Without: one CTA per token, warps 0..3 on the latent, the others on the queries,
// whose rotated parts turn in place.
constexpr int kPrepCols = 1024;
constexpr int kPrepLatent = 128;                 // threads on the latent

template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_kernel(T* __restrict__ inp, const float* __restrict__ planes, int n_planes, int M, T* __restrict__ cache,
                   RowCache rc, const int* __restrict__ positions, const long long* __restrict__ slots,
                   const float* __restrict__ freqs, const T* __restrict__ norm_w, PrepArgs a) {
  extern __shared__ float sm[];                  // cos, sin [rot_dims / 2] each; latent [kv_rank]
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, np = a.rot_dims / 2, qk = a.dim + a.rot;
  float* cs = sm;
  float* sn = sm + np;
  float* lat = sn + np;
  T* in = inp + size_t(t) * a.ld;
  const size_t plane = size_t(M) * a.ld;
  const float* pl = planes + size_t(t) * a.ld;
  auto value = [&](int c) {
    if (n_planes == 0) return to_f32(in[c]);
    float v = 0.f;
#pragma unroll 4
    for (int p = 0; p < n_planes; ++p) v += pl[p * plane + c];
    return v;
  };
  const float pos = float(positions[t]);
  for (int i = threadIdx.x; i < np; i += blockDim.x) sincosf(pos * freqs[i], &sn[i], &cs[i]);
  __syncthreads();
  if (n_planes == 0 && threadIdx.x >= kPrepLatent) {             // one thread per rotated pair
    const int step = blockDim.x - kPrepLatent, total = a.heads * np;
#pragma unroll 4
    for (int i = threadIdx.x - kPrepLatent; i < total; i += step) {
      const int h = i / np, j = i % np, c = h * qk + a.dim + 2 * j;
      const float u = to_f32(in[c]), v = to_f32(in[c + 1]);
      in[c] = from_f32<T>(u * cs[j] - v * sn[j]);
      in[c + 1] = from_f32<T>(v * cs[j] + u * sn[j]);
    }
    return;
  }
  if (blockIdx.y > 0) {
    const int c0 = (blockIdx.y - 1) * kPrepCols, qw = a.heads * qk;
#pragma unroll
    for (int k = 0; k < kPrepCols / 256; ++k) {
      const int i = c0 + threadIdx.x + k * 256;
      if (i >= qw + a.gate_w) break;
      if (i >= qw) {
        const int c = a.gate_col + i - qw;
        in[c] = from_f32<T>(value(c));
        continue;
      }
      const int j = i % qk - a.dim;              // place in the rotated part
      float v = value(i);
      if (j >= 0 && j < a.rot_dims) v = v * cs[j >> 1] + ((j & 1) ? value(i - 1) : -value(i + 1)) * sn[j >> 1];
      in[i] = from_f32<T>(v);
    }
    return;
  }
  if (threadIdx.x >= kPrepLatent) return;
  float ss = 0.f;
#pragma unroll 4
  for (int i = threadIdx.x; i < a.kv_rank; i += kPrepLatent) {
    const float v = value(a.latent_col + i);
    lat[i] = v;
    ss += v * v;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  asm volatile("bar.sync 1, %0;" ::"n"(kPrepLatent) : "memory");
  const float total = warp_sum((threadIdx.x & 31) < kPrepLatent / 32 ? red[threadIdx.x & 31] : 0.f);
  const float inv = 1.f / sqrtf(total / float(a.kv_rank) + a.eps);
  const long long slot = slots[t];
  if (slot < 0) return;
  T* dst = cache + (slot / rc.block_size) * rc.block_stride + (slot % rc.block_size) * rc.row;
  for (int i = threadIdx.x; i < a.kv_rank; i += kPrepLatent) dst[i] = from_f32<T>(lat[i] * inv * to_f32(norm_w[i]));
  const int r0 = a.latent_col + a.kv_rank;
  for (int j = threadIdx.x; j < a.rot; j += kPrepLatent) {
    float v = value(r0 + j);
    if (j < a.rot_dims) v = v * cs[j >> 1] + ((j & 1) ? value(r0 + j - 1) : -value(r0 + j + 1)) * sn[j >> 1];
    dst[a.kv_rank + j] = from_f32<T>(v);
  }
}

// ---- tokens against the cached rows: any shape, any type ---------------------------------------------------------------
// grid (heads, tokens), 4 warps that take every fourth key.
template <typename T>
__global__ void __launch_bounds__(128)
latent_attn_simple_kernel(const T* __restrict__ q_lat, const T* __restrict__ cache, RowCache rc,
                          const int* __restrict__ row_seq, const int* __restrict__ positions, T* __restrict__ o_lat,
                          int heads, int used, int kv_rank, int window, float scale) {
  extern __shared__ float sm[];                  // q [used], acc [4][kv_rank], then m, l [4] each
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* q = sm;
  float* acc = sm + used + warp * kv_rank;
  float* ml = sm + used + 4 * kv_rank;
  const T* qp = q_lat + (size_t(t) * heads + h) * rc.row;
  for (int i = threadIdx.x; i < used; i += blockDim.x) q[i] = to_f32(qp[i]);
  for (int i = lane; i < kv_rank; i += 32) acc[i] = 0.f;
  __syncthreads();
  const int seq = row_seq != nullptr ? row_seq[t] : t, pos = positions[t];
  const int* table = rc.tables + size_t(seq) * rc.max_blocks;
  const int lo = window > 0 ? max(0, pos + 1 - window) : 0;
  float m = -INFINITY, l = 0.f;
  for (int j = lo + warp; j <= pos; j += 4) {
    const int blk = table[j / rc.block_size];
    if (blk < 0) continue;
    const T* row = cache + blk * rc.block_stride + size_t(j % rc.block_size) * rc.row;
    float s = 0.f;
    for (int i = lane; i < used; i += 32) s = fmaf(q[i], to_f32(row[i]), s);
    s = warp_sum(s) * scale;
    const float mn = fmaxf(m, s), corr = expf(m - mn), p = expf(s - mn);
    l = l * corr + p;
    m = mn;
    for (int i = lane; i < kv_rank; i += 32) acc[i] = acc[i] * corr + p * to_f32(row[i]);
  }
  if (lane == 0) {
    ml[warp] = m;
    ml[4 + warp] = l;
  }
  __syncthreads();
  const float mx = fmaxf(fmaxf(ml[0], ml[1]), fmaxf(ml[2], ml[3]));
  float f[4], L = 0.f;
  for (int w = 0; w < 4; ++w) {
    f[w] = ml[w] == -INFINITY ? 0.f : expf(ml[w] - mx);
    L += f[w] * ml[4 + w];
  }
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) {
    float v = 0.f;
    for (int w = 0; w < 4; ++w) v += f[w] * sm[used + w * kv_rank + i];
    o_lat[(size_t(t) * heads + h) * kv_rank + i] = from_f32<T>(L > 0.f ? v / L : 0.f);
  }
}

// ---- tokens against the cached rows: bfloat16 tensor cores ----------------------------------------------------------
// CTA = (group of 16 * MT heads, token, key split), 8 warps.  Tiles of 64 keys (aligned to 64, so a tile is a whole number
// of blocks, or part of one) arrive by bulk copies, one per block, in a two-stage ring.  A cached row is an odd number of
// 16-byte pieces, which makes ldmatrix conflict-free on the rows exactly as they lie in the cache: nothing is rearranged.
// Scores: warp (kg, g) takes keys 16 kg .. 16 kg + 15 for head tile g (MT = 2), or for half of the row's columns with the
// halves exchanged through shared memory (MT = 1).  Values: warp w takes NTW blocks of 8 latent columns for every key.
constexpr int kLatKeys = 64;
constexpr int kLatWarps = 8;

__host__ __device__ inline int latent_qpitch(int used) { return (used + 15) / 16 * 32 + 16; }     // bytes
inline size_t latent_smem(int mt, int row, int used) {
  return size_t(16 * mt) * latent_qpitch(used) + size_t(2 * kLatKeys) * row * 2 + 64 + 2 * size_t(16 * mt) * (kLatKeys * 2 + 16) +
         size_t(2 * kLatWarps * 16 * mt) * 4 + kLatWarps * 32 * 16 + 2 * kLatKeys * 4 + 64;
}

template <int MT, int NTW>
__global__ void __launch_bounds__(kLatWarps * 32)
latent_attn_kernel(const bf16* __restrict__ q_lat, const bf16* __restrict__ cache, RowCache rc,
                   const int* __restrict__ row_seq, const int* __restrict__ positions, bf16* __restrict__ o_lat,
                   float* __restrict__ scratch, int heads, int used, int kv_rank, int window, float scale_log2,
                   int num_splits, Status* status) {
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int kRows = 16 * MT;
  constexpr int kPPitch = kLatKeys * 2 + 16;
  const int row = rc.row, pitch = row * 2, qpitch = latent_qpitch(used), ksteps = (used + 15) / 16, chunks = row / 8;
  const int stage_bytes = kLatKeys * pitch;
  uint8_t* sq = smem;
  uint8_t* sk = sq + kRows * qpitch;                             // two stages, then 64 bytes that the last k step may read
  uint8_t* sp = sk + 2 * stage_bytes + 64;                       // [hi, lo][kRows][kPPitch]
  float* smax = reinterpret_cast<float*>(sp + 2 * kRows * kPPitch);   // [warps][kRows]
  float* ssum = smax + kLatWarps * kRows;
  float4* swap = reinterpret_cast<float4*>(ssum + kLatWarps * kRows); // [warps][32]
  int* valid = reinterpret_cast<int*>(swap + kLatWarps * 32);         // [2][kLatKeys]
  uint64_t* full = reinterpret_cast<uint64_t*>(valid + 2 * kLatKeys); // [2]
  int* abort_flag = reinterpret_cast<int*>(full + 2);
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kg = warp & 3, g = warp >> 2;
  if (threadIdx.x == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  // a hole is not copied and its weights are 0: what lies there has to be finite
  for (int i = threadIdx.x; i < (2 * stage_bytes + 64) / 16; i += blockDim.x)
    reinterpret_cast<uint4*>(sk)[i] = make_uint4(0, 0, 0, 0);
  fence_proxy_async_smem();
  pdl_wait();
  const int h0 = blockIdx.x * kRows, t = blockIdx.y, split = blockIdx.z;
  const int nh = min(kRows, heads - h0);
  const int seq = row_seq != nullptr ? row_seq[t] : t, pos = positions[t];
  const int* table = rc.tables + size_t(seq) * rc.max_blocks;
  const int lo = window > 0 ? max(0, pos + 1 - window) : 0;
  const int tile0 = lo / kLatKeys, n_tiles = pos / kLatKeys + 1 - tile0;
  const int per = (n_tiles + num_splits - 1) / num_splits;
  const int first = tile0 + split * per;
  const int count = max(0, min(tile0 + n_tiles, first + per) - first);
  for (int r = warp; r < kRows; r += kLatWarps) {                // queries (zero rows beyond the heads)
    const bf16* src = q_lat + (size_t(t) * heads + h0 + r) * row;
    for (int c = lane; c < ksteps * 2; c += 32)
      *reinterpret_cast<uint4*>(sq + r * qpitch + c * 16) =
          r < nh && c < chunks ? *reinterpret_cast<const uint4*>(src + c * 8) : make_uint4(0, 0, 0, 0);
  }
  __syncthreads();

  const int piece = min(rc.block_size, kLatKeys);                // keys of a tile that lie in one block
  auto issue = [&](int i) {                                      // warp 0
    const int st = i & 1, key0 = (first + i) * kLatKeys;
    const int k = lane * piece;                                  // first key of this lane's piece
    int blk = -1;
    if (k < kLatKeys && key0 + k <= pos) blk = table[(key0 + k) / rc.block_size];
    const unsigned have = __ballot_sync(0xffffffffu, blk >= 0);
    for (int j = lane; j < kLatKeys; j += 32) {
      const int key = key0 + j;
      valid[st * kLatKeys + j] = key >= lo && key <= pos && (have >> (j / piece) & 1);
    }
    if (lane == 0) mbar_arrive_expect_tx(&full[st], __popc(have) * piece * pitch);
    __syncwarp();
    if (blk >= 0)
      bulk_g2s(sk + st * stage_bytes + k * pitch,
               cache + blk * rc.block_stride + size_t((key0 + k) % rc.block_size) * row, piece * pitch, &full[st]);
  };

  float o[MT][NTW][4];
  float m[MT][2], l[2] = {0.f, 0.f};
#pragma unroll
  for (int a = 0; a < MT; ++a) {
    m[a][0] = m[a][1] = -INFINITY;
#pragma unroll
    for (int n = 0; n < NTW; ++n) o[a][n][0] = o[a][n][1] = o[a][n][2] = o[a][n][3] = 0.f;
  }
  const int rq = lane >> 2, cq = (lane & 3) * 2;
  constexpr int kMaxParts = MT == 1 ? kLatWarps : 4;             // warps that share a head tile's keys
  const int part = MT == 1 ? warp : kg, tile_row = MT == 1 ? 0 : g * 16;
  const uint32_t q_addr = smem_u32(sq) + (tile_row + (lane & 15)) * qpitch + (lane >> 4) * 16;
  const uint32_t p_addr = smem_u32(sp) + (lane & 15) * kPPitch + (lane >> 4) * 16;
  const int half_steps = (ksteps + 1) / 2;
  const int kk0 = MT == 1 ? g * half_steps : 0;
  const int kk1 = MT == 1 ? min(ksteps, kk0 + half_steps) : ksteps;
  const int key_w = MT == 1 ? kg * 16 + g * 8 : kg * 16;         // first key this warp weighs

  bool ok = true;
  if (warp == 0 && count > 0) issue(0);
  for (int i = 0; i < count; ++i) {
    if (warp == 0 && i + 1 < count) issue(i + 1);
    ok = mbar_wait(&full[i & 1], (i >> 1) & 1, abort_flag, status, 81, i);
    ok = __syncthreads_and(ok) != 0;
    if (!ok) {                                                   // reported; let the copies in flight land
      if (threadIdx.x == 0)
        for (int j = i; j < min(count, i + 2); ++j) {
          SpinClock clock;
          while (!mbar_try_wait(&full[j & 1], (j >> 1) & 1) && !clock.expired(0xFF)) {
          }
        }
      break;
    }
    const uint32_t kbase = smem_u32(sk) + (i & 1) * stage_bytes;
    float s[2][2][4];                                            // [even, odd step][8 keys]
#pragma unroll
    for (int e = 0; e < 4; ++e) s[0][0][e] = s[0][1][e] = s[1][0][e] = s[1][1][e] = 0.f;
    const uint32_t k_addr = kbase + (kg * 16 + (lane >> 4) * 8 + (lane & 7)) * pitch + (lane >> 3 & 1) * 16;
    int kk = kk0;
#pragma unroll 2
    for (; kk + 1 < kk1; kk += 2) {
      uint32_t qa[4], qb[4], b[4], c[4];
      ldm_x4(q_addr + kk * 32, qa);
      ldm_x4(k_addr + kk * 32, b);
      ldm_x4(q_addr + kk * 32 + 32, qb);
      ldm_x4(k_addr + kk * 32 + 32, c);
      mma_bf16(s[0][0], qa, b[0], b[1]);
      mma_bf16(s[0][1], qa, b[2], b[3]);
      mma_bf16(s[1][0], qb, c[0], c[1]);
      mma_bf16(s[1][1], qb, c[2], c[3]);
    }
    if (kk < kk1) {
      uint32_t qa[4], b[4];
      ldm_x4(q_addr + kk * 32, qa);
      ldm_x4(k_addr + kk * 32, b);
      mma_bf16(s[0][0], qa, b[0], b[1]);
      mma_bf16(s[0][1], qa, b[2], b[3]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      s[0][0][e] += s[1][0][e];
      s[0][1][e] += s[1][1][e];
    }
    if (MT == 1) {                                               // the other half of the columns of this warp's 8 keys
      const float* give = g == 0 ? s[0][1] : s[0][0];
      swap[warp * 32 + lane] = make_float4(give[0], give[1], give[2], give[3]);
      __syncthreads();
      const float4 got = swap[(warp ^ 4) * 32 + lane];
      if (g == 1) {
#pragma unroll
        for (int e = 0; e < 4; ++e) s[0][0][e] = s[0][1][e];
      }
      s[0][0][0] += got.x;
      s[0][0][1] += got.y;
      s[0][0][2] += got.z;
      s[0][0][3] += got.w;
    }
    float x[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < MT; ++nb) {
      const int* ok_key = valid + (i & 1) * kLatKeys + key_w + nb * 8 + cq;
      const bool ok0 = ok_key[0] != 0, ok1 = ok_key[1] != 0;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[0][nb][e] = ((e & 1) ? ok1 : ok0) ? s[0][nb][e] * scale_log2 : -INFINITY;
        x[e >> 1] = fmaxf(x[e >> 1], s[0][nb][e]);
      }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      x[half] = fmaxf(x[half], __shfl_xor_sync(0xffffffffu, x[half], 1));
      x[half] = fmaxf(x[half], __shfl_xor_sync(0xffffffffu, x[half], 2));
      if ((lane & 3) == 0) smax[part * kRows + tile_row + rq + half * 8] = x[half];
    }
    __syncthreads();
    bool moved = false;
    float corr[MT][2];
#pragma unroll
    for (int a = 0; a < MT; ++a) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float mn = m[a][half];
#pragma unroll
        for (int w = 0; w < kMaxParts; ++w) mn = fmaxf(mn, smax[w * kRows + a * 16 + rq + half * 8]);
        const float base = mn == -INFINITY ? 0.f : mn;
        corr[a][half] = ex2(m[a][half] - base);                // 0 when there was nothing before
        moved |= mn > m[a][half];
        m[a][half] = mn;
      }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int a0 = MT == 1 ? 0 : g;
      const float mine = MT == 1 ? m[0][half] : (a0 == 0 ? m[0][half] : m[MT - 1][half]);
      const float base = mine == -INFINITY ? 0.f : mine;
      l[half] *= MT == 1 ? corr[0][half] : (a0 == 0 ? corr[0][half] : corr[MT - 1][half]);
      const int r = tile_row + rq + half * 8;
#pragma unroll
      for (int nb = 0; nb < MT; ++nb) {
        const float p0 = ex2(s[0][nb][half * 2] - base), p1 = ex2(s[0][nb][half * 2 + 1] - base);
        l[half] += p0 + p1;
        const int key = key_w + nb * 8 + cq;
        *reinterpret_cast<uint32_t*>(sp + r * kPPitch + key * 2) = pack_bf16(p0, p1);
        *reinterpret_cast<uint32_t*>(sp + (kRows + r) * kPPitch + key * 2) = pack_bf16_rest(p0, p1);
      }
    }
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int n = 0; n < NTW; ++n) {
          o[a][n][0] *= corr[a][0];
          o[a][n][1] *= corr[a][0];
          o[a][n][2] *= corr[a][1];
          o[a][n][3] *= corr[a][1];
        }
    }
    __syncthreads();
    const int vr = (lane >> 3 & 1) * 8 + (lane & 7), vc = lane >> 4;
#pragma unroll
    for (int kv = 0; kv < kLatKeys / 16; ++kv) {
      uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
      for (int a = 0; a < MT; ++a) {
        ldm_x4(p_addr + a * 16 * kPPitch + kv * 32, ph[a]);
        ldm_x4(p_addr + (kRows + a * 16) * kPPitch + kv * 32, pl[a]);
      }
#pragma unroll
      for (int n = 0; n < NTW; n += 2) {
        const int col = warp * NTW + n;                          // block of 8 columns (warp-uniform bound)
        if (col * 8 < kv_rank) {
          uint32_t v[4];
          ldm_x4_t(kbase + (kv * 16 + vr) * pitch + (col + vc) * 16, v);
#pragma unroll
          for (int a = 0; a < MT; ++a) {
            mma_bf16(o[a][n], ph[a], v[0], v[1]);
            mma_bf16(o[a][n + 1], ph[a], v[2], v[3]);
            mma_bf16(o[a][n], pl[a], v[0], v[1]);
            mma_bf16(o[a][n + 1], pl[a], v[2], v[3]);
          }
        }
      }
    }
    __syncthreads();                                             // the stage may be refilled
  }
  if (!ok) return;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    float v = l[half];
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    if ((lane & 3) == 0) ssum[part * kRows + tile_row + rq + half * 8] = v;
  }
  __syncthreads();
#pragma unroll
  for (int a = 0; a < MT; ++a) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = a * 16 + rq + half * 8;
      if (r >= nh) continue;
      float L = 0.f;
#pragma unroll
      for (int w = 0; w < kMaxParts; ++w) L += ssum[w * kRows + r];
      const size_t hh = size_t(t) * heads + h0 + r;
      const float inv = L > 0.f ? 1.f / L : 0.f;
      float* out = scratch + (hh * num_splits + split) * (kv_rank + 2);
#pragma unroll
      for (int n = 0; n < NTW; ++n) {
        const int c = (warp * NTW + n) * 8 + cq;
        const float x = o[a][n][half * 2], y = o[a][n][half * 2 + 1];
        if (c >= kv_rank) continue;                              // kv_rank is a multiple of 8, c + 1 is below it too
        if (num_splits == 1)
          *reinterpret_cast<uint32_t*>(o_lat + hh * kv_rank + c) = pack_bf16(x * inv, y * inv);
        else
          *reinterpret_cast<float2*>(out + c) = make_float2(x, y);
      }
      if (num_splits > 1 && warp == 0 && (lane & 3) == 0) {
        out[kv_rank] = m[a][half];
        out[kv_rank + 1] = L;
      }
    }
  }
}

__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ scratch, bf16* __restrict__ o_lat, int heads, int kv_rank,
                      int num_splits) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t hh = size_t(blockIdx.y) * heads + blockIdx.x;
  const float* src = scratch + hh * num_splits * (kv_rank + 2);
  float M = -INFINITY, L = 0.f;
  for (int s = 0; s < num_splits; ++s) M = fmaxf(M, src[s * (kv_rank + 2) + kv_rank]);
  for (int s = 0; s < num_splits; ++s) {
    const float ms = src[s * (kv_rank + 2) + kv_rank];
    L += ms == -INFINITY ? 0.f : exp2f(ms - M) * src[s * (kv_rank + 2) + kv_rank + 1];
  }
  const float inv = L > 0.f ? 1.f / L : 0.f;
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < num_splits; ++s) {
      const float ms = src[s * (kv_rank + 2) + kv_rank];
      if (ms != -INFINITY) v += exp2f(ms - M) * src[s * (kv_rank + 2) + i];
    }
    o_lat[hh * kv_rank + i] = from_f32<bf16>(v * inv);
  }
}

// ---- per-head products (bfloat16) -------------------------------------------------------------------------------------
// out[t, h, n] = sum_k A[t, h, k] * B[h][k, n] (KN) or B[h][n, k] (NK).  64 tokens x 64 columns per CTA, 4 warps of 16
// tokens, K in steps of 64 through a four-stage cp.async ring.  All of dim, kv_rank and vdim are multiples of 8.
struct HeadGemmArgs {
  const bf16* a;
  long long lda, a_head;
  const bf16* b;
  long long b_head;
  bf16* out;
  long long ldo, o_head;
  int M, N, K;
  // KN form (absorb): `tail` more columns are copied behind the N products, zero up to tail_pad
  const bf16* tail;
  int tail_n, tail_pad;
  // NK form: result times sigmoid(gate) when gate is given
  const bf16* gate;
  long long ldg, gate_head;
};
constexpr int kHgPitch = 144;             // bytes of a 64-element row + 16
constexpr int kHgStages = 4;
constexpr int kHgSmem = kHgStages * 2 * 64 * kHgPitch;

template <bool KN>
__global__ void __launch_bounds__(128) head_gemm_kernel(const HeadGemmArgs p) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * 64, h = blockIdx.y, m0 = blockIdx.z * 64;
  const bf16* A = p.a + h * p.a_head;
  const bf16* B = p.b + h * p.b_head;
  const int iters = (p.K + 63) / 64;
  auto issue = [&](int it) {
    if (it < iters) {
      uint8_t* sa = smem + (it % kHgStages) * 2 * 64 * kHgPitch;
      uint8_t* sb = sa + 64 * kHgPitch;
      const int k0 = it * 64;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int idx = threadIdx.x + j * 128, r = idx >> 3, c = idx & 7;
        if (m0 + r < p.M && k0 + c * 8 < p.K)
          cpa16(sa + r * kHgPitch + c * 16, A + size_t(m0 + r) * p.lda + k0 + c * 8);
        else
          *reinterpret_cast<uint4*>(sa + r * kHgPitch + c * 16) = make_uint4(0, 0, 0, 0);
        const bool okb = KN ? (k0 + r < p.K && n0 + c * 8 < p.N) : (n0 + r < p.N && k0 + c * 8 < p.K);
        const bf16* src = KN ? B + size_t(k0 + r) * p.N + n0 + c * 8 : B + size_t(n0 + r) * p.K + k0 + c * 8;
        if (okb)
          cpa16(sb + r * kHgPitch + c * 16, src);
        else
          *reinterpret_cast<uint4*>(sb + r * kHgPitch + c * 16) = make_uint4(0, 0, 0, 0);
      }
    }
    cpa_commit();
  };
  float acc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll
  for (int i = 0; i < kHgStages - 1; ++i) issue(i);
  for (int it = 0; it < iters; ++it) {
    cpa_wait<kHgStages - 2>();
    __syncthreads();
    issue(it + kHgStages - 1);
    if (m0 + warp * 16 >= p.M) continue;
    const uint32_t sa = smem_u32(smem + (it % kHgStages) * 2 * 64 * kHgPitch), sb = sa + 64 * kHgPitch;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t a[4];
      ldm_x4(sa + (warp * 16 + (lane & 15)) * kHgPitch + kk * 32 + (lane >> 4) * 16, a);
#pragma unroll
      for (int n = 0; n < 8; n += 2) {
        uint32_t b[4];
        if (KN)
          ldm_x4_t(sb + (kk * 16 + (lane >> 3 & 1) * 8 + (lane & 7)) * kHgPitch + (n + (lane >> 4)) * 16, b);
        else
          ldm_x4(sb + ((n + (lane >> 4)) * 8 + (lane & 7)) * kHgPitch + kk * 32 + (lane >> 3 & 1) * 16, b);
        mma_bf16(acc[n], a, b[0], b[1]);
        mma_bf16(acc[n + 1], a, b[2], b[3]);
      }
    }
  }
  cpa_wait<0>();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = m0 + warp * 16 + (lane >> 2) + half * 8;
    if (t >= p.M) continue;
    bf16* out = p.out + size_t(t) * p.ldo + h * p.o_head;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int c = n0 + n * 8 + (lane & 3) * 2;
      if (c >= p.N) continue;
      float x = acc[n][half * 2], y = acc[n][half * 2 + 1];
      if (!KN && p.gate != nullptr) {
        const __nv_bfloat162 g =
            *reinterpret_cast<const __nv_bfloat162*>(p.gate + size_t(t) * p.ldg + h * p.gate_head + c);
        x *= sigmoid_exact(__bfloat162float(g.x));
        y *= sigmoid_exact(__bfloat162float(g.y));
      }
      *reinterpret_cast<uint32_t*>(out + c) = pack_bf16(x, y);
    }
    if (KN && blockIdx.x == 0 && p.tail_pad > 0) {
      const bf16* src = p.tail + size_t(t) * p.lda + h * p.a_head;
      for (int i = (lane & 3); i < p.tail_pad; i += 4)
        out[p.N + i] = i < p.tail_n ? src[i] : from_f32<bf16>(0.f);
    }
  }
}

// ---- chunks: gather and attend -----------------------------------------------------------------------------------------
struct ChunkArgs {
  const int* cu_q;          // first query row of each sequence (+ end)
  const int* q_pos0;        // position of each sequence's first query
  const int* ctx_off;       // first expanded row of each sequence
  int first, last;          // sequences of the group
  int window;
};
__device__ __forceinline__ int chunk_lo(int pos0, int window) { return window > 0 ? max(0, pos0 + 1 - window) : 0; }

// One warp per expanded row.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const bf16* __restrict__ cache, RowCache rc, ChunkArgs g, int rows, int kv_rank, int rot_pad,
                     bf16* __restrict__ c_out, bf16* __restrict__ kr_out) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  int s = g.first;
  {
    int lo = g.first, hi = g.last - 1;           // last s with ctx_off[s] <= r
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (g.ctx_off[mid] <= r) lo = mid; else hi = mid - 1;
    }
    s = lo;
  }
  const int p = chunk_lo(g.q_pos0[s], g.window) + r - g.ctx_off[s];
  const int blk = rc.tables[size_t(s) * rc.max_blocks + p / rc.block_size];
  const bf16* src = cache + (blk < 0 ? 0 : blk) * rc.block_stride + size_t(p % rc.block_size) * rc.row;
  for (int c = lane; c < kv_rank / 8; c += 32)
    *reinterpret_cast<uint4*>(c_out + size_t(r) * kv_rank + c * 8) =
        blk < 0 ? make_uint4(0, 0, 0, 0) : *reinterpret_cast<const uint4*>(src + c * 8);
  for (int c = lane; c < rot_pad / 8; c += 32)
    *reinterpret_cast<uint4*>(kr_out + size_t(r) * rot_pad + c * 8) =
        blk < 0 ? make_uint4(0, 0, 0, 0) : *reinterpret_cast<const uint4*>(src + kv_rank + c * 8);
}

// CTA = (64 queries of a sequence, head), 4 warps of 16 queries; key tiles of 64 through a two-stage ring.  Keys are
// [unrotated (expanded) | rotated (shared by the heads)], values `vdim` wide (DVT blocks of 8).
constexpr int kChKeys = 64;
__host__ __device__ inline int chunk_pitch(int n) { return (n + 15) / 16 * 32 + 16; }
inline size_t chunk_smem(int qk, int vdim) {
  return size_t(64 + 2 * kChKeys) * chunk_pitch(qk) + size_t(2 * kChKeys) * chunk_pitch(vdim) + 2 * kChKeys * 4;
}

// Rows r, r + step, .. of a key tile, one 16-byte column of each; rows past the end are zero.
__device__ __forceinline__ void copy_rows(uint8_t* dst, int pitch, const bf16* src, int ld, int r, int step, int rows) {
  dst += r * pitch;
  src += size_t(r) * ld;
#pragma unroll 4
  for (; r < kChKeys; r += step) {
    if (r < rows)
      cpa16(dst, src);
    else
      *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    dst += step * pitch;
    src += size_t(step) * ld;
  }
}

template <int DVT>
__global__ void __launch_bounds__(128)
latent_chunk_kernel(const bf16* __restrict__ inp, int ld, const bf16* __restrict__ kvx, int ldkv, int v_col,
                    const bf16* __restrict__ kr_ctx, int rot_pad, RowCache rc, ChunkArgs g, bf16* __restrict__ out,
                    int ldo, const bf16* __restrict__ gate, int dim, int rot, int vdim, float scale_log2) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int s = g.first + blockIdx.z, h = blockIdx.y;
  const int q_begin = g.cu_q[s], q_len = g.cu_q[s + 1] - q_begin;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * 64;              // the longest key ranges first
  if (q0 >= q_len) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qk = dim + rot, qp = chunk_pitch(qk), vp = chunk_pitch(vdim), ksteps = (qk + 15) / 16;
  uint8_t* sq = smem;
  uint8_t* sk = sq + 64 * qp;
  uint8_t* sv = sk + 2 * kChKeys * qp;
  int* valid = reinterpret_cast<int*>(sv + 2 * kChKeys * vp);
  const int pos0 = g.q_pos0[s], lo = chunk_lo(pos0, g.window), off = g.ctx_off[s];
  const int* table = rc.tables + size_t(s) * rc.max_blocks;
  const int p_first = pos0 + q0, p_last = pos0 + min(q_len, q0 + 64) - 1;
  const int k_begin = chunk_lo(p_first, g.window), k_end = p_last + 1;
  const int count = (k_end - k_begin + kChKeys - 1) / kChKeys;
  const int qch = qk / 8, vch = vdim / 8, dch = dim / 8;

  for (int i = threadIdx.x; i < 64 * ksteps * 2; i += 128) {
    const int r = i / (ksteps * 2), c = i % (ksteps * 2);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (q0 + r < q_len && c < qch)
      v = *reinterpret_cast<const uint4*>(inp + size_t(q_begin + q0 + r) * ld + size_t(h) * qk + c * 8);
    *reinterpret_cast<uint4*>(sq + r * qp + c * 16) = v;
  }
  for (int r = threadIdx.x; r < 2 * kChKeys; r += 128) {         // pad columns of the rings
    if (qch < ksteps * 2) *reinterpret_cast<uint4*>(sk + r * qp + qch * 16) = make_uint4(0, 0, 0, 0);
    for (int c = vch; c * 16 < vp; ++c) *reinterpret_cast<uint4*>(sv + r * vp + c * 16) = make_uint4(0, 0, 0, 0);
  }
  bool whole[2] = {true, true};                  // this thread's key of the stage exists
  auto issue = [&](int i) {
    if (i < count) {
      const int st = i & 1, key0 = k_begin + i * kChKeys;
      if (threadIdx.x < kChKeys) {
        const int p = key0 + threadIdx.x;
        const bool v = p < k_end && table[p / rc.block_size] >= 0;
        valid[st * kChKeys + threadIdx.x] = v;
        if (st == 0) whole[0] = v; else whole[1] = v;
      }
      // a warp takes 16 rows; a lane keeps its 16-byte columns, so its addresses only move by whole rows
      const int rows = min(kChKeys, k_end - key0);
      const size_t x0 = size_t(off + key0 - lo);
      for (int c = lane; c < qch; c += 32) {
        const bf16* src = c < dch ? kvx + x0 * ldkv + size_t(h) * dim + c * 8 : kr_ctx + x0 * rot_pad + (c - dch) * 8;
        const int step = c < dch ? ldkv : rot_pad;
        copy_rows(sk + st * kChKeys * qp + c * 16, qp, src, step, warp, 4, rows);
      }
      if (vch <= 16) {                                           // two rows of values per pass
        const int c = lane & 15;
        if (c < vch)
          copy_rows(sv + st * kChKeys * vp + c * 16, vp, kvx + x0 * ldkv + v_col + size_t(h) * vdim + c * 8, ldkv,
                    warp * 2 + (lane >> 4), 8, rows);
      } else {
        for (int c = lane; c < vch; c += 32)
          copy_rows(sv + st * kChKeys * vp + c * 16, vp, kvx + x0 * ldkv + v_col + size_t(h) * vdim + c * 8, ldkv, warp, 4,
                    rows);
      }
    }
    cpa_commit();
  };
  float o[DVT][4];
#pragma unroll
  for (int n = 0; n < DVT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int rq = lane >> 2, cq = (lane & 3) * 2;
  const int pr0 = p_first + warp * 16 + rq;                      // positions of this thread's two query rows
  const uint32_t q_addr = smem_u32(sq) + (warp * 16 + (lane & 15)) * qp + (lane >> 4) * 16;

  issue(0);
  for (int i = 0; i < count; ++i) {
    issue(i + 1);
    cpa_wait<1>();
    const bool all_there = __syncthreads_and((i & 1) == 0 ? whole[0] : whole[1]) != 0;
    const uint32_t kb = smem_u32(sk + (i & 1) * kChKeys * qp), vb = smem_u32(sv + (i & 1) * kChKeys * vp);
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
        ldm_x4(kb + ((n + (lane >> 4)) * 8 + (lane & 7)) * qp + kk * 32 + (lane >> 3 & 1) * 16, b);
        mma_bf16(sc[n], a, b[0], b[1]);
        mma_bf16(sc[n + 1], a, b[2], b[3]);
      }
    }
    const int key0 = k_begin + i * kChKeys;
    float x[2] = {-INFINITY, -INFINITY};
    if (all_there && key0 + kChKeys - 1 <= p_first && (g.window <= 0 || p_last - key0 < g.window)) {
#pragma unroll
      for (int n = 0; n < 8; ++n) {              // every query sees every key
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          sc[n][e] *= scale_log2;
          x[e >> 1] = fmaxf(x[e >> 1], sc[n][e]);
        }
      }
    } else
#pragma unroll
    for (int n = 0; n < 8; ++n) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = n * 8 + cq + (e & 1), dist = pr0 + (e >> 1) * 8 - (key0 + c);
        const bool see = dist >= 0 && (g.window <= 0 || dist < g.window) && valid[(i & 1) * kChKeys + c] != 0;
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
        if (n * 8 < vdim) {
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
    const float inv = L > 0.f ? 1.f / L : 0.f;
    const size_t t = size_t(q_begin + r);
#pragma unroll
    for (int n = 0; n < DVT; ++n) {
      const int c = n * 8 + cq;
      if (c >= vdim) continue;
      float a = o[n][half * 2] * inv, b = o[n][half * 2 + 1] * inv;
      if (gate != nullptr) {
        const __nv_bfloat162 gv = *reinterpret_cast<const __nv_bfloat162*>(gate + t * ld + size_t(h) * vdim + c);
        a *= sigmoid_exact(__bfloat162float(gv.x));
        b *= sigmoid_exact(__bfloat162float(gv.y));
      }
      *reinterpret_cast<uint32_t*>(out + t * ldo + size_t(h) * vdim + c) = pack_bf16(a, b);
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

template <int MT, int NTW>
int launch_latent(const void* q, const void* cache, const RowCache& rc, const void* row_seq, const void* positions,
                  void* o, void* scratch, int M, int heads, int used, int kv_rank, int window, float scale, int splits,
                  Status* status, cudaStream_t st) {
  static size_t done[kMaxDevices] = {};
  auto kern = latent_attn_kernel<MT, NTW>;
  const size_t smem = latent_smem(MT, rc.row, used);
  if (int r = raise_smem(kern, smem, done)) return r;
  dim3 grid((heads + 16 * MT - 1) / (16 * MT), M, splits);
  return launch_pdl(kern, grid, dim3(kLatWarps * 32), smem, st, reinterpret_cast<const bf16*>(q),
                    reinterpret_cast<const bf16*>(cache), rc, reinterpret_cast<const int*>(row_seq),
                    reinterpret_cast<const int*>(positions), reinterpret_cast<bf16*>(o),
                    reinterpret_cast<float*>(scratch), heads, used, kv_rank, window, scale * kLog2E, splits,
                    status) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

constexpr size_t kSmemLimit = 227 * 1024;

}  // namespace
}  // namespace zse

using namespace zse;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

static RowCache row_cache(const ZseRowCache* c) {
  return RowCache{(long long)c->block_stride, c->block_size, c->row, reinterpret_cast<const int*>(c->tables),
                  c->max_blocks};
}

extern "C" int zse_latent_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, int M,
                               const ZseRowCache* c, const void* positions, const void* slots, const void* freqs,
                               const void* norm_w, int heads, int dim, int rot, int rot_dims, int kv_rank,
                               int latent_col, int gate_col, int gate_w, float eps, void* stream) {
  if (M <= 0) return 0;
  if (rot_dims % 2 || rot_dims > rot || heads <= 0 || kv_rank <= 0) return ZSE_ERR_SHAPE;
  const PrepArgs a{ld, heads, dim, rot, rot_dims, kv_rank, latent_col, gate_col, gate_w, eps};
  const size_t smem = size_t(rot_dims + kv_rank) * sizeof(float);
  if (smem > 48 * 1024) return ZSE_ERR_LIMIT;
  const int work = n_planes > 0 ? heads * (dim + rot) + gate_w : 0;
  const dim3 grid(M, 1 + (work + kPrepCols - 1) / kPrepCols), block(256);
  cudaError_t e;
  if (dtype == kBF16)
    e = launch_pdl(latent_prep_kernel<bf16>, grid, block, smem, ST(stream), reinterpret_cast<bf16*>(inp),
                   reinterpret_cast<const float*>(planes), n_planes, M, reinterpret_cast<bf16*>(c->rows), row_cache(c),
                   reinterpret_cast<const int*>(positions), reinterpret_cast<const long long*>(slots),
                   reinterpret_cast<const float*>(freqs), reinterpret_cast<const bf16*>(norm_w), a);
  else
    e = launch_pdl(latent_prep_kernel<float>, grid, block, smem, ST(stream), reinterpret_cast<float*>(inp),
                   reinterpret_cast<const float*>(planes), n_planes, M, reinterpret_cast<float*>(c->rows), row_cache(c),
                   reinterpret_cast<const int*>(positions), reinterpret_cast<const long long*>(slots),
                   reinterpret_cast<const float*>(freqs), reinterpret_cast<const float*>(norm_w), a);
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

// 1 when the tensor-core kernels take this shape (bfloat16): per-head products and latent_attn, and the chunk kernel.
extern "C" int zse_latent_mma_ok(int heads, int dim, int rot, int vdim, int kv_rank, int row) {
  return dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && kv_rank % 8 == 0 && dim > 0 && kv_rank <= 512 && row % 16 == 8 &&
         vdim <= 256 && heads > 0 && latent_smem(1, row, kv_rank + rot) <= kSmemLimit && chunk_smem(dim + rot, vdim) <= kSmemLimit;
}

extern "C" int zse_latent_attn(int dtype, const void* q_lat, const ZseRowCache* c, const void* row_seq,
                               const void* positions, void* o_lat, void* scratch, int M, int heads, int used,
                               int kv_rank, int window, float scale, int num_splits, int tensor_cores, void* status,
                               void* stream) {
  if (M <= 0) return 0;
  if (M > 65535 || num_splits < 1) return ZSE_ERR_LIMIT;
  const RowCache rc = row_cache(c);
  cudaStream_t st = ST(stream);
  if (dtype == kBF16 && tensor_cores == 1 && latent_tc_ok(rc, c->num_blocks, used, kv_rank) &&
      !((reinterpret_cast<uintptr_t>(c->rows) & 15) || (rc.block_stride & 7))) {
    const int r = launch_latent_tc(reinterpret_cast<const bf16*>(q_lat), c->rows, rc, c->num_blocks,
                                   reinterpret_cast<const int*>(row_seq), reinterpret_cast<const int*>(positions),
                                   reinterpret_cast<bf16*>(o_lat), reinterpret_cast<float*>(scratch), M, heads, used,
                                   kv_rank, window, scale, num_splits, reinterpret_cast<Status*>(status), st);
    if (r || num_splits == 1) return r;
    return launch_pdl(latent_combine_kernel, dim3(heads, M), dim3(128), 0, st, reinterpret_cast<const float*>(scratch),
                      reinterpret_cast<bf16*>(o_lat), heads, kv_rank, num_splits) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
  }
  if (dtype == kBF16 && tensor_cores) {
    if (rc.row % 16 != 8 || kv_rank % 8 || kv_rank > 512 || 64 % min(rc.block_size, 64) ||
        rc.block_size % min(rc.block_size, 64) || latent_smem(1, rc.row, used) > kSmemLimit) return ZSE_ERR_SHAPE;
    if ((reinterpret_cast<uintptr_t>(c->rows) & 15) || (rc.block_stride & 7)) return ZSE_ERR_ALIGN;
    const bool two = heads > 16 && latent_smem(2, rc.row, used) <= kSmemLimit;
    int r = ZSE_ERR_SHAPE;
#define ZSE_LAT(MT_, NTW_)                                                                                           \
  r = launch_latent<MT_, NTW_>(q_lat, c->rows, rc, row_seq, positions, o_lat, scratch, M, heads, used, kv_rank,       \
                               window, scale, num_splits, reinterpret_cast<Status*>(status), st)
    if (kv_rank <= 128) {
      if (two) ZSE_LAT(2, 2); else ZSE_LAT(1, 2);
    } else if (kv_rank <= 256) {
      if (two) ZSE_LAT(2, 4); else ZSE_LAT(1, 4);
    } else {
      if (two) ZSE_LAT(2, 8); else ZSE_LAT(1, 8);
    }
#undef ZSE_LAT
    if (r || num_splits == 1) return r;
    return launch_pdl(latent_combine_kernel, dim3(heads, M), dim3(128), 0, st, reinterpret_cast<const float*>(scratch),
                      reinterpret_cast<bf16*>(o_lat), heads, kv_rank, num_splits) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
  }
  const size_t smem = size_t(used + 4 * kv_rank + 8) * sizeof(float);
  if (smem > 48 * 1024) return ZSE_ERR_LIMIT;
  cudaError_t e;
  if (dtype == kBF16)
    e = launch_pdl(latent_attn_simple_kernel<bf16>, dim3(heads, M), dim3(128), smem, st,
                   reinterpret_cast<const bf16*>(q_lat), reinterpret_cast<const bf16*>(c->rows), rc,
                   reinterpret_cast<const int*>(row_seq), reinterpret_cast<const int*>(positions),
                   reinterpret_cast<bf16*>(o_lat), heads, used, kv_rank, window, scale);
  else
    e = launch_pdl(latent_attn_simple_kernel<float>, dim3(heads, M), dim3(128), smem, st,
                   reinterpret_cast<const float*>(q_lat), reinterpret_cast<const float*>(c->rows), rc,
                   reinterpret_cast<const int*>(row_seq), reinterpret_cast<const int*>(positions),
                   reinterpret_cast<float*>(o_lat), heads, used, kv_rank, window, scale);
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

static int launch_head_gemm(bool kn, const HeadGemmArgs& p, int heads, void* stream) {
  static size_t done[2][kMaxDevices] = {};
  dim3 grid((p.N + 63) / 64, heads, (p.M + 63) / 64);
  int r = kn ? raise_smem(head_gemm_kernel<true>, kHgSmem, done[0]) : raise_smem(head_gemm_kernel<false>, kHgSmem, done[1]);
  if (r) return r;
  const cudaError_t e = kn ? launch_pdl(head_gemm_kernel<true>, grid, dim3(128), size_t(kHgSmem), ST(stream), p)
                           : launch_pdl(head_gemm_kernel<false>, grid, dim3(128), size_t(kHgSmem), ST(stream), p);
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

// q_lat[t, h] = [q_unrotated[t, h] W_uk[h] | q_rotated[t, h]]; `inp` holds the heads [dim | rot] side by side
extern "C" int zse_latent_absorb(const void* inp, int ld, const void* uk, void* q_lat, int M, int heads, int dim, int rot,
                                 int kv_rank, int row, void* stream) {
  if (M <= 0) return 0;
  if (dim % 8 || rot % 8 || kv_rank % 8 || row % 8 || ld % 8) return ZSE_ERR_SHAPE;
  const bf16* x = reinterpret_cast<const bf16*>(inp);
  HeadGemmArgs p{};
  p.a = x;
  p.lda = ld;
  p.a_head = dim + rot;
  p.b = reinterpret_cast<const bf16*>(uk);
  p.b_head = (long long)dim * kv_rank;
  p.out = reinterpret_cast<bf16*>(q_lat);
  p.ldo = (long long)heads * row;
  p.o_head = row;
  p.M = M;
  p.N = kv_rank;
  p.K = dim;
  p.tail = x + dim;
  p.tail_n = rot;
  p.tail_pad = row - kv_rank;
  return launch_head_gemm(true, p, heads, stream);
}

// out[t, h] = (o_lat[t, h] W_uv[h]^T) * sigmoid(gate[t, h])
extern "C" int zse_latent_unabsorb(const void* o_lat, const void* uv, const void* gate, int ldg, void* out, int ldo,
                                   int M, int heads, int vdim, int kv_rank, void* stream) {
  if (M <= 0) return 0;
  if (vdim % 8 || kv_rank % 8 || ldo % 2 || ldg % 2) return ZSE_ERR_SHAPE;
  HeadGemmArgs p{};
  p.a = reinterpret_cast<const bf16*>(o_lat);
  p.lda = (long long)heads * kv_rank;
  p.a_head = kv_rank;
  p.b = reinterpret_cast<const bf16*>(uv);
  p.b_head = (long long)vdim * kv_rank;
  p.out = reinterpret_cast<bf16*>(out);
  p.ldo = ldo;
  p.o_head = vdim;
  p.M = M;
  p.N = vdim;
  p.K = kv_rank;
  p.gate = reinterpret_cast<const bf16*>(gate);
  p.ldg = ldg;
  p.gate_head = vdim;
  return launch_head_gemm(false, p, heads, stream);
}

static ChunkArgs chunk_args(const ZseChunks* g) {
  return ChunkArgs{reinterpret_cast<const int*>(g->cu_q), reinterpret_cast<const int*>(g->q_pos0),
                   reinterpret_cast<const int*>(g->ctx_off), g->first, g->last, g->window};
}

extern "C" int zse_latent_gather(const ZseRowCache* c, const ZseChunks* g, int rows, int kv_rank, int rot, void* c_out,
                                 void* kr_out, void* stream) {
  if (rows <= 0) return 0;
  if (kv_rank % 8 || rot % 8) return ZSE_ERR_SHAPE;
  return launch_pdl(latent_gather_kernel, dim3((rows + 7) / 8), dim3(256), 0, ST(stream),
                    reinterpret_cast<const bf16*>(c->rows), row_cache(c), chunk_args(g), rows, kv_rank, rot,
                    reinterpret_cast<bf16*>(c_out), reinterpret_cast<bf16*>(kr_out)) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_latent_chunk(const void* inp, int ld, const void* kvx, int ldkv, int v_col, const void* kr_ctx,
                                const ZseRowCache* c, const ZseChunks* g, int max_q, void* out, int ldo,
                                const void* gate, int heads, int dim, int rot, int vdim, float scale, void* stream) {
  if (g->last <= g->first || max_q <= 0) return 0;
  if (dim % 8 || rot % 8 || vdim % 8 || vdim > 256 || ld % 8 || ldkv % 8 || v_col % 8 || ldo % 2) return ZSE_ERR_SHAPE;
  const size_t smem = chunk_smem(dim + rot, vdim);
  if (smem > kSmemLimit) return ZSE_ERR_LIMIT;
  dim3 grid((max_q + 63) / 64, heads, g->last - g->first);
  static size_t done[4][kMaxDevices] = {};
#define ZSE_CH(I_, DVT_)                                                                                               \
  {                                                                                                                    \
    auto kern = latent_chunk_kernel<DVT_>;                                                                             \
    if (int r = raise_smem(kern, smem, done[I_])) return r;                                                            \
    return launch_pdl(kern, grid, dim3(128), smem, ST(stream), reinterpret_cast<const bf16*>(inp), ld,                 \
                      reinterpret_cast<const bf16*>(kvx), ldkv, v_col, reinterpret_cast<const bf16*>(kr_ctx), rot,     \
                      row_cache(c), chunk_args(g), reinterpret_cast<bf16*>(out), ldo,                                  \
                      reinterpret_cast<const bf16*>(gate), dim, rot, vdim, scale * kLog2E) == cudaSuccess              \
               ? 0                                                                                                     \
               : ZSE_ERR_LAUNCH;                                                                                       \
  }
  if (vdim <= 32) ZSE_CH(0, 4)
  if (vdim <= 64) ZSE_CH(1, 8)
  if (vdim <= 128) ZSE_CH(2, 16)
  ZSE_CH(3, 32)
#undef ZSE_CH
}
