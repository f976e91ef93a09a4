// Latent attention of decoding tokens on the 5th-generation tensor cores (bfloat16).
//
// CTA = (16 or 32 heads, token, key split).  Every head of the group uses the same cached rows, as keys and as values, so
// both products put the rows on the wide side of the MMA and the heads on the narrow one:
//
//   S^T [keys, heads]      = K [64 keys, row] . Q^T          A = cached rows, K-major;  B = queries
//   O^T [latent, heads]   += V^T [latent, 64 keys] . P^T     A = the SAME shared-memory tile, MN-major (the latent part of
//                                                            a row is the value);  B = softmax weights
//
// Both accumulators live in TMEM.  A tile of 64 keys is a set of 64-column panels with the 128-byte swizzle, each brought by
// one TMA box per cache block through the block table.  The MMA's 128 rows are more than the 64 keys of a tile: its upper
// half multiplies whatever follows the panel in shared memory and is never read.  Roles: a TMA producer, two MMA
// issuers for the scores (even and odd k steps, added when they are read) and one for the values, four softmax warps.  The products of tile i + 1 with the queries run while tile i is weighed; softmax weights
// are split into two bfloat16 terms that stand side by side as columns of P^T (their results are added at the end); the running maximum is only moved (and O rescaled) when a score exceeds it by more than 2^8.  Every wait is
// bounded and reports through the status word.
#include <mutex>
#include <unordered_map>

#include "api.h"
#include "gemm_common.cuh"
#include "latent.cuh"

namespace zse {
namespace {

constexpr int kTcKeys = 64;
constexpr int kTcPanelBytes = kTcKeys * 128;
constexpr int kTcMaxPanels = 9;                 // rows of up to 576 columns
constexpr int kTcThreads = 288;                 // warp 0 producer, 1 and 2 scores, 3 and 8 values, 4..7 softmax
constexpr float kTcSlack = 8.f;                 // log2 of how far a score may exceed the reference

struct LatentTcArgs {
  const bf16* q_lat;
  RowCache rc;
  const int *row_seq, *positions;
  bf16* o_lat;
  float* scratch;
  int heads, used, kv_rank, window, num_splits;
  float scale_log2;
  int one_box;                                  // a block's piece of a tile is one TMA box (all panels)
  Status* status;
};

struct LatentTcBars {
  uint64_t full[2], s_ready[2], p_ready[2], pv_done[2], q_ready;
  uint32_t tmem_base;
  int abort_flag;
};

template <int N>
struct LatentTcCfg {
  static constexpr int kSPitch = kTcKeys + 4;   // floats
  static constexpr int kTmemCols = N == 16 ? 256 : 512;
  static constexpr int kOCol = 4 * N;           // O^T blocks [2 terms of P][N] after two S^T buffers of two parts
  __host__ __device__ static int q_bytes(int panels) { return panels * N * 128; }
  __host__ __device__ static size_t smem(int panels) {
    return 1024 + size_t(2) * panels * kTcPanelBytes + q_bytes(panels) + 4 * N * 128 + size_t(N) * kSPitch * 4 +
           3 * N * 4 + 64 + sizeof(LatentTcBars);
  }
};

__device__ __forceinline__ void tma_load_3d(void* dst, const void* map, int x, int y, int z, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(
          smem_u32(dst)),
      "l"(map), "r"(x), "r"(y), "r"(z), "r"(smem_u32(bar))
      : "memory");
}
__device__ __forceinline__ void tma_load_4d(void* dst, const void* map, int x, int y, int p, int z, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];" ::"r"(
          smem_u32(dst)),
      "l"(map), "r"(x), "r"(y), "r"(p), "r"(z), "r"(smem_u32(bar))
      : "memory");
}
// MN-major operand, 128-byte swizzle: rows of the K dimension hold 64 MN elements, eight rows per 1024 bytes, the next 64 MN
// elements one panel on.
__device__ __forceinline__ uint64_t make_desc_panel_mn(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= uint64_t((smem_addr >> 4) & 0x3FFF);
  d |= uint64_t(kTcPanelBytes >> 4) << 16;
  d |= uint64_t(1024 >> 4) << 32;
  d |= uint64_t(1) << 46;
  d |= uint64_t(2) << 61;
  return d;
}
// Barrier of the softmax warps; true on every thread when `ok` was true on all of them.
__device__ __forceinline__ bool softmax_agree(bool ok) {
  uint32_t all;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.and.pred q, 1, 128, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(all)
      : "r"(uint32_t(ok))
      : "memory");
  return all != 0;
}
__device__ __forceinline__ bool softmax_any(bool v) { return !softmax_agree(!v); }

// N consecutive 32-bit columns of the thread's TMEM lane
template <int N>
__device__ __forceinline__ void tmem_load(uint32_t* r, uint32_t addr) {
#pragma unroll
  for (int c = 0; c < N; c += 16) ZSE_TMEM_LD_X16((r + c), addr + c);
  tc_wait_ld();
}

template <int N>
__global__ void __launch_bounds__(kTcThreads, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap map, const LatentTcArgs a) {
  using Cfg = LatentTcCfg<N>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int panels = (a.used + 63) / 64, ksteps = (a.used + 15) / 16, blocks = (a.kv_rank + 127) / 128;
  const int stage_bytes = panels * kTcPanelBytes;
  uint8_t* sk = smem;                                            // [2 stages][panels][64 keys][128 bytes]
  uint8_t* sq = sk + 2 * stage_bytes;                            // [panels][N heads][128 bytes]
  uint8_t* sp = sq + Cfg::q_bytes(panels);                       // [2][hi, lo][N heads][128 bytes]
  float* ss = reinterpret_cast<float*>(sp + 4 * N * 128);        // scores [N][kSPitch]
  float* corr = ss + N * Cfg::kSPitch;                           // [N]
  float* ref_out = corr + N;                                     // [N] reference, [N] sum
  LatentTcBars* bars = reinterpret_cast<LatentTcBars*>(
      (reinterpret_cast<uintptr_t>(ref_out + 2 * N) + 15) & ~uintptr_t(15));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->full[i], 1);
      mbar_init(&bars->s_ready[i], ksteps > 1 ? 2 : 1);
      mbar_init(&bars->p_ready[i], 128);
      mbar_init(&bars->pv_done[i], blocks > 1 ? 2 : 1);
    }
    mbar_init(&bars->q_ready, 128);
    bars->abort_flag = 0;
    mbar_fence_init();
    prefetch_tmap(&map);
  }
  if (warp == 2) {
    tmem_alloc(&bars->tmem_base, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = bars->tmem_base;
  volatile int* abort_flag = &bars->abort_flag;
  pdl_wait();
  const int h0 = blockIdx.x * N, t = blockIdx.y, split = blockIdx.z;
  const int nh = min(N, a.heads - h0);
  const int seq = a.row_seq != nullptr ? a.row_seq[t] : t, pos = a.positions[t];
  const int* table = a.rc.tables + size_t(seq) * a.rc.max_blocks;
  const int lo = a.window > 0 ? max(0, pos + 1 - a.window) : 0;
  const int tile0 = lo / kTcKeys, n_tiles = pos / kTcKeys + 1 - tile0;
  const int per = (n_tiles + a.num_splits - 1) / a.num_splits;
  const int first = tile0 + split * per;
  const int count = max(0, min(tile0 + n_tiles, first + per) - first);
  const int piece = min(a.rc.block_size, kTcKeys);

  if (warp == 0) {
    // keys that are not copied (a hole, what follows the newest token) weigh 0, but what lies in their place has to be finite
    bool missing = false;
    for (int i = lane; i < count * (kTcKeys / piece); i += 32) {
      const int key = first * kTcKeys + i * piece;
      missing |= key > pos || table[key / a.rc.block_size] < 0;
    }
    if (__any_sync(0xffffffffu, missing)) {
      for (int i = lane; i < 2 * stage_bytes / 16; i += 32) reinterpret_cast<uint4*>(sk)[i] = make_uint4(0, 0, 0, 0);
      fence_proxy_async_smem();
      __syncwarp();
    }
    int issued = 0;
    for (int i = 0; i < count; ++i) {
      const int st = i & 1, key0 = (first + i) * kTcKeys;
      int blk = -1;                                              // looked up while the stage is still in use
      if (lane * piece < kTcKeys && key0 + lane * piece <= pos) blk = table[(key0 + lane * piece) / a.rc.block_size];
      const bool go = i < 2 || mbar_wait_spin(&bars->pv_done[st], ((i >> 1) - 1) & 1, abort_flag, a.status, 91, i);
      if (!__all_sync(0xffffffffu, go)) break;
      const unsigned have = __ballot_sync(0xffffffffu, blk >= 0);
      if (lane == 0) mbar_arrive_expect_tx(&bars->full[st], __popc(have) * piece * panels * 128);
      __syncwarp();
      if (a.one_box) {                                           // a whole block's tile: lane 0 only (piece = tile)
        if (blk >= 0)
          tma_load_4d(sk + st * stage_bytes, &map, 0, key0 % a.rc.block_size, 0, blk, &bars->full[st]);
      } else {
        for (int j = 0; j * piece < kTcKeys; ++j) {              // lane p brings panel p of every block
          const int b = __shfl_sync(0xffffffffu, blk, j);
          if (b >= 0 && lane < panels)
            tma_load_3d(sk + st * stage_bytes + lane * kTcPanelBytes + j * piece * 128, &map, lane * 64,
                        (key0 + j * piece) % a.rc.block_size, b, &bars->full[st]);
        }
      }
      issued = i + 1;
    }
    if (*abort_flag && lane == 0) {
      for (int i = max(0, issued - 2); i < issued; ++i) {        // the copies in flight land before the CTA leaves
        SpinClock clock;
        while (!mbar_try_wait(&bars->full[i & 1], (i >> 1) & 1) && !clock.expired(0xFF)) {
        }
      }
    }
  } else if (warp == 1 || warp == 2) {
    if (lane == 0) {                                             // S^T = K Q^T, every other k step each
      constexpr uint32_t idesc = make_idesc_f16(128, N, 1);
      const bool go = mbar_wait_spin(&bars->q_ready, 0, abort_flag, a.status, 90, 0);
      for (int i = 0; go && i < count && warp - 1 < ksteps; ++i) {
        if (!mbar_wait_spin(&bars->full[i & 1], (i >> 1) & 1, abort_flag, a.status, 92, i)) break;
        // the scores of tile i - 2 have been read
        if (i >= 2 && !mbar_wait_spin(&bars->p_ready[i & 1], ((i >> 1) - 1) & 1, abort_flag, a.status, 93, i)) break;
        tc_fence_after_sync();
        const uint64_t k = make_desc_sw128(smem_u32(sk) + (i & 1) * stage_bytes), q = make_desc_sw128(smem_u32(sq));
#pragma unroll 4
        for (int kk = warp - 1; kk < ksteps; kk += 2)            // addresses are in units of 16 bytes
          umma_ss(tmem + (i & 1) * 2 * N + (warp - 1) * N, k + (kk >> 2) * (kTcPanelBytes / 16) + (kk & 3) * 2,
                  q + (kk >> 2) * (N * 8) + (kk & 3) * 2, idesc, kk > 1);
        tc_commit(&bars->s_ready[i & 1]);
      }
    }
  } else if (warp == 3 || warp == 8) {
    const int half = warp == 3 ? 0 : 1;                          // every other block of 128 latent columns
    if (lane == 0 && half < blocks) {                            // O^T += V^T P^T; both terms of P side by side
      constexpr uint32_t idesc = make_idesc_f16(128, 2 * N, 1) | (1u << 15);            // A is MN-major
      for (int i = 0; i < count; ++i) {
        if (!mbar_wait_spin(&bars->p_ready[i & 1], (i >> 1) & 1, abort_flag, a.status, 94, i)) break;
        if (!mbar_wait_spin(&bars->full[i & 1], (i >> 1) & 1, abort_flag, a.status, 99, i)) break;
        tc_fence_after_sync();
        const uint64_t v = make_desc_panel_mn(smem_u32(sk) + (i & 1) * stage_bytes),
                       p = make_desc_sw128(smem_u32(sp) + (i & 1) * 2 * N * 128);
        for (int b = half; b < blocks; b += 2)
#pragma unroll
          for (int j = 0; j < kTcKeys / 16; ++j)
            umma_ss(tmem + Cfg::kOCol + b * 2 * N, v + b * (kTcPanelBytes / 8) + j * 128, p + j * 2, idesc, (i | j) != 0);
        tc_commit(&bars->pv_done[i & 1]);
      }
    }
  } else if (warp >= 4) {
    constexpr int kPerHead = 128 / N, kMine = kTcKeys / kPerHead;        // threads per head, keys per thread (8 or 16)
    const int tid = threadIdx.x - 128, quarter = warp & 3;
    const int head = tid / kPerHead, sub = tid % kPerHead;
    const uint32_t lane_base = tmem + (uint32_t(quarter * 32) << 16);
    const int chunks = a.rc.row / 8;
    for (int h = tid >> 3; h < N; h += 16) {                     // queries; zero beyond the heads and the row
      const uint4* src = reinterpret_cast<const uint4*>(a.q_lat + (size_t(t) * a.heads + h0 + min(h, nh - 1)) * a.rc.row);
      const int c0 = tid & 7;
#pragma unroll
      for (int p = 0; p < kTcMaxPanels; ++p) {
        const int c = p * 8 + c0;
        if (p < panels)
          *reinterpret_cast<uint4*>(sq + p * N * 128 + h * 128 + ((c0 ^ (h & 7)) << 4)) =
              h < nh && c < chunks ? src[c] : make_uint4(0, 0, 0, 0);
      }
    }
    fence_proxy_async_smem();
    mbar_arrive(&bars->q_ready);
    float ref = -INFINITY, sum = 0.f;
    bool ok = true;
    for (int i = 0; i < count; ++i) {
      const int k = quarter * 32 + lane, key = (first + i) * kTcKeys + k;
      const bool see = quarter < 2 && key >= lo && key <= pos && table[key / a.rc.block_size] >= 0;
      ok = __all_sync(0xffffffffu, mbar_wait_spin(&bars->s_ready[i & 1], (i >> 1) & 1, abort_flag, a.status, 95, i));
      if (ok && quarter < 2) {                                   // lanes 0..63 of S^T are the tile's keys
        tc_fence_after_sync();
        uint32_t r[N], odd[N];
        tmem_load<N>(r, lane_base + (i & 1) * 2 * N);
        if (ksteps > 1) {
          tmem_load<N>(odd, lane_base + (i & 1) * 2 * N + N);
#pragma unroll
          for (int h = 0; h < N; ++h) r[h] = __float_as_uint(__uint_as_float(r[h]) + __uint_as_float(odd[h]));
        }
#pragma unroll
        for (int h = 0; h < N; ++h)
          ss[h * Cfg::kSPitch + k] = see ? __uint_as_float(r[h]) * a.scale_log2 : -INFINITY;
        tc_fence_before_sync();
      }
      ok = softmax_agree(ok);
      if (!ok) break;
      float s[kMine], mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < kMine; c += 4) {
        const float4 v = *reinterpret_cast<const float4*>(ss + head * Cfg::kSPitch + sub * kMine + c);
        s[c] = v.x;
        s[c + 1] = v.y;
        s[c + 2] = v.z;
        s[c + 3] = v.w;
        mx = fmaxf(fmaxf(fmaxf(mx, v.x), fmaxf(v.y, v.z)), v.w);
      }
#pragma unroll
      for (int d = 1; d < kPerHead; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const bool move = mx > ref + kTcSlack || (ref == -INFINITY && mx > ref);
      const float next = move ? mx : ref;
      const float factor = ref == -INFINITY ? 0.f : exp2f(ref - next);   // 1 when the reference stays
      ref = next;
      sum *= factor;
      if (sub == 0) corr[head] = move ? factor : 1.f;
      const bool rescale = softmax_any(move) && i > 0;
      if (rescale) {                                             // O^T so far is relative to the old references
        ok = mbar_wait_spin(&bars->pv_done[(i - 1) & 1], ((i - 1) >> 1) & 1, abort_flag, a.status, 96, i);
        ok = softmax_agree(ok);
        if (!ok) break;
        tc_fence_after_sync();
        for (int b = 0; b < blocks; ++b) {
#pragma unroll
          for (int c = 0; c < 2 * N; c += 16) {
            uint32_t r[16];
            const uint32_t addr = lane_base + Cfg::kOCol + b * 2 * N + c;
            ZSE_TMEM_LD_X16(r, addr);
            tc_wait_ld();
#pragma unroll
            for (int e = 0; e < 16; ++e) r[e] = __float_as_uint(__uint_as_float(r[e]) * corr[(c & (N - 1)) + e]);
            ZSE_TMEM_ST_X16(addr, r);
          }
        }
        tc_wait_st();
        tc_fence_before_sync();
      } else if (i >= 2) {                                       // the weights of tile i - 2 have been used
        ok = mbar_wait_spin(&bars->pv_done[i & 1], ((i >> 1) - 1) & 1, abort_flag, a.status, 97, i);
        ok = softmax_agree(ok);
        if (!ok) break;
      }
      const float base = ref == -INFINITY ? 0.f : ref;
      uint8_t* p = sp + (i & 1) * 2 * N * 128 + head * 128;
#pragma unroll
      for (int c = 0; c < kMine; c += 8) {
        float w[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          w[e] = ex2(s[c + e] - base);
          sum += w[e];
        }
        const int chunk = ((sub * kMine + c) >> 3) ^ (head & 7);
        *reinterpret_cast<uint4*>(p + (chunk << 4)) =
            make_uint4(pack_bf16(w[0], w[1]), pack_bf16(w[2], w[3]), pack_bf16(w[4], w[5]), pack_bf16(w[6], w[7]));
        *reinterpret_cast<uint4*>(p + N * 128 + (chunk << 4)) =
            make_uint4(pack_bf16_rest(w[0], w[1]), pack_bf16_rest(w[2], w[3]), pack_bf16_rest(w[4], w[5]),
                       pack_bf16_rest(w[6], w[7]));
      }
      fence_proxy_async_smem();
      mbar_arrive(&bars->p_ready[i & 1]);
    }
    if (ok && count > 0) {
      const int i = count - 1;
      ok = mbar_wait(&bars->pv_done[i & 1], (i >> 1) & 1, abort_flag, a.status, 98, i);
    }
#pragma unroll
    for (int d = 1; d < kPerHead; d <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
    if (sub == 0) {
      ref_out[head] = ref;
      ref_out[N + head] = a.num_splits > 1 ? sum : sum > 0.f ? 1.f / sum : 0.f;
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (*abort_flag == 0 && warp < 8) {            // eight warps write the blocks: two for each quarter of the lanes
    tc_fence_after_sync();
    const int quarter = warp & 3;
    const size_t hh0 = size_t(t) * a.heads + h0;
    for (int b = warp >> 2; b < blocks; b += 2) {
      uint32_t r[N];
      if (count > 0) {
        uint32_t rest[N];
        const uint32_t addr = tmem + (uint32_t(quarter * 32) << 16) + Cfg::kOCol + b * 2 * N;
        tmem_load<N>(r, addr);
        tmem_load<N>(rest, addr + N);
#pragma unroll
        for (int h = 0; h < N; ++h) r[h] = __float_as_uint(__uint_as_float(r[h]) + __uint_as_float(rest[h]));
      } else {
#pragma unroll
        for (int h = 0; h < N; ++h) r[h] = 0u;
      }
      const int c = b * 128 + quarter * 32 + lane;
      if (c < a.kv_rank) {
        if (a.num_splits == 1) {
          bf16* out = a.o_lat + hh0 * a.kv_rank + c;
#pragma unroll
          for (int h = 0; h < N; ++h)
            if (h < nh) out[size_t(h) * a.kv_rank] = from_f32<bf16>(__uint_as_float(r[h]) * ref_out[N + h]);
        } else {
          const int step = a.num_splits * (a.kv_rank + 2);
          float* out = a.scratch + (hh0 * a.num_splits + split) * (a.kv_rank + 2) + c;
#pragma unroll
          for (int h = 0; h < N; ++h)
            if (h < nh) out[size_t(h) * step] = __uint_as_float(r[h]);
        }
      }
    }
    if (a.num_splits > 1 && int(threadIdx.x) < nh) {
      float* part = a.scratch + ((hh0 + threadIdx.x) * a.num_splits + split) * (a.kv_rank + 2) + a.kv_rank;
      part[0] = ref_out[threadIdx.x];
      part[1] = ref_out[N + threadIdx.x];
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 2) tmem_dealloc(tmem, Cfg::kTmemCols);
}

template <int N>
int launch_tc(const CUtensorMap& map, const LatentTcArgs& a, int M, cudaStream_t st) {
  const int panels = (a.used + 63) / 64;
  const size_t smem = LatentTcCfg<N>::smem(panels);
  static size_t granted[kMaxDevices] = {};
  const int slot = current_device_slot();
  auto kern = latent_tc_kernel<N>;
  if (smem > granted[slot]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)) != cudaSuccess)
      return ZSE_ERR_LAUNCH;
    granted[slot] = smem;
  }
  return launch_pdl(kern, dim3((a.heads + N - 1) / N, M, a.num_splits), dim3(kTcThreads), smem, st, map, a) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

}  // namespace

bool latent_tc_ok(const RowCache& rc, int num_blocks, int used, int kv_rank) {
  const int panels = (used + 63) / 64;
  return panels <= kTcMaxPanels && kv_rank % 8 == 0 && kv_rank <= 512 && rc.row % 8 == 0 && num_blocks > 0 &&
         (rc.block_size == 16 || rc.block_size == 32 || rc.block_size % kTcKeys == 0) &&
         (kv_rank + 127) / 128 * 2 <= panels + 2 && LatentTcCfg<32>::smem(panels) <= 227 * 1024;
}

int launch_latent_tc(const bf16* q_lat, const void* rows, const RowCache& rc, int num_blocks, const int* row_seq,
                     const int* positions, bf16* o_lat, float* scratch, int M, int heads, int used, int kv_rank, int window,
                     float scale, int num_splits, Status* status, cudaStream_t st) {
  CUtensorMap map;
  // all panels in one box where they are whole (nothing past a row's end is touched) and a tile lies in one block
  const int panels = (used + 63) / 64;
  const bool one_box = used % 64 == 0 && rc.block_size % kTcKeys == 0;
  if (int r = get_tmap_rows3(rows, num_blocks, rc.block_size, rc.row, rc.block_stride,
                             rc.block_size < kTcKeys ? rc.block_size : kTcKeys, one_box ? panels : 0, &map))
    return r;
  LatentTcArgs a{q_lat, rc, row_seq, positions, o_lat, scratch, heads, used, kv_rank, window, num_splits,
                 scale * kLog2E, one_box, status};
  return heads <= 16 ? launch_tc<16>(map, a, M, st) : launch_tc<32>(map, a, M, st);
}

}  // namespace zse
