// Tiles of queries against cached keys on the tcgen05 tensor cores: keys and values up to 128 wide, chunk or window masks,
// grouped-query, bfloat16 (heads.cu has the other forms).
//
// One CTA owns 128 query rows of one head of one sequence and walks the keys its rows see in tiles of 128, with the pipeline
// of attention_tc.cu (a loader warp, an MMA issuer, 128 softmax threads that own a row each, two CTAs per SM):
//   S = Q K^T     both from shared memory (TMA boxes of 64 columns x 16, 32 or 64 tokens through the block table; columns past
//                 a key's width are the tensor map's zero fill)
//   softmax       row maximum, then exp2 of the scores (soft-capped first, where a cap is set); the reference maximum moves
//                 only when a row outgrew it by 2^8
//   O += P V      P from TMEM in TWO bfloat16 terms, the weight and what rounding took from it, 64 columns each: together they
//                 take the place of the 128 columns of scores; V is an MN-major operand as it lies in the cache
// Tiles start at a multiple of the box, at or before the first key that the tile's first query sees; tiles of the tokens that
// are always kept, or of the means of older blocks of tokens, come before them.
// Every wait is bounded; on a failure the loader waits for its copies and the CTA frees its TMEM and leaves.
#include <cuda.h>

#include <type_traits>

#include "api.h"
#include "gemm_common.cuh"
#include "heads.cuh"

namespace zse {
namespace {

constexpr int kHtRows = 128, kHtKeys = 128;
constexpr int kHtThreads = 192;                  // warps 0-3 softmax, warp 4 loader, warp 5 MMA issuer
constexpr int kHtPanel = 128 * 128;              // bytes of 128 rows of 64 columns

struct HtBars {
  uint64_t q_full, k_full, v_full, v_empty, s_full, p_full;
  uint32_t tmem_base;
  int abort_flag;
};

struct HtArgs {
  Heads h;
  const int *cu_q, *q_pos0;
  int first;
  bf16* out;
  int ldo;
  const bf16* gate;
  int ld;
  int box_rows, k_panels, v_panels;
  Status* status;
};

__device__ __forceinline__ void ht_load(void* dst, const void* map, int x, int y, int z, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(
          smem_u32(dst)),
      "l"(map), "r"(x), "r"(y), "r"(z), "r"(smem_u32(bar))
      : "memory");
}
// MN-major operand, 128-byte swizzle: rows of the K dimension hold 64 MN elements, eight rows per 1024 bytes, the next 64 MN
// elements one panel on.
__device__ __forceinline__ uint64_t ht_desc_mn(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= uint64_t((smem_addr >> 4) & 0x3FFF);
  d |= uint64_t(kHtPanel >> 4) << 16;
  d |= uint64_t(1024 >> 4) << 32;
  d |= uint64_t(1) << 46;
  d |= uint64_t(2) << 61;
  return d;
}

// A cap bounds the scores: with one of up to kHtFixedCap the cap itself is the reference maximum of every row (weights down to
// exp(-2 cap) are ordinary fp32 numbers), and a tile is read once.
enum HtMode { kHtPlain = 0 /* no kept tokens, no cap */, kHtNoCap = 1, kHtCap = 2, kHtFixed = 3, kHtPooled = 4 };
constexpr float kHtFixedCap = 40.f;

template <int MODE>
__global__ void __launch_bounds__(kHtThreads, 2)
heads_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                const __grid_constant__ CUtensorMap map_v, const HtArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + a.k_panels * kHtPanel;
  uint8_t* v_s = k_s + a.k_panels * kHtPanel;
  HtBars* bars = reinterpret_cast<HtBars*>(v_s + a.v_panels * kHtPanel);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // the longest key ranges first
  const int qt = int(gridDim.x) - 1 - int(blockIdx.x), head = blockIdx.y, seq = a.first + blockIdx.z;
  pdl_launch_dependents();
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  if (qt * kHtRows >= q_len) return;             // before any barrier or TMEM use: the whole CTA leaves
  const int kvh = head / (a.h.heads / a.h.kv_heads);
  const int p_first = a.q_pos0[seq] + qt * kHtRows, p_last = a.q_pos0[seq] + min(q_len, qt * kHtRows + kHtRows) - 1;
  const int br = a.box_rows;
  const int k_begin = a.h.first_seen(p_first) / br * br, k_end = p_last + 1;
  // kept tokens before the others, in whole boxes; or the means that the tile's last query sees
  const int kept_end = MODE == kHtPlain    ? 0
                       : MODE == kHtPooled ? a.h.means_seen(p_last)
                                           : min(k_begin, (a.h.keep + br - 1) / br * br);
  const int kept = (kept_end + kHtKeys - 1) / kHtKeys, n_tiles = kept + (k_end - k_begin + kHtKeys - 1) / kHtKeys;
  auto key_of = [&](int t) { return MODE != kHtPlain && t < kept ? t * kHtKeys : k_begin + (t - kept) * kHtKeys; };
  auto end_of = [&](int t) { return MODE != kHtPlain && t < kept ? kept_end : k_end; };
  const int* table = a.h.tables + size_t(seq) * a.h.max_blocks;
  auto block_at = [&](int t, int tok) { return table[(MODE == kHtPooled && t < kept ? a.h.means_at : 0) + a.h.block_of(tok)]; };

  if (threadIdx.x == 0) {
    mbar_init(&bars->q_full, 1);
    mbar_init(&bars->k_full, 1);
    mbar_init(&bars->v_full, 1);
    mbar_init(&bars->v_empty, 1);
    mbar_init(&bars->s_full, 1);
    mbar_init(&bars->p_full, 128);
    bars->abort_flag = 0;
    mbar_fence_init();
    prefetch_tmap(&map_q);
    prefetch_tmap(&map_k);
    prefetch_tmap(&map_v);
  }
  // V must never hold a NaN bit pattern where a weight is zero (0 * NaN): clear it once; afterwards it only ever holds cache
  // contents
  for (int i = threadIdx.x; i < a.v_panels * kHtPanel / 16; i += kHtThreads)
    reinterpret_cast<uint4*>(v_s)[i] = make_uint4(0, 0, 0, 0);
  fence_proxy_async_smem();
  if (warp == 5) {
    tmem_alloc(&bars->tmem_base, 256);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tm_s = bars->tmem_base, tm_o = tm_s + 128;      // scores, then the two terms of P; O
  volatile int* abort_flag = &bars->abort_flag;
  pdl_wait();                                    // queries, gates and cache rows come from the kernels before

  if (warp == 4) {
    // loader: lane 2 g + panel looks up group g of the NEXT tile while the current one is in flight, and issues one box of
    // keys and one of values
    if (lane == 0) {
      mbar_arrive_expect_tx(&bars->q_full, uint32_t(a.k_panels) * kHtPanel);
      for (int p = 0; p < a.k_panels; ++p)
        tma_load_2d(q_s + p * kHtPanel, &map_q, head * a.h.dim + p * 64, q_begin + qt * kHtRows, &bars->q_full);
    }
    const int n_groups = kHtKeys / br, g = lane >> 1, panel = lane & 1;
    const uint32_t box_bytes = uint32_t(br) * 128u;
    auto group_block = [&](int t) {              // block of group g of tile t; -1: a hole, or past the end
      const int tok = key_of(t) + g * br;
      return (g < n_groups && t < n_tiles && tok < end_of(t)) ? block_at(t, tok) : -1;
    };
    int next = group_block(0), issued_k = 0, issued_v = 0;
    uint32_t ph = 1;                             // "empty" barriers: the first wait passes
    for (int t = 0; t < n_tiles; ++t) {
      const int block = next;
      const int tok = key_of(t) + g * br;
      const int y = kvh * a.h.block_size + a.h.in_block(tok);
      const bool load_k = block >= 0 && panel < a.k_panels, load_v = block >= 0 && panel < a.v_panels;
      const uint32_t n_k = __popc(__ballot_sync(0xffffffffu, load_k)), n_v = __popc(__ballot_sync(0xffffffffu, load_v));
      next = group_block(t + 1);
      // the K slot is free once Q K^T of the tile before is complete
      bool ok = true;
      if (lane == 0 && t > 0) ok = mbar_wait_spin(&bars->s_full, ph, abort_flag, a.status, 91, t);
      if (!__shfl_sync(0xffffffffu, ok, 0)) break;
      if (lane == 0) mbar_arrive_expect_tx(&bars->k_full, n_k * box_bytes);
      __syncwarp();
      if (load_k) ht_load(k_s + panel * kHtPanel + g * box_bytes, &map_k, panel * 64, y, block, &bars->k_full);
      issued_k = t + 1;
      __syncwarp();
      if (lane == 0) ok = mbar_wait_spin(&bars->v_empty, ph, abort_flag, a.status, 92, t);
      if (!__shfl_sync(0xffffffffu, ok, 0)) break;
      if (lane == 0) mbar_arrive_expect_tx(&bars->v_full, n_v * box_bytes);
      __syncwarp();
      if (load_v) ht_load(v_s + panel * kHtPanel + g * box_bytes, &map_v, panel * 64, y, block, &bars->v_full);
      issued_v = t + 1;
      __syncwarp();
      ph ^= 1;
    }
    if (lane == 0 && *abort_flag) {              // the copies in flight land before the CTA leaves
      const uint64_t t0 = globaltimer_ns();
      auto drain = [&](uint64_t* bar, uint32_t parity) {
        while (!mbar_try_wait(bar, parity) && globaltimer_ns() - t0 < kWaitLimitNs) {
        }
      };
      drain(&bars->q_full, 0);
      if (issued_k > 0) drain(&bars->k_full, uint32_t(issued_k - 1) & 1u);
      if (issued_v > 0) drain(&bars->v_full, uint32_t(issued_v - 1) & 1u);
    }
  } else if (warp == 5) {
    if (lane == 0) {
      const int n16 = (a.h.vdim + 15) / 16 * 16, ksteps = (a.h.dim + 15) / 16;
      const uint32_t idesc_qk = make_idesc_f16(kHtRows, kHtKeys, 1);
      const uint32_t idesc_pv = make_idesc_f16(kHtRows, n16, 1) | (1u << 16);        // B is MN-major
      const uint64_t q_desc = make_desc_sw128(smem_u32(q_s)), k_desc = make_desc_sw128(smem_u32(k_s));
      bool ok = mbar_wait_spin(&bars->q_full, 0, abort_flag, a.status, 93, 0);
      uint32_t ph = 0;
      for (int t = 0; t < n_tiles && ok; ++t) {
        if (!mbar_wait_spin(&bars->k_full, ph, abort_flag, a.status, 94, t)) break;
        // the weights of the tile before live in the columns this product overwrites: let P V finish reading them
        if (t > 0 && !mbar_wait_spin(&bars->v_empty, ph ^ 1, abort_flag, a.status, 95, t)) break;
        tc_fence_after_sync();
        for (int j = 0; j < ksteps; ++j) {
          const uint64_t adv = uint64_t((j >> 2) * (kHtPanel >> 4) + (j & 3) * 2);
          umma_ss(tm_s, q_desc + adv, k_desc + adv, idesc_qk, j != 0);
        }
        tc_commit(&bars->s_full);                // S complete, and every MMA before it
        if (!mbar_wait_spin(&bars->v_full, ph, abort_flag, a.status, 96, t)) break;
        if (!mbar_wait_spin(&bars->p_full, ph, abort_flag, a.status, 97, t)) break;
        tc_fence_after_sync();
#pragma unroll
        for (int j = 0; j < 8; ++j) {            // 16 keys per step: two groups of eight cache rows
          const uint64_t v_desc = ht_desc_mn(smem_u32(v_s) + j * 2048);
          umma_ts(tm_o, tm_s + j * 8, v_desc, idesc_pv, (t != 0) || (j != 0));
          umma_ts(tm_o, tm_s + 64 + j * 8, v_desc, idesc_pv, 1);
        }
        tc_commit(&bars->v_empty);
        ph ^= 1;
      }
    }
  } else {
    const int row = qt * kHtRows + warp * 32 + lane;               // in the sequence's portion
    const int limit = a.q_pos0[seq] + row, lo = a.h.first_seen(limit);
    const uint32_t lane_addr = uint32_t(warp * 32) << 16;
    const float scale_log2 = a.h.scale * kLog2E;
    const int means = MODE == kHtPooled ? a.h.means_seen(limit) : 0;
    bool of_means = false;                       // the tile at hand
    auto sees = [&](int k) {
      if (MODE == kHtPooled && of_means) return k < means;
      return MODE == kHtPlain || MODE == kHtPooled ? k <= limit && k >= lo : a.h.sees(k, limit, lo);
    };
    auto log2_score = [&](float s) {
      return MODE == kHtCap || MODE == kHtFixed ? a.h.capped(s * a.h.scale) * kLog2E : s * scale_log2;
    };
    const int o_cols = (a.h.vdim + 15) / 16 * 16;
    const float cap_in = 2.f * a.h.scale * kLog2E / a.h.cap, cap_out = -2.f * a.h.cap * kLog2E;        // kHtFixed
    // a sink is one more key of every row, with a value of zero
    float m_used = a.h.sink != nullptr ? a.h.sink_log2(head) : -INFINITY, l = a.h.sink != nullptr ? 1.f : 0.f;
    uint32_t ph = 0;
    bool ok = true;
    for (int t = 0; t < n_tiles; ++t) {
      const int k0 = key_of(t), t_end = end_of(t);
      // which groups of 16 keys of the tile exist; looked up while S is still being computed
      const int g_tok = k0 + (lane & 7) * 16;
      const uint32_t groups = __ballot_sync(0xffffffffu, g_tok < t_end && block_at(t, g_tok) >= 0) & 0xFFu;
      if constexpr (MODE == kHtPooled) of_means = t < kept;
      // one verdict per warp: the tcgen05.ld / st below are warp-wide
      if (!__all_sync(0xffffffffu, mbar_wait(&bars->s_full, ph, abort_flag, a.status, 98, t))) {
        ok = false;
        break;
      }
      tc_fence_after_sync();
      const bool from_lo = k0 >= lo || (MODE != kHtPlain && MODE != kHtPooled && k0 + kHtKeys <= a.h.keep);
      const bool whole = MODE == kHtPooled && of_means ? k0 + kHtKeys <= means : from_lo && k0 + kHtKeys - 1 <= limit;
      const bool full = __all_sync(0xffffffffu, groups == 0xFFu && whole);
      float mx = -INFINITY;
#pragma unroll 1
      for (int c = 0; MODE != kHtFixed && c < 4; ++c) {
        uint32_t v[32];
        ZSE_TMEM_LD_X16(v, tm_s + lane_addr + c * 32);
        ZSE_TMEM_LD_X16((v + 16), tm_s + lane_addr + c * 32 + 16);
        tc_wait_ld();
        if (full) {
          float m0 = mx, m1 = -INFINITY;
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            m0 = fmaxf(m0, __uint_as_float(v[i]));
            m1 = fmaxf(m1, __uint_as_float(v[i + 1]));
          }
          mx = fmaxf(m0, m1);
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int k = k0 + c * 32 + i;
            const bool seen = ((groups >> (c * 2 + (i >> 4))) & 1u) && sees(k);
            mx = seen ? fmaxf(mx, __uint_as_float(v[i])) : mx;
          }
        }
      }
      // scale > 0 and the cap's tanh is monotone: the maximum commutes with both
      if (mx != -INFINITY) mx = log2_score(mx);
      // move the reference maximum only when some row of the warp needs it
      if (__any_sync(0xffffffffu, mx > m_used + 8.f)) {
        const float m_new = fmaxf(m_used, mx);
        const float alpha = m_used == -INFINITY ? 0.f : ex2(m_used - m_new);
        if (t > 0) {                             // s_full of this tile: every earlier MMA has completed, O is stable
#pragma unroll 1
          for (int c = 0; c < o_cols; c += 16) {
            uint32_t o[16];
            ZSE_TMEM_LD_X16(o, tm_o + lane_addr + c);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            ZSE_TMEM_ST_X16(tm_o + lane_addr + c, o);
          }
          tc_wait_st();
        }
        l *= alpha;
        m_used = m_new;
      }
      const float m_ref = m_used == -INFINITY ? 0.f : m_used;
      uint32_t rest[64];                         // the second terms wait until every score has been read
      float s0 = 0.f, s1 = 0.f;
      auto weights = [&](auto all) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t hi[16];
#pragma unroll
          for (int b = 0; b < 2; ++b) {
            uint32_t v[16];
            ZSE_TMEM_LD_X16(v, tm_s + lane_addr + c * 32 + b * 16);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              float p0, p1;
              if constexpr (MODE == kHtFixed) {     // cap tanh(s / cap) - cap = -2 cap / (1 + exp(2 s / cap))
                p0 = ex2(cap_out * rcp(1.f + ex2(__uint_as_float(v[2 * i]) * cap_in)));
                p1 = ex2(cap_out * rcp(1.f + ex2(__uint_as_float(v[2 * i + 1]) * cap_in)));
              } else if constexpr (MODE == kHtCap) {
                p0 = ex2(log2_score(__uint_as_float(v[2 * i])) - m_ref);
                p1 = ex2(log2_score(__uint_as_float(v[2 * i + 1])) - m_ref);
              } else {
                p0 = ex2(fmaf(__uint_as_float(v[2 * i]), scale_log2, -m_ref));
                p1 = ex2(fmaf(__uint_as_float(v[2 * i + 1]), scale_log2, -m_ref));
              }
              if constexpr (!decltype(all)::value) {
                const int k = k0 + c * 32 + b * 16 + 2 * i;
                const bool there = (groups >> (c * 2 + b)) & 1u;
                p0 = there && sees(k) ? p0 : 0.f;
                p1 = there && sees(k + 1) ? p1 : 0.f;
              }
              s0 += p0;
              s1 += p1;
              const uint32_t x = pack_bf16(p0, p1);
              hi[b * 8 + i] = x;
              // bf16 -> fp32 is a shift
              rest[c * 16 + b * 8 + i] = pack_bf16(p0 - __uint_as_float(x << 16), p1 - __uint_as_float(x & 0xFFFF0000u));
            }
          }
          ZSE_TMEM_ST_X16(tm_s + lane_addr + c * 16, hi);          // under scores that have been read
        }
      };
      if (full)
        weights(std::true_type{});
      else
        weights(std::false_type{});
      ZSE_TMEM_ST_X32(tm_s + lane_addr + 64, rest);
      ZSE_TMEM_ST_X32(tm_s + lane_addr + 96, (rest + 32));
      l += s0 + s1;
      tc_wait_st();
      tc_fence_before_sync();
      mbar_arrive(&bars->p_full);
      ph ^= 1;
    }
    // O is complete when P V of the last tile is
    if (ok)
      ok = __all_sync(0xffffffffu,
                      mbar_wait_spin(&bars->v_empty, uint32_t(n_tiles - 1) & 1u, abort_flag, a.status, 99, 0));
    tc_fence_after_sync();
    if (ok) {
      const bool live = row < q_len;
      const size_t t = size_t(q_begin + (live ? row : 0));
      float inv = l > 0.f ? a.h.out_scale / l : 0.f;
      const bf16* gates = a.gate != nullptr && a.h.gate_each ? a.gate + t * a.ld + size_t(head) * a.h.vdim : nullptr;
      if (a.gate != nullptr && gates == nullptr) inv *= sigmoid_exact(to_f32(a.gate[t * a.ld + head]));
      bf16* dst = a.out + t * a.ldo + size_t(head) * a.h.vdim;
#pragma unroll 1
      for (int c = 0; c < o_cols; c += 16) {     // every lane takes part in the warp-wide loads
        uint32_t o[16];
        ZSE_TMEM_LD_X16(o, tm_o + lane_addr + c);
        tc_wait_ld();
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          if (!live || c + b * 8 >= a.h.vdim) continue;
          uint4 w;
          uint32_t* x = o + b * 8;
          if (gates != nullptr) {
            const uint4 g = *reinterpret_cast<const uint4*>(gates + c + b * 8);
            const uint32_t two[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const float z = __uint_as_float(i & 1 ? two[i / 2] & 0xFFFF0000u : two[i / 2] << 16);
              x[i] = __float_as_uint(__uint_as_float(x[i]) * sigmoid_fast(z));
            }
          }
          w.x = pack_bf16(__uint_as_float(x[0]) * inv, __uint_as_float(x[1]) * inv);
          w.y = pack_bf16(__uint_as_float(x[2]) * inv, __uint_as_float(x[3]) * inv);
          w.z = pack_bf16(__uint_as_float(x[4]) * inv, __uint_as_float(x[5]) * inv);
          w.w = pack_bf16(__uint_as_float(x[6]) * inv, __uint_as_float(x[7]) * inv);
          *reinterpret_cast<uint4*>(dst + c + b * 8) = w;
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 5) tmem_dealloc(tm_s, 256);
}

}  // namespace

bool heads_tc_ok(const Heads& h, int num_blocks, int ld, int ldo) {
  return h.dim % 8 == 0 && h.vdim % 8 == 0 && h.dim > 0 && h.vdim > 0 && h.dim <= 128 && h.vdim <= 128 &&
         h.block_size % 16 == 0 && num_blocks > 0 && ld % 8 == 0 && ldo % 8 == 0 && h.block_stride % 8 == 0 && h.scale > 0.f;
}

int launch_heads_tc(const bf16* inp, int ld, int rows, const void* k, const void* v, int num_blocks, const Heads& h,
                    const int* cu_q, const int* q_pos0, int first, int last, int max_q, bf16* out, int ldo,
                    const bf16* gate, Status* status, cudaStream_t st) {
  if ((reinterpret_cast<uintptr_t>(out) & 15) != 0) return ZSE_ERR_ALIGN;
  if (gate != nullptr && h.gate_each && (reinterpret_cast<uintptr_t>(gate) & 15) != 0) return ZSE_ERR_ALIGN;
  const int br = h.block_size % 64 == 0 ? 64 : h.block_size % 32 == 0 ? 32 : 16;
  CUtensorMap mq, mk, mv;
  if (int rc = get_tmap(inp, uint64_t(rows), uint64_t(ld), uint32_t(kHtRows), &mq)) return rc;
  // a block of one layer: [kv heads * tokens] rows of dp (vp) elements
  const int per_block = h.kv_heads * h.block_size;
  if (int rc = get_tmap_rows3(k, num_blocks, per_block, h.dp, h.block_stride, br, 0, &mk)) return rc;
  if (int rc = get_tmap_rows3(v, num_blocks, per_block, h.vp, h.block_stride, br, 0, &mv)) return rc;
  const HtArgs a{h, cu_q, q_pos0, first, out, ldo, gate, ld, br, (h.dim + 63) / 64, (h.vdim + 63) / 64, status};
  const size_t smem = size_t(2 * a.k_panels + a.v_panels) * kHtPanel + 1024 + sizeof(HtBars);
  static bool done[5][kMaxDevices] = {};
  const int slot = current_device_slot();
  const int mode = h.pool > 0 ? kHtPooled : h.cap <= 0.f ? (h.keep > 0 ? kHtNoCap : kHtPlain) : h.cap <= kHtFixedCap ? kHtFixed : kHtCap;
  auto kern = mode == kHtPlain    ? heads_tc_kernel<kHtPlain>
              : mode == kHtNoCap  ? heads_tc_kernel<kHtNoCap>
              : mode == kHtCap    ? heads_tc_kernel<kHtCap>
              : mode == kHtPooled ? heads_tc_kernel<kHtPooled>
                                  : heads_tc_kernel<kHtFixed>;
  if (!done[mode][slot]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             int(6 * kHtPanel + 1024 + sizeof(HtBars))) != cudaSuccess)
      return ZSE_ERR_LAUNCH;
    done[mode][slot] = true;
  }
  return launch_pdl(kern, dim3((max_q + kHtRows - 1) / kHtRows, h.heads, last - first), dim3(kHtThreads), smem, st,
                    mq, mk, mv, a) == cudaSuccess
             ? 0
             : ZSE_ERR_LAUNCH;
}

}  // namespace zse
