// Routed feed-forward: which tokens go to which expert, and the experts' products.
//
//   topk      scores of the router's fp32 logits (sigmoid, or softmax over the experts), the `top` largest per token (lower
//             id first on a tie) among the experts of the best groups, their weights, and each (token, choice) slot's place
//             within its expert
//   plan      one CTA: first row of every expert in the sorted order, table of token tiles for the grouped products
//   permute   the tokens' rows, copied into sorted order, with the score and the slot of each sorted row
//   products  grouped GEMM on tcgen05 (moe_gemm_kernel), the shared expert's dense product in the same launch
//
// The order of rows inside an expert depends on the order of atomic adds; a row's result does not depend on its place.
#include <cuda.h>

#include "api.h"
#include "gemm_common.cuh"
#include "moe.cuh"
#include "typed.cuh"

namespace zse {
namespace {

constexpr int kTopkWarps = 8;

// Router rows are `cols` wide: column E, if there is one, is the shared expert's gate, whose sigmoid goes to shared_score.
__global__ void __launch_bounds__(kTopkWarps * 32)
moe_topk_kernel(const float* __restrict__ planes, int n_planes, int M, int E, int cols, int top, int softmax, int normalise,
                float scale, int groups, int keep, int* __restrict__ counts, int* __restrict__ slot_expert,
                int* __restrict__ slot_rank, float* __restrict__ slot_score, float* __restrict__ shared_score) {
  extern __shared__ float scores[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * kTopkWarps + warp;
  if (t >= M) return;
  float* s = scores + warp * (E + top + groups);
  float* chosen = s + E;
  float* group = chosen + top;
  auto logit = [&](int e) {
    float z = 0.f;
    for (int p = 0; p < n_planes; ++p) z += planes[(size_t(p) * M + t) * cols + e];
    return z;
  };
  float most = -INFINITY;
  for (int e = lane; e < E; e += 32) {
    const float z = logit(e);
    s[e] = softmax ? z : sigmoid_exact(z);
    most = fmaxf(most, z);
  }
  if (cols > E && lane == 0) shared_score[t] = sigmoid_exact(logit(E));
  if (softmax) {
    most = warp_max(most);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) {
      s[e] = expf(s[e] - most);
      sum += s[e];
    }
    sum = warp_sum(sum);
    for (int e = lane; e < E; e += 32) s[e] /= sum;
  }
  // the largest of n values, the lowest index on a tie; every lane gets it
  auto largest = [&](const float* v, int n, float& best, int& at) {
    best = -2.f;
    at = 0x7fffffff;
    for (int e = lane; e < n; e += 32)
      if (v[e] > best) {
        best = v[e];
        at = e;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b2 = __shfl_xor_sync(0xffffffffu, best, o);
      const int a2 = __shfl_xor_sync(0xffffffffu, at, o);
      if (b2 > best || (b2 == best && a2 < at)) {
        best = b2;
        at = a2;
      }
    }
  };
  if (keep < groups) {                               // only experts of the best groups remain (scores are >= 0)
    const int per = E / groups;
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
      float a = 0.f, b = 0.f;                        // the two largest
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float x = s[e];
        b = fmaxf(b, fminf(a, x));
        a = fmaxf(a, x);
      }
      group[g] = a + b;
    }
    __syncwarp();
    for (int k = 0; k < keep; ++k) {
      float best;
      int at;
      largest(group, groups, best, at);
      if (at >= groups) at = 0;
      __syncwarp();
      if (lane == (at & 31)) group[at] = -1.5f;
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (group[e / per] != -1.5f) s[e] = -1.f;
  }
  float total = 0.f;
  for (int k = 0; k < top; ++k) {
    float best;
    int at;
    largest(s, E, best, at);
    if (at >= E) at = 0;                              // a row of NaN scores: still a valid expert
    if (lane == (at & 31)) s[at] = -1.f;              // the lane that owns this expert
    if (lane == 0) {
      const int slot = t * top + k;
      slot_expert[slot] = at;
      slot_rank[slot] = atomicAdd(&counts[at], 1);
      chosen[k] = best;
    }
    total += best;
  }
  __syncwarp();
  const float w = normalise ? scale / (total + 1e-20f) : scale;
  for (int k = lane; k < top; k += 32) slot_score[t * top + k] = chosen[k] * w;
}

constexpr int kPlanThreads = 1024;

// `counts` is zero again afterwards.
__global__ void __launch_bounds__(kPlanThreads)
moe_plan_kernel(int* __restrict__ counts, int E, int tile_rows, int* __restrict__ first_row,
                MoeTile* __restrict__ tiles, int* __restrict__ n_tiles) {
  __shared__ int warp_rows[32], warp_tiles[32];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int row_base = 0, tile_base = 0;
  for (int e0 = 0; e0 < E; e0 += kPlanThreads) {
    const int e = e0 + threadIdx.x;
    const int n = e < E ? counts[e] : 0;
    const int nt = (n + tile_rows - 1) / tile_rows;
    int a = n, b = nt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int x = __shfl_up_sync(0xffffffffu, a, o), y = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) {
        a += x;
        b += y;
      }
    }
    if (lane == 31) {
      warp_rows[warp] = a;
      warp_tiles[warp] = b;
    }
    __syncthreads();
    int wr = 0, wt = 0, all_r = 0, all_t = 0;
    for (int w = 0; w < 32; ++w) {
      if (w < warp) {
        wr += warp_rows[w];
        wt += warp_tiles[w];
      }
      all_r += warp_rows[w];
      all_t += warp_tiles[w];
    }
    const int r0 = row_base + wr + a - n, t0 = tile_base + wt + b - nt;
    if (e < E) {
      first_row[e] = r0;
      counts[e] = 0;
      for (int i = 0; i < nt; ++i)
        tiles[t0 + i] = MoeTile{e, r0 + i * tile_rows, min(tile_rows, n - i * tile_rows), 0};
    }
    row_base += all_r;
    tile_base += all_t;
    __syncthreads();
  }
  if (threadIdx.x == 0) *n_tiles = tile_base;
}

// One warp per slot: x[token] -> xs[first_row[expert] + rank]; out_rows[row] = the slot's row of the result.
template <typename T>
__global__ void __launch_bounds__(256)
moe_permute_kernel(const T* __restrict__ x, int H, int slots, int top, int out_per_token,
                   const int* __restrict__ slot_expert, const int* __restrict__ slot_rank,
                   const float* __restrict__ slot_score, const int* __restrict__ first_row, T* __restrict__ xs,
                   float* __restrict__ row_score, int* __restrict__ out_rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int slot = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (slot >= slots) return;
  const int t = slot / top;
  const int row = first_row[slot_expert[slot]] + slot_rank[slot];
  const T* src = x + size_t(t) * H;
  T* dst = xs + size_t(row) * H;
  constexpr int kVec = 16 / sizeof(T);
  if (H % kVec == 0) {
    for (int i = lane; i < H / kVec; i += 32) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
  } else {
    for (int i = lane; i < H; i += 32) dst[i] = src[i];
  }
  if (lane == 0) {
    row_score[row] = slot_score[slot];
    out_rows[row] = t * out_per_token + slot % top;
  }
}

// ---- grouped products on tcgen05 --------------------------------------------------------------------------------------
// Two products share a launch: the routed experts' (token tiles from the table, weights W[group * N + n, :]) and the
// shared expert's (all tokens, its own weights, sizes and activations).  Like gemm_f16_kernel the UMMA M dimension (128)
// runs over weight rows and N over tokens.
struct MoeProduct {
  int N, K;                 // weight rows of a group, reduction length
  void* out;
  int ldo;                  // output row stride
  int cols;                 // output columns (kMoeGlu: half of N, or less where N is padded)
  float limit;              // kMoeGlu
  const float* row_scale;   // per token row, or null: before the activation (up), on the result (down)
  const int* out_rows;      // output row of a token row, or null: row * mul + add
  int mul, add;
};
struct MoeGemmArgs {
  MoeProduct routed, shared;
  const MoeTile* tiles;
  const int* n_tiles;
  int dense_tiles;          // token tiles of the shared expert (0: none)
  int M;                    // tokens
  int glu;                  // kMoeGlu: which gated activation
  Status* status;
};

template <int NT>
struct MoeCfg {
  static constexpr int kABytes = kTileN * 128;
  static constexpr int kXBytes = NT * 128;
  static constexpr int kStageBytes = kABytes + kXBytes;
  static constexpr int kStages = NT <= 32 ? 5 : NT == 64 ? 4 : NT == 128 ? 3 : 2;   // two CTAs share an SM:
  static constexpr int kTmemCols = NT < 32 ? 32 : NT;                               // one computes while the
  static constexpr int kSmemBytes = kStages * kStageBytes + 1024 + 256;             // other writes its results
  static constexpr int kMinBlocks = 2;
};
struct MoeBars {
  uint64_t full[8], empty[8], acc_ready;
  uint32_t tmem_base;
  int abort_flag;
};

// gelu(scale * acc) -> bf16; scale * acc -> OutT; glu -> bf16 (a tile of W: 64 gate rows, then their 64 up rows)
enum MoeEpi { kMoeUp = 0, kMoeDown = 1, kMoeGlu = 2 };

template <int NT, int EPI, typename OutT>
__global__ void __launch_bounds__(kGemmThreads, MoeCfg<NT>::kMinBlocks)
moe_gemm_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x,
                const __grid_constant__ CUtensorMap map_ws, const __grid_constant__ CUtensorMap map_xs,
                const MoeGemmArgs a) {
  using Cfg = MoeCfg<NT>;
  constexpr int S = Cfg::kStages;
  extern __shared__ uint8_t smem_raw[];
  pdl_launch_dependents();
  pdl_wait();
  const bool dense = int(blockIdx.y) < a.dense_tiles;
  const MoeProduct& p = dense ? a.shared : a.routed;
  const int n0 = blockIdx.x * kTileN;
  if (n0 >= p.N) return;
  MoeTile tile;
  if (dense) {
    tile = MoeTile{0, int(blockIdx.y) * NT, min(NT, a.M - int(blockIdx.y) * NT), 0};
  } else {
    const int i = blockIdx.y - a.dense_tiles;
    if (i >= *a.n_tiles) return;
    tile = a.tiles[i];
  }
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  MoeBars* bars = reinterpret_cast<MoeBars*>(smem + S * Cfg::kStageBytes);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_iter = (p.K + 63) / 64;
  if (threadIdx.x == 0) {
    for (int i = 0; i < S; ++i) {
      mbar_init(&bars->full[i], 1);
      mbar_init(&bars->empty[i], 1);
    }
    mbar_init(&bars->acc_ready, 1);
    bars->abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&bars->tmem_base, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = bars->tmem_base;
  volatile int* abort_flag = &bars->abort_flag;

  if (warp == 0) {
    if (lane == 0) {
      const CUtensorMap* mw = dense ? &map_ws : &map_w;
      const CUtensorMap* mx = dense ? &map_xs : &map_x;
      const int wrow = tile.group * p.N + n0;
      int issued = 0;
      for (int it = 0; it < n_iter; ++it) {
        const int s = it % S;
        if (it >= S && !mbar_wait(&bars->empty[s], ((it / S) - 1) & 1, abort_flag, a.status, 71, it)) break;
        uint8_t* st = smem + s * Cfg::kStageBytes;
        mbar_arrive_expect_tx(&bars->full[s], Cfg::kStageBytes);
        tma_load_2d(st, mw, it * 64, wrow, &bars->full[s]);
        tma_load_2d(st + Cfg::kABytes, mx, it * 64, tile.row0, &bars->full[s]);
        issued = it + 1;
      }
      if (*abort_flag) {
        for (int it = max(0, issued - S); it < issued; ++it) {
          const uint64_t t0 = globaltimer_ns();
          while (!mbar_try_wait(&bars->full[it % S], (it / S) & 1) && globaltimer_ns() - t0 < kWaitLimitNs) {
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc_f16(kTileN, NT, 1);
      for (int it = 0; it < n_iter; ++it) {
        const int s = it % S;
        if (!mbar_wait(&bars->full[s], (it / S) & 1, abort_flag, a.status, 72, it)) break;
        tc_fence_after_sync();
        const uint32_t ab = smem_u32(smem + s * Cfg::kStageBytes);
#pragma unroll
        for (int j = 0; j < 4; ++j)
          umma_ss(tmem, make_desc_sw128(ab + j * 32), make_desc_sw128(ab + Cfg::kABytes + j * 32), idesc,
                  (it | j) != 0);
        tc_commit(&bars->empty[s]);
      }
      tc_commit(&bars->acc_ready);
    }
  } else {
    const bool ok = mbar_wait(&bars->acc_ready, 0, abort_flag, a.status, 73, 0);
    tc_fence_after_sync();
    const int q = warp & 3, ch = (warp - 2) >> 2;
    constexpr int kCols = NT >= 32 ? NT / 2 : NT;
    const bool mine = __all_sync(0xffffffffu, ok && (NT >= 32 || ch == 0));
    if constexpr (EPI == kMoeGlu) {
      // warps with up rows (q = 2, 3) park them in shared memory, their partners with the gate rows combine; a warp with
      // nothing to do still meets its partner
      float* park = reinterpret_cast<float*>(smem) + ((q & 1) + 2 * ch) * (32 * kCols);
      const int bar = 1 + (q & 1) + 2 * ch;
      const bool work = mine && ch * kCols < tile.rows;
      if (q >= 2) {
        if (work) {
#pragma unroll 1
          for (int c = 0; c < kCols && ch * kCols + c < tile.rows; c += 16) {
            uint32_t r[16];
            ZSE_TMEM_LD_X16(r, tmem + (uint32_t(q * 32) << 16) + ch * kCols + c);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 16; ++i) park[(c + i) * 32 + lane] = __uint_as_float(r[i]);
          }
        }
        asm volatile("bar.sync %0, 64;" ::"r"(bar) : "memory");
      } else {
        asm volatile("bar.sync %0, 64;" ::"r"(bar) : "memory");
        const int n = blockIdx.x * 64 + q * 32 + lane;
        if (work) {
#pragma unroll 1
          for (int c = 0; c < kCols && ch * kCols + c < tile.rows; c += 16) {
            uint32_t r[16];
            ZSE_TMEM_LD_X16(r, tmem + (uint32_t(q * 32) << 16) + ch * kCols + c);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              const int col = ch * kCols + c + i;
              if (col < tile.rows && n < p.cols)
                reinterpret_cast<OutT*>(p.out)[size_t(tile.row0 + col) * p.ldo + n] =
                    from_f32<OutT>(glu<true>(a.glu, __uint_as_float(r[i]), park[(c + i) * 32 + lane], p.limit));
            }
          }
        }
      }
    }
    const int n = n0 + q * 32 + lane;
    if (EPI != kMoeGlu && mine && ch * kCols < tile.rows) {
#pragma unroll 1
      for (int c = 0; c < kCols; c += 16) {
        if (ch * kCols + c >= tile.rows) break;
        uint32_t r[16];
        ZSE_TMEM_LD_X16(r, tmem + (uint32_t(q * 32) << 16) + ch * kCols + c);
        tc_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int col = ch * kCols + c + i;
          if (col < tile.rows && n < p.N) {
            const int row = tile.row0 + col;
            float v = __uint_as_float(r[i]);
            if (p.row_scale != nullptr) v *= p.row_scale[row];
            if (EPI == kMoeUp) v = gelu_exact(v);
            const size_t orow = p.out_rows != nullptr ? p.out_rows[row] : size_t(row) * p.mul + p.add;
            reinterpret_cast<OutT*>(p.out)[orow * p.ldo + n] = from_f32<OutT>(v);
          }
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, Cfg::kTmemCols);
}

template <int NT, int EPI, typename OutT>
int launch_moe(const CUtensorMap* m, const MoeGemmArgs& a, dim3 grid, cudaStream_t st) {
  auto kern = moe_gemm_kernel<NT, EPI, OutT>;
  static bool attr_done[kMaxDevices] = {};
  const int slot = current_device_slot();
  if (!attr_done[slot]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MoeCfg<NT>::kSmemBytes) != cudaSuccess)
      return ZSE_ERR_LAUNCH;
    attr_done[slot] = true;
  }
  return launch_pdl(kern, grid, dim3(kGemmThreads), size_t(MoeCfg<NT>::kSmemBytes), st, m[0], m[1], m[2], m[3], a) ==
                 cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

}  // namespace
}  // namespace zse

using namespace zse;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int zse_moe_route(int dtype, const ZseRouter* r, int M, int tile_rows, const void* x, int H, int out_per_token,
                             void* counts, void* slot_expert, void* slot_rank, void* slot_score, void* first_row,
                             void* tiles, void* n_tiles, void* xs, void* row_score, void* out_rows, void* shared_score,
                             void* stream) {
  const int E = r->experts, top = r->top;
  if (M <= 0) return 0;
  if (E <= 0 || top <= 0 || top > E || tile_rows <= 0 || E + top + r->groups > 1536) return ZSE_ERR_SHAPE;
  if (r->groups <= 0 || E % r->groups || r->keep <= 0 || r->keep > r->groups || top > r->keep * (E / r->groups))
    return ZSE_ERR_SHAPE;
  cudaStream_t st = ST(stream);
  const size_t smem = size_t(kTopkWarps) * (E + top + r->groups) * sizeof(float);
  if (launch_pdl(moe_topk_kernel, dim3((M + kTopkWarps - 1) / kTopkWarps), dim3(kTopkWarps * 32), smem, st,
                 reinterpret_cast<const float*>(r->planes), r->n_planes, M, E, r->cols, top, r->softmax, r->normalise,
                 r->scale, r->groups, r->keep, reinterpret_cast<int*>(counts), reinterpret_cast<int*>(slot_expert),
                 reinterpret_cast<int*>(slot_rank), reinterpret_cast<float*>(slot_score),
                 reinterpret_cast<float*>(shared_score)) != cudaSuccess)
    return ZSE_ERR_LAUNCH;
  if (launch_pdl(moe_plan_kernel, dim3(1), dim3(kPlanThreads), 0, st, reinterpret_cast<int*>(counts), E, tile_rows,
                 reinterpret_cast<int*>(first_row), reinterpret_cast<MoeTile*>(tiles),
                 reinterpret_cast<int*>(n_tiles)) != cudaSuccess)
    return ZSE_ERR_LAUNCH;
  const int slots = M * top;
  cudaError_t e;
  if (dtype == kBF16)
    e = launch_pdl(moe_permute_kernel<bf16>, dim3((slots + 7) / 8), dim3(256), 0, st, reinterpret_cast<const bf16*>(x),
                   H, slots, top, out_per_token, reinterpret_cast<const int*>(slot_expert),
                   reinterpret_cast<const int*>(slot_rank), reinterpret_cast<const float*>(slot_score),
                   reinterpret_cast<const int*>(first_row), reinterpret_cast<bf16*>(xs),
                   reinterpret_cast<float*>(row_score), reinterpret_cast<int*>(out_rows));
  else
    e = launch_pdl(moe_permute_kernel<float>, dim3((slots + 7) / 8), dim3(256), 0, st,
                   reinterpret_cast<const float*>(x), H, slots, top, out_per_token,
                   reinterpret_cast<const int*>(slot_expert), reinterpret_cast<const int*>(slot_rank),
                   reinterpret_cast<const float*>(slot_score), reinterpret_cast<const int*>(first_row),
                   reinterpret_cast<float*>(xs), reinterpret_cast<float*>(row_score), reinterpret_cast<int*>(out_rows));
  return e == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_moe_tile_rows(int M, int E, int top) {
  const int avg = (M * top + E - 1) / E;
  const int want = avg + avg / 4;
  return want <= 16 ? 16 : want <= 32 ? 32 : want <= 64 ? 64 : want <= 160 ? 128 : 256;
}

// Up (epilogue 0: gelu(scale * acc) in bfloat16; 3: gated) or down (1: bfloat16, 2: fp32 result rows) products of all
// experts.
extern "C" int zse_moe_gemm(const ZseMoeGemm* g, int M, int E, int max_rows, int tile_rows, int max_tiles, int epilogue,
                            void* status, void* stream) {
  if (M <= 0) return 0;
  const bool shared = g->shared_n > 0;
  if (g->routed_k % 8 || (shared && g->shared_k % 8)) return ZSE_ERR_SHAPE;
  CUtensorMap m[4];
  if (int rc = get_tmap(g->routed_w, uint64_t(E) * g->routed_n, g->routed_k, kTileN, &m[0])) return rc;
  if (int rc = get_tmap(g->routed_x, max_rows, g->routed_k, tile_rows, &m[1])) return rc;
  m[2] = m[0];
  m[3] = m[1];
  if (shared) {
    if (int rc = get_tmap(g->shared_w, g->shared_n, g->shared_k, kTileN, &m[2])) return rc;
    if (int rc = get_tmap(g->shared_x, g->shared_x_rows, g->shared_k, tile_rows, &m[3])) return rc;
  }
  MoeGemmArgs a{};
  if (epilogue == 3 && (g->routed_n % kTileN || (shared && g->shared_n % kTileN))) return ZSE_ERR_SHAPE;
  a.routed = MoeProduct{g->routed_n, g->routed_k, g->routed_out, g->routed_ldo, g->routed_cols, g->routed_limit,
                        reinterpret_cast<const float*>(g->row_score), reinterpret_cast<const int*>(g->out_rows), 1, 0};
  if (shared)
    a.shared = MoeProduct{g->shared_n, g->shared_k, g->shared_out, g->shared_ldo, g->shared_cols, g->shared_limit,
                          reinterpret_cast<const float*>(g->shared_score), nullptr, g->shared_mul, g->shared_add};
  a.tiles = reinterpret_cast<const MoeTile*>(g->tiles);
  a.n_tiles = reinterpret_cast<const int*>(g->n_tiles);
  a.dense_tiles = shared ? (M + tile_rows - 1) / tile_rows : 0;
  a.M = M;
  a.glu = g->glu;
  a.status = reinterpret_cast<Status*>(status);
  const int nmax = shared && g->shared_n > g->routed_n ? g->shared_n : g->routed_n;
  if (a.dense_tiles + max_tiles > 65535) return ZSE_ERR_LIMIT;
  dim3 grid((nmax + kTileN - 1) / kTileN, a.dense_tiles + max_tiles);
  int rc = ZSE_ERR_SHAPE;
#define ZSE_MOE(E_, T_) ZSE_DISPATCH_NT(tile_rows, rc = (launch_moe<NT, E_, T_>(m, a, grid, ST(stream))))
  if (epilogue == 0) {
    ZSE_MOE(kMoeUp, bf16)
  } else if (epilogue == 1) {
    ZSE_MOE(kMoeDown, bf16)
  } else if (epilogue == 3) {
    ZSE_MOE(kMoeGlu, bf16)
  } else {
    ZSE_MOE(kMoeDown, float)
  }
#undef ZSE_MOE
  return rc;
}
