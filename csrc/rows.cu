// Row kernels for activations of bfloat16 or float: embedding (plain, or with a bigram table, a sinusoid and a norm),
// residual sum + RMSNorm (+ a causal convolution over the normed rows), RMSNorm + residual sum, logits epilogue, arg-max of
// fp32 logits.  Any row length.
#include <initializer_list>

#include "api.h"
#include "typed.cuh"

namespace zse {
namespace {

template <typename T, int VEC>
__global__ void __launch_bounds__(256) embedding_typed_kernel(const T* __restrict__ table, const int* __restrict__ ids,
                                       float* __restrict__ out, int H, int vocab, float scale, T* __restrict__ copy,
                                       int ld_copy, Status* st) {
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
#pragma unroll 4
  for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
    F32Vec<VEC> x = load_vec<VEC>(src + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x.v[e] *= scale;
    store_vec<VEC>(dst + i, x);
    if (copy != nullptr) store_vec<VEC>(copy + size_t(row) * ld_copy + i, x);
  }
}

// y = sum of fp32 planes [n_planes][M][H] + sum of the row's slots [M][n_slots][H], times scale [H] if there is one;
// residual += y, or residual = y (replace); out [M, ldo] = RMSNorm(residual) * (weight + offset), or the residual itself
// without a weight.  A row is split over the CTAs of a cluster (gridDim.x), each thread keeps its
// columns in registers between the sum and the norm; VEC consecutive columns per access (4 when H % 4 == 0).
constexpr int kRowThreads = 256;
constexpr int kRowRegs = 8;          // accesses per thread: H <= 8 * VEC * 256 * cluster

// Sum of a value over the CTAs of the cluster (every thread of a CTA holds the CTA's value).
__device__ __forceinline__ float row_cluster_sum(float total, float* slot, int cs) {
  if (cs == 1) return total;
  if (threadIdx.x == 0) *slot = total;
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
  total = 0.f;
  const uint32_t local = smem_u32(slot);
  for (int r = 0; r < cs; ++r) {                           // same order in every CTA: identical sums
    uint32_t remote;
    float t;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(r));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(t) : "r"(remote) : "memory");
    total += t;
  }
  // nobody exits while its value may still be read
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
  return total;
}

// A causal convolution along every sequence, per channel, of rows h [M, H]: y = h + sum_j w[j] h_(t - taps + 1 + j).  State rows
// hold a sequence's last taps - 1 rows of h, the oldest first: a pass reads them in one row of the pool (-1: zeros) and leaves
// its own last ones in another.
struct RowConv {
  const float* w;                     // [taps][H], the row's own tap last
  int taps;
  float* states;
  long long row_floats;
  const int* state_rows;              // [2][state_ld]
  int state_ld;
};

// CONV: every row is a sequence of its own; conv_out [M, H] = the row (as rounded into `out`) plus its convolution.
template <typename T, typename S, int VEC, bool CONV>
__global__ void __launch_bounds__(kRowThreads)
add_norm_kernel(float* __restrict__ residual, const float* __restrict__ planes, int n_planes,
                const S* __restrict__ slots, int n_slots, const T* __restrict__ scale, int replace,
                const T* __restrict__ weight, float offset, T* __restrict__ out, int ldo, int M, int H, float eps,
                const RowConv cv, T* __restrict__ conv_out) {
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
      F32Vec<VEC> old{}, f;
      if (!replace) old = load_vec<VEC>(residual + at);
      if (scale != nullptr) f = load_vec<VEC>(scale + size_t(i) * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[j].v[e] = scale == nullptr ? old.v[e] : 0.f;
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
      if (scale != nullptr) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[j].v[e] = fmaf(x[j].v[e], f.v[e], old.v[e]);
      }
      if (n_planes + n_slots > 0) store_vec<VEC>(residual + at, x[j]);
      if (weight == nullptr) store_vec<VEC>(out + size_t(row) * ldo + size_t(i) * VEC, x[j]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x[j].v[e] * x[j].v[e];
    }
  }
  if (weight == nullptr) return;                           // the same for every CTA of the cluster
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = warp_sum((threadIdx.x & 31) < (kRowThreads >> 5) ? red[threadIdx.x & 31] : 0.f);
  total = row_cluster_sum(total, &cluster_ss, cs);
  const float inv = 1.f / sqrtf(total / float(H) + eps);
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i < v1) {
      F32Vec<VEC> w = load_vec<VEC>(weight + size_t(i) * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) w.v[e] = (w.v[e] + offset) * (x[j].v[e] * inv);
      store_vec<VEC>(out + size_t(row) * ldo + size_t(i) * VEC, w);
      if constexpr (CONV) {
        const int read = cv.state_rows[row], write = cv.state_rows[cv.state_ld + row];
        const int c = i * VEC;
        const F32Vec<VEC> own = load_vec<VEC>(cv.w + size_t(cv.taps - 1) * H + c);
        F32Vec<VEC> y;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          w.v[e] = to_f32(from_f32<T>(w.v[e]));
          y.v[e] = fmaf(own.v[e], w.v[e], w.v[e]);
        }
        for (int k = 0; k + 1 < cv.taps; ++k) {
          F32Vec<VEC> b{};
          if (read >= 0) b = load_vec<VEC>(cv.states + size_t(read) * cv.row_floats + size_t(k) * H + c);
          const F32Vec<VEC> f = load_vec<VEC>(cv.w + size_t(k) * H + c);
#pragma unroll
          for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(f.v[e], b.v[e], y.v[e]);
          if (write >= 0 && k > 0) store_vec<VEC>(cv.states + size_t(write) * cv.row_floats + size_t(k - 1) * H + c, b);
        }
        if (write >= 0 && cv.taps > 1)
          store_vec<VEC>(cv.states + size_t(write) * cv.row_floats + size_t(cv.taps - 2) * H + c, w);
        store_vec<VEC>(conv_out + size_t(row) * H + c, y);
      }
    }
  }
}

// The convolution alone, over packed sequences.  A thread takes VEC columns of `rows` rows; TAPS 0: any number of taps.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kRowThreads)
row_conv_kernel(const T* __restrict__ h, T* __restrict__ out, const RowConv cv, const int* __restrict__ row_seq,
                const int* __restrict__ cu_q, int M, int H, int rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * kRowThreads + threadIdx.x) * VEC, t0 = blockIdx.y * rows, t1 = min(M, t0 + rows);
  if (c >= H) return;
  const int taps = TAPS > 0 ? TAPS : cv.taps;
  constexpr int kWin = TAPS > 1 ? TAPS - 1 : 1;
  F32Vec<VEC> w[TAPS > 0 ? TAPS : 1], win[kWin];
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = load_vec<VEC>(cv.w + size_t(j) * H + c);
  }
  int begin = 0, end = -1, read = -1, write = -1;
  // the row `back` rows before row t (back < taps): of this pass, of the state, or zero
  auto before = [&](int t, int back) {
    if (t - back >= begin) return load_vec<VEC>(h + size_t(t - back) * H + c);
    if (read < 0) return F32Vec<VEC>{};
    return load_vec<VEC>(cv.states + size_t(read) * cv.row_floats + size_t(taps - 1 + t - back - begin) * H + c);
  };
  constexpr int kAhead = 4;                      // rows whose loads are under way together
  for (int tb = t0; tb < t1; tb += kAhead) {
    F32Vec<VEC> in[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (tb + j < t1) in[j] = load_vec<VEC>(h + size_t(tb + j) * H + c);
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int t = tb + j;
      if (t >= t1) break;
      if (t >= end) {                            // the block's first row, or a sequence's
        const int s = row_seq[t];
        begin = cu_q[s];
        end = cu_q[s + 1];
        read = cv.state_rows[s];
        write = cv.state_rows[cv.state_ld + s];
        if constexpr (TAPS > 1) {
#pragma unroll
          for (int k = 0; k < TAPS - 1; ++k) win[k] = before(t, TAPS - 1 - k);
        }
      }
      float* last = write >= 0 ? cv.states + size_t(write) * cv.row_floats + c : nullptr;
      if (last != nullptr && t == begin && end - begin < taps - 1)   // what stays of the rows before a short portion
        for (int k = 0; k + end - begin < taps - 1; ++k)
          store_vec<VEC>(last + size_t(k) * H, before(t, taps - 1 - k - (end - begin)));
      const F32Vec<VEC> x = in[j];
      F32Vec<VEC> y = x;
      if constexpr (TAPS > 0) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(w[TAPS - 1].v[e], x.v[e], y.v[e]);
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
          for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(w[k].v[e], win[k].v[e], y.v[e]);
        if constexpr (TAPS > 1) {
#pragma unroll
          for (int k = 0; k + 1 < TAPS - 1; ++k) win[k] = win[k + 1];
          win[TAPS - 2] = x;
        }
      } else {
        for (int k = 0; k < taps; ++k) {
          const F32Vec<VEC> f = load_vec<VEC>(cv.w + size_t(k) * H + c);
          const F32Vec<VEC> v = k + 1 == taps ? x : before(t, taps - 1 - k);
#pragma unroll
          for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(f.v[e], v.v[e], y.v[e]);
        }
      }
      store_vec<VEC>(out + size_t(t) * H + c, y);
      const int place = t - (end - (taps - 1));
      if (last != nullptr && place >= 0) store_vec<VEC>(last + size_t(place) * H, x);
    }
  }
}

// Launch over (cluster, rows) with VEC 4 where sizes and addresses allow it, else VEC `ANY`.
template <int ANY = 1, typename K, typename... Args>
int launch_rows(K vec_kern, K any_kern, bool aligned, int M, int H, cudaStream_t st, Args... args) {
  const bool vec = H % 4 == 0 && aligned;
  const int n = vec ? H / 4 : (H + ANY - 1) / ANY;
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
  return cudaLaunchKernelEx(&cfg, vec ? vec_kern : any_kern, args...) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

inline bool aligned16(std::initializer_list<const void*> ps) {
  for (const void* p : ps)
    if (reinterpret_cast<uintptr_t>(p) & 15) return false;
  return true;
}

template <typename T, typename S>
int launch_add_norm(void* residual, const void* planes, int n_planes, const void* slots, int n_slots, const void* scale,
                    int replace, const void* weight, float offset, void* out, int ldo, int M, int H, float eps,
                    cudaStream_t st) {
  return launch_rows(add_norm_kernel<T, S, 4, false>, add_norm_kernel<T, S, 1, false>,
                     aligned16({residual, weight, out, scale}) && ldo % 4 == 0, M, H, st,
                     reinterpret_cast<float*>(residual), reinterpret_cast<const float*>(planes), n_planes,
                     reinterpret_cast<const S*>(slots), n_slots, reinterpret_cast<const T*>(scale), replace,
                     reinterpret_cast<const T*>(weight), offset, reinterpret_cast<T*>(out), ldo, M, H, eps, RowConv{},
                     static_cast<T*>(nullptr));
}

RowConv conv_of(const ZseRowConv* z) {
  return RowConv{reinterpret_cast<const float*>(z->w), z->taps, reinterpret_cast<float*>(z->states),
                 (long long)(z->row_floats), reinterpret_cast<const int*>(z->state_rows), z->state_ld};
}

template <typename T>
int launch_add_norm_conv(void* residual, const void* planes, int n_planes, const void* weight, void* out, const ZseRowConv* z,
                         void* conv_out, int M, int H, float eps, cudaStream_t st) {
  return launch_rows(add_norm_kernel<T, float, 4, true>, add_norm_kernel<T, float, 1, true>,
                     aligned16({residual, weight, out, z->w, z->states, conv_out}) && z->row_floats % 4 == 0, M, H, st,
                     reinterpret_cast<float*>(residual), reinterpret_cast<const float*>(planes), n_planes,
                     static_cast<const float*>(nullptr), 0, static_cast<const T*>(nullptr), 0,
                     reinterpret_cast<const T*>(weight), 0.f, reinterpret_cast<T*>(out), H, M, H, eps, conv_of(z),
                     reinterpret_cast<T*>(conv_out));
}

template <typename T, int VEC>
cudaError_t launch_row_conv(const void* h, void* out, const ZseRowConv* z, const void* row_seq, const void* cu_q, int M, int H,
                            cudaStream_t st) {
  const int rows = M >= 4096 ? 32 : M >= 512 ? 8 : 4;
  const dim3 grid((H / VEC + kRowThreads - 1) / kRowThreads, (M + rows - 1) / rows);
  auto kern = z->taps == 2   ? row_conv_kernel<T, VEC, 2>
              : z->taps == 3 ? row_conv_kernel<T, VEC, 3>
              : z->taps == 4 ? row_conv_kernel<T, VEC, 4>
                             : row_conv_kernel<T, VEC, 0>;
  return launch_pdl(kern, grid, dim3(kRowThreads), 0, st, reinterpret_cast<const T*>(h), reinterpret_cast<T*>(out), conv_of(z),
                    reinterpret_cast<const int*>(row_seq), reinterpret_cast<const int*>(cu_q), M, H, rows);
}

// y = sum of fp32 planes + sum of the row's slots; residual += RMSNorm(y) * weight; out = residual, or (next != null)
// RMSNorm(residual) * next.  Rows are split as in add_norm_kernel.
template <typename T, typename S, int VEC>
__global__ void __launch_bounds__(kRowThreads)
post_norm_kernel(float* __restrict__ residual, const float* __restrict__ planes, int n_planes,
                 const S* __restrict__ slots, int n_slots, const T* __restrict__ weight, const T* __restrict__ next,
                 T* __restrict__ out, int M, int H, float eps) {
  __shared__ float red[2][32];
  __shared__ float cluster_ss[2];
  pdl_launch_dependents();
  const int row = blockIdx.y, cs = gridDim.x;
  const int nv = (H / VEC + cs - 1) / cs;
  const int v0 = blockIdx.x * nv, v1 = min(H / VEC, v0 + nv);
  const size_t base = size_t(row) * H, plane = size_t(M) * H;
  pdl_wait();
  F32Vec<VEC> x[kRowRegs];
  auto total_of = [&](float ss, int k) {
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[k][threadIdx.x >> 5] = ss;
    __syncthreads();
    const float t = warp_sum((threadIdx.x & 31) < (kRowThreads >> 5) ? red[k][threadIdx.x & 31] : 0.f);
    return row_cluster_sum(t, &cluster_ss[k], cs);
  };
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i < v1) {
      const size_t at = base + size_t(i) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[j].v[e] = 0.f;
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
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x[j].v[e] * x[j].v[e];
    }
  }
  float inv = 1.f / sqrtf(total_of(ss, 0) / float(H) + eps);
  ss = 0.f;
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i < v1) {
      const size_t at = base + size_t(i) * VEC;
      const F32Vec<VEC> r = load_vec<VEC>(residual + at), w = load_vec<VEC>(weight + size_t(i) * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        x[j].v[e] = r.v[e] + x[j].v[e] * inv * w.v[e];
        ss += x[j].v[e] * x[j].v[e];
      }
      store_vec<VEC>(residual + at, x[j]);
      if (next == nullptr) store_vec<VEC>(out + at, x[j]);
    }
  }
  if (next == nullptr) return;
  inv = 1.f / sqrtf(total_of(ss, 1) / float(H) + eps);
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i < v1) {
      F32Vec<VEC> w = load_vec<VEC>(next + size_t(i) * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) w.v[e] *= x[j].v[e] * inv;
      store_vec<VEC>(out + base + size_t(i) * VEC, w);
    }
  }
}

template <typename T, typename S>
int launch_post_norm(void* residual, const void* planes, int n_planes, const void* slots, int n_slots,
                     const void* weight, const void* next, void* out, int M, int H, float eps, cudaStream_t st) {
  return launch_rows(post_norm_kernel<T, S, 4>, post_norm_kernel<T, S, 1>, aligned16({residual, weight, out, next}), M, H,
                     st, reinterpret_cast<float*>(residual), reinterpret_cast<const float*>(planes), n_planes,
                     reinterpret_cast<const S*>(slots), n_slots, reinterpret_cast<const T*>(weight),
                     reinterpret_cast<const T*>(next), reinterpret_cast<T*>(out), M, H, eps);
}

// Embedding of a token, scaled, plus the row of a hashed bigram table (null: none), plus a sinusoidal position vector;
// residual = RMSNorm of the sum, `out` the same in the activations' type.
//   row of the table: (token before * mul_prev + token * mul_cur) mod buckets; `buckets` itself for a sequence's first token
//   position vector: entries 2i, 2i + 1 are the sine and cosine of position * turns[i] turns
// The token before the first one of a pass comes from last_token[state_rows[s]]; the sequence's last one goes to
// last_token[state_rows[ld + s]].
template <typename T, int VEC>                       // VEC 4, or 2 with a last column of its own when H is odd
__global__ void __launch_bounds__(kRowThreads)
embed_design_kernel(const ZseEmbed a, const T* __restrict__ table, const T* __restrict__ bigram, const T* __restrict__ norm,
                    const float* __restrict__ turns, T* __restrict__ out, Status* st) {
  __shared__ float red[32];
  __shared__ float cluster_ss;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.y, cs = gridDim.x, H = a.H;
  const int nv = ((H + VEC - 1) / VEC + cs - 1) / cs;
  const int v0 = blockIdx.x * nv, v1 = min((H + VEC - 1) / VEC, v0 + nv);
  const int* ids = reinterpret_cast<const int*>(a.ids);
  const int* row_seq = reinterpret_cast<const int*>(a.row_seq);
  const int* cu_q = reinterpret_cast<const int*>(a.cu_q);
  const int* state_rows = reinterpret_cast<const int*>(a.state_rows);
  int* last = reinterpret_cast<int*>(a.last_token);
  const bool first_cta = blockIdx.x == 0;
  int id = ids[t];
  const float p = float(reinterpret_cast<const int*>(a.positions)[t]);
  if (id < 0 || id >= a.vocab) {
    if (threadIdx.x == 0 && first_cta) report(st, kBadArgument, 62, unsigned(id));
    id = 0;
  }
  const T* src = table + size_t(id) * H;
  const T* add = nullptr;
  if (bigram != nullptr) {
    const int s = row_seq != nullptr ? row_seq[t] : t;
    long long prev = -1;
    if (cu_q != nullptr && cu_q[s] != t) {
      prev = ids[t - 1];
    } else {
      const int r = state_rows[s];
      if (r >= 0) prev = last[r];
    }
    long long row = a.buckets;
    if (prev >= 0) {
      row = (prev * a.mul_prev + (long long)(id) * a.mul_cur) % a.buckets;
      if (row < 0) row += a.buckets;
    }
    add = bigram + size_t(row) * H;
    if (threadIdx.x == 0 && first_cta && (cu_q == nullptr || cu_q[s + 1] == t + 1)) {
      const int w = state_rows[a.state_ld + s];
      if (w >= 0) last[w] = id;
    }
  }
  float ss = 0.f;
  F32Vec<VEC> x[kRowRegs];
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i < v1) {
      F32Vec<VEC> y{}, z{};
      if constexpr (VEC == 4) {
        y = load_vec<4>(src + i * 4);
        if (add != nullptr) z = load_vec<4>(add + i * 4);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e)
          if (i * VEC + e < H) {
            y.v[e] = to_f32(src[i * VEC + e]);
            if (add != nullptr) z.v[e] = to_f32(add[i * VEC + e]);
          }
      }
#pragma unroll
      for (int e = 0; e < VEC; e += 2) {
        const float f = turns[i * VEC + e], lo = turns[i * VEC + e + 1];       // turns per token, as two floats
        const float hi = p * f;
        const float r = (hi - rintf(hi)) + fmaf(p, lo, fmaf(p, f, -hi));
        float sn, cn;
        sincospif(2.f * r, &sn, &cn);
        y.v[e] = y.v[e] * a.scale + sn + z.v[e];
        y.v[e + 1] = i * VEC + e + 1 < H ? y.v[e + 1] * a.scale + cn + z.v[e + 1] : 0.f;
        ss += y.v[e] * y.v[e] + y.v[e + 1] * y.v[e + 1];
      }
      x[j] = y;
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = warp_sum((threadIdx.x & 31) < (kRowThreads >> 5) ? red[threadIdx.x & 31] : 0.f);
  total = row_cluster_sum(total, &cluster_ss, cs);
  const float inv = 1.f / sqrtf(total / float(H) + a.eps);
  float* res = reinterpret_cast<float*>(a.residual) + size_t(t) * H;
#pragma unroll
  for (int j = 0; j < kRowRegs; ++j) {
    const int i = v0 + threadIdx.x + j * kRowThreads;
    if (i >= v1) continue;
    if constexpr (VEC == 4) {
      F32Vec<4> w = load_vec<4>(norm + i * 4);
#pragma unroll
      for (int e = 0; e < 4; ++e) w.v[e] *= x[j].v[e] * inv;
      store_vec<4>(res + i * 4, w);
      store_vec<4>(out + size_t(t) * H + i * 4, w);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e)
        if (i * VEC + e < H) {
          const float y = x[j].v[e] * inv * to_f32(norm[i * VEC + e]);
          res[i * VEC + e] = y;
          out[size_t(t) * H + i * VEC + e] = from_f32<T>(y);
        }
    }
  }
}

template <typename T>
int launch_embed(const ZseEmbed* a, int M, void* status, cudaStream_t st) {
  return launch_rows<2>(embed_design_kernel<T, 4>, embed_design_kernel<T, 2>,
                        aligned16({a->table, a->bigram, a->norm, a->residual, a->out}), M, a->H, st, *a,
                        reinterpret_cast<const T*>(a->table), reinterpret_cast<const T*>(a->bigram),
                        reinterpret_cast<const T*>(a->norm), reinterpret_cast<const float*>(a->turns),
                        reinterpret_cast<T*>(a->out), reinterpret_cast<Status*>(status));
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

template <typename T>
static cudaError_t launch_embedding_typed(const void* table, const void* ids, void* out, int M, int H, int vocab, float scale,
                                          void* copy, int ld_copy, void* status, cudaStream_t st) {
  const bool vec = H % 4 == 0 && ld_copy % 4 == 0 && aligned16({table, out}) && !(reinterpret_cast<uintptr_t>(copy) & 7) &&
                   (sizeof(T) == 2 || aligned16({copy}));
  return launch_pdl(vec ? embedding_typed_kernel<T, 4> : embedding_typed_kernel<T, 1>, dim3(M), dim3(256), 0, st,
                    reinterpret_cast<const T*>(table), reinterpret_cast<const int*>(ids), reinterpret_cast<float*>(out), H,
                    vocab, scale, reinterpret_cast<T*>(copy), ld_copy, reinterpret_cast<Status*>(status));
}

extern "C" int zse_embedding_typed(int dtype, const void* table, const void* ids, void* out, int M, int H, int vocab,
                                   float scale, void* copy, int ld_copy, void* status, void* stream) {
  if (M <= 0) return 0;
  auto run = dtype == kBF16 ? launch_embedding_typed<bf16> : launch_embedding_typed<float>;
  return run(table, ids, out, M, H, vocab, scale, copy, ld_copy, status, ST(stream)) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_add_norm(int dtype, int slot_dtype, void* residual, const void* planes, int n_planes,
                            const void* slots, int n_slots, const void* scale, int replace, const void* weight,
                            float offset, void* out, int ldo, int M, int H, float eps, void* stream) {
  if (M <= 0) return 0;
  auto run = dtype == kF32        ? launch_add_norm<float, float>
             : slot_dtype == kF32 ? launch_add_norm<bf16, float>
                                  : launch_add_norm<bf16, bf16>;
  return run(residual, planes, n_planes, slots, n_slots, scale, replace, weight, offset, out, ldo, M, H, eps, ST(stream));
}

extern "C" int zse_add_norm_conv(int dtype, void* residual, const void* planes, int n_planes, const void* weight, void* out,
                                 const ZseRowConv* z, void* conv_out, int M, int H, float eps, void* stream) {
  if (M <= 0) return 0;
  if (z->taps < 1) return ZSE_ERR_SHAPE;
  auto run = dtype == kF32 ? launch_add_norm_conv<float> : launch_add_norm_conv<bf16>;
  return run(residual, planes, n_planes, weight, out, z, conv_out, M, H, eps, ST(stream));
}

extern "C" int zse_row_conv(int dtype, const void* h, void* out, const ZseRowConv* z, const void* row_seq, const void* cu_q,
                            int M, int H, void* stream) {
  if (M <= 0) return 0;
  if (z->taps < 1 || M > 65535 * 4) return ZSE_ERR_SHAPE;
  const bool vec = H % 4 == 0 && z->row_floats % 4 == 0 && aligned16({h, out, z->w, z->states});
  auto run = dtype == kF32 ? (vec ? launch_row_conv<float, 4> : launch_row_conv<float, 1>)
                           : (vec ? launch_row_conv<bf16, 4> : launch_row_conv<bf16, 1>);
  return run(h, out, z, row_seq, cu_q, M, H, ST(stream)) == cudaSuccess ? 0 : ZSE_ERR_LAUNCH;
}

extern "C" int zse_post_norm(int dtype, int slot_dtype, void* residual, const void* planes, int n_planes,
                             const void* slots, int n_slots, const void* weight, const void* next, void* out, int M, int H,
                             float eps, void* stream) {
  if (M <= 0) return 0;
  auto run = dtype == kF32        ? launch_post_norm<float, float>
             : slot_dtype == kF32 ? launch_post_norm<bf16, float>
                                  : launch_post_norm<bf16, bf16>;
  return run(residual, planes, n_planes, slots, n_slots, weight, next, out, M, H, eps, ST(stream));
}

extern "C" int zse_embed_design(int dtype, const ZseEmbed* a, int M, void* status, void* stream) {
  if (M <= 0) return 0;
  if (a->bigram != nullptr && a->buckets <= 0) return ZSE_ERR_SHAPE;
  return dtype == kBF16 ? launch_embed<bf16>(a, M, status, ST(stream)) : launch_embed<float>(a, M, status, ST(stream));
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
