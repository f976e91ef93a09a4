// Addressing and masks of attention over cached heads (heads.cu, heads_tc.cu).
#pragma once
#include "typed.cuh"

namespace zse {

struct Heads {
  long long block_stride;
  int block_size, dp, vp, max_blocks;            // dp, vp: padded widths
  int block_shift;                               // log2 of the block size, -1: no power of two
  const int* tables;
  int heads, kv_heads, dim, vdim, chunk, window;
  float scale;
  int keep;                                      // first positions that are seen whatever the window
  float cap;                                     // > 0: scores become cap * tanh(score / cap)
  int gate_each;                                 // a gate per dimension of a head's result, not per head
  int pool, means_at;                            // > 0: what lies before the window is seen as means of blocks of `pool` tokens;
                                                 // rows of the cache whose blocks stand from column means_at on in the tables
  const float* sink;                             // a score per head without a value, null: none
  float out_scale;                               // factor of the result
  // means that a row at `pos` sees: those of the blocks that lie wholly before its window
  __device__ __forceinline__ int means_seen(int pos) const { return max(0, pos + 1 - window) / pool; }
  // a head's sink as a score in units of ln 2
  __device__ __forceinline__ float sink_log2(int head) const { return sink[head] * kLog2E; }
  // whether a row at `pos`, which sees from lo = first_seen(pos) on, sees position p
  __device__ __forceinline__ bool sees(int p, int pos, int lo) const { return p <= pos && (p >= lo || p < keep); }
  // cap * tanh(score / cap) of a scaled score; within 2^-22 of cap
  __device__ __forceinline__ float capped(float s) const {
    const float e = ex2(s * (2.f * kLog2E / cap));
    return fmaf(-2.f * cap, rcp(1.f + e), cap);
  }
  // place of the gate of a head's dimension d among a row's gates
  __device__ __forceinline__ int gate_at(int head, int d) const { return gate_each ? head * vdim + d : head; }
  __device__ __forceinline__ int first_seen(int pos) const {
    return chunk > 0 ? pos / chunk * chunk : window > 0 ? max(0, pos + 1 - window) : 0;
  }
  __device__ __forceinline__ int block_of(int token) const {
    return block_shift >= 0 ? token >> block_shift : token / block_size;
  }
  __device__ __forceinline__ int in_block(int token) const {
    return block_shift >= 0 ? token & (block_size - 1) : token % block_size;
  }
  // first element of a token's key (dp) or value (vp)
  __device__ __forceinline__ size_t at(int block, int head, int token, int width) const {
    return size_t(block) * block_stride + (size_t(head) * block_size + token) * width;
  }
};

bool heads_tc_ok(const Heads& h, int num_blocks, int ld, int ldo);
// `rows`: rows of inp; num_blocks: blocks of the pool
int launch_heads_tc(const bf16* inp, int ld, int rows, const void* k, const void* v, int num_blocks, const Heads& h,
                    const int* cu_q, const int* q_pos0, int first, int last, int max_q, bf16* out, int ldo,
                    const bf16* gate, Status* status, cudaStream_t st);

}  // namespace zse
