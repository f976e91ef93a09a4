// C ABI of libzse_b200.so.  Every function takes raw device pointers and a cudaStream_t (as void*), launches
// asynchronously on that stream and returns 0 or a negative ZSE_ERR_* code; nothing here allocates device memory
// unless its name says so.  A device-side failure (a bounded wait that ran out, an index check) is reported through
// the 16-byte status word the caller passes in (see zse_status_*).
#pragma once
#include <stdint.h>

#define ZSE_ERR_SHAPE (-1)
#define ZSE_ERR_ALIGN (-2)
#define ZSE_ERR_DRIVER (-3)
#define ZSE_ERR_LAUNCH (-4)
#define ZSE_ERR_LIMIT (-5)

#ifdef __cplusplus
extern "C" {
#endif

// ---- runtime.cu ---------------------------------------------------------------------------------------------
// Programmatic dependent launch for the kernels of the decode path (on by default; ZSE_PDL=0 switches it off).
void zse_set_pdl(int on);
int zse_get_pdl(void);

// ---- gemm.cu ------------------------------------------------------------------------------------------------
// epilogue: 0 = fp16 store (+bias), 1 = SwiGLU (N counts gate+up rows, output has N/2 columns), 2 = fp32 partial planes
int zse_gemm_w4(const void* w_tiled, const void* x, int x_rows_cap, const void* bias, void* out, int M, int N, int K,
                int ldo, int epilogue, int k_split, void* status, void* stream);
int zse_gemm_w4_splits(int M, int N, int K, int k_split);
// the launcher's plan for a call: out4 = {tiles per wide CTA, K splits, cluster size, CTA shape: 0 wide, 1 narrow,
// -1 CUDA-core GEMV}
void zse_gemm_w4_plan(int M, int N, int K, int epilogue, int k_split, int sm_count, int* out4);
// ---- gemm_w4_dec.cu -----------------------------------------------------------------------------------------
// Decode-sized INT4 GEMM (M <= 64): one persistent CTA per SM over an even split of the weight stream.
// epilogue: 0 = fp16 store (+bias), 1 = SwiGLU, 2 = fp32 store.  `workspace`: zse_gemm_w4_dec_workspace_bytes bytes,
// zeroed once; one workspace serves the calls of ONE stream (calls that overlap on the GPU must not share it).
long long zse_gemm_w4_dec_workspace_bytes(int sm_count);
int zse_gemm_w4_dec_supported(int M, int N, int K, int epilogue);
int zse_gemm_w4_dec(const void* w_tiled, const void* x, int x_rows_cap, const void* bias, void* out, int M, int N,
                    int K, int ldo, int epilogue, void* workspace, void* status, void* stream);
// Fused QKV projection, head_dim 128, full rotary: bias + rotate-half RoPE (cos/sin table [max_position][64] of
// float2) + K/V rows into the paged cache [blocks][2][nkv][block_size][128]; qkv_out receives the rotated q heads.
int zse_gemm_w4_dec_qkv_rope(const void* w_tiled, const void* x, int x_rows_cap, const void* bias, void* qkv_out,
                             int ldo, int M, int K, int nh, int nkv, void* kv_layer, int block_size,
                             const void* positions_i32, const void* slots_i64, const void* cos_sin_f32x2,
                             int max_position, void* workspace, void* status, void* stream);
// the plan of a call: out2 = {CTAs, K segments per tile pair (0: the stream plan)}
void zse_gemm_w4_dec_plan(int N, int K, int epilogue, int sm_count, int* out2);
void zse_gemm_w4_dec_set_tuning(int min_steps, int max_split);

int zse_gemm_f16(const void* w, int w_rows_cap, const void* x, int x_rows_cap, const void* bias, void* out, int M,
                 int N, int K, int ldo, int epilogue, int k_split, void* status, void* stream);
int zse_gemm_f16_splits(int M, int N, int K, int k_split);
// the same kernel on bfloat16 weights and activations (epilogue 0: bfloat16 store, 2: fp32 planes)
// gated activation of two up products (tiles of 64 gate rows and their 64 up rows): out [M, cols]; kinds as in zse_glu
int zse_gemm_bf16_glu(const void* w, const void* x, int x_rows_cap, void* out, int M, int N, int K, int ldo, int cols,
                      int kind, void* status, void* stream);
// store in bfloat16, columns from side_col on in fp32 to side [M, N - side_col] instead
int zse_gemm_bf16_side(const void* w, const void* x, int x_rows_cap, void* out, int M, int N, int K, int ldo, void* side,
                       int side_col, void* status, void* stream);
int zse_gemm_bf16(const void* w, int w_rows_cap, const void* x, int x_rows_cap, void* out, int M, int N, int K, int ldo,
                  int epilogue, int k_split, void* status, void* stream);

// ---- gemm_tile.cu -------------------------------------------------------------------------------------------
// dtype of the functions below: 1 = bfloat16, 2 = float.
typedef struct ZseTileGemm {
  const void* a;            // [M, K], row stride lda, batch stride a_batch
  int64_t lda, a_batch;
  const void* b;            // element (n, k) at n * ldb_n + k * ldb_k, batch stride b_batch, expert stride b_group
  int64_t ldb_n, ldb_k, b_batch, b_group;
  void* out;                // row stride ldo, batch stride o_batch; row m goes to out_rows[m] or m * out_row_mul + add
  int64_t ldo, o_batch;
  int32_t M, N, K, epilogue;   // 0 store, 1 fp32 store, 2 gelu, 3 times sigmoid(gate), 4 square of relu
  const float* row_scale;      // factor of a row of the product, or null
  const int32_t* out_rows;
  int32_t out_row_mul, out_row_add;
  const void* gate;
  int64_t ldg, gate_batch;
  const void* tiles;        // grouped: MoeTile table and its length on the device (tiles of 64 rows)
  const int32_t* n_tiles;
} ZseTileGemm;
int zse_gemm_tile(int dtype, const ZseTileGemm* a, int batch, int max_tiles, void* stream);
// in [rows, 2 * ff] (gate, up) -> out [rows, ff]; kind 0: g sigmoid(1.702 g) (u + 1), g clamped from above and u from both
// sides; 1: silu(g) u; 2: gelu(g) u with the tanh form of gelu
int zse_glu(int dtype, const void* in, void* out, int ldo, int rows, int ff, int kind, float limit, void* stream);

int zse_apply_repetition_penalty_f32(void* logits, int ld, const void* rows_i32, const void* tokens_i32,
                                     const void* counts_i32, int n, const void* penalty_f32, int V, void* stream);

// ---- rows.cu ------------------------------------------------------------------------------------------------
int zse_embedding_typed(int dtype, const void* table, const void* ids, void* out_f32, int M, int H, int vocab,
                        float scale, void* copy, int ld_copy, void* status, void* stream);
// causal convolution along every sequence, per channel, of normed rows
typedef struct ZseRowConv {
  const void* w;                // fp32 [taps][H], a row's own tap last
  int32_t taps;
  void* states;                 // state rows, row_floats apart; this layer's part: the last taps - 1 rows, the oldest first
  int64_t row_floats;
  const void* state_rows;       // [2][state_ld]: rows that sequences read and write (-1: none)
  int32_t state_ld;
} ZseRowConv;
// residual += planes; out [M, H] = RMSNorm(residual) * weight; conv_out = out plus its convolution; every row is a sequence of
// its own
int zse_add_norm_conv(int dtype, void* residual, const void* planes, int n_planes, const void* weight, void* out,
                      const ZseRowConv* z, void* conv_out, int M, int H, float eps, void* stream);
// out = h plus its convolution, packed sequences: cu_q their first rows, row_seq the rows' sequences
int zse_row_conv(int dtype, const void* h, void* out, const ZseRowConv* z, const void* row_seq, const void* cu_q, int M, int H,
                 void* stream);
// y = planes [n_planes][M][H] + slots [M][n_slots][H], times scale [H] (null: 1); residual += y, or = y with replace;
// out [M, ldo] = RMSNorm(residual) * (weight + offset), or the residual itself without a weight
int zse_add_norm(int dtype, int slot_dtype, void* residual, const void* planes, int n_planes, const void* slots,
                 int n_slots, const void* scale, int replace, const void* weight, float offset, void* out, int ldo, int M,
                 int H, float eps, void* stream);
// y = planes + slots; residual += RMSNorm(y) * weight; out = residual, or (next not null) RMSNorm(residual) * next
int zse_post_norm(int dtype, int slot_dtype, void* residual, const void* planes, int n_planes, const void* slots,
                  int n_slots, const void* weight, const void* next, void* out, int M, int H, float eps, void* stream);
typedef struct ZseEmbed {
  const void *table, *bigram;   // [vocab, H], [buckets + 1, H] or null
  const void* norm;
  const void* turns;            // [ceil(H / 2)] pairs of floats: high and low part of the turns per token
  const void *ids, *positions;
  const void *row_seq, *cu_q;   // null: every row is a sequence of its own
  const void* state_rows;       // [2][state_ld]: rows of last_token that sequences read and write (-1: none)
  void* last_token;
  void *residual, *out;
  int64_t buckets, mul_prev, mul_cur;
  int32_t H, vocab, state_ld;
  float scale, eps;
} ZseEmbed;
int zse_embed_design(int dtype, const ZseEmbed* a, int M, void* status, void* stream);
// fp32 logits in place: cap * tanh(scale * x / cap) (cap 0: scale * x)
int zse_logits_finish(void* logits, int ld, int M, int V, float scale, float cap, void* stream);
int zse_argmax_f32(const void* logits, int ld, void* out_i32, int M, int V, void* stream);

// ---- latent.cu ----------------------------------------------------------------------------------------------
typedef struct ZseRowCache {
  void* rows;               // one layer's cached rows [blocks][block_size][row], blocks block_stride elements apart
  int64_t block_stride;
  int32_t block_size, row;
  const void* tables;       // block tables [sequences][max_blocks]
  int32_t max_blocks;
  int32_t num_blocks;       // blocks in the pool (0: unknown, the kernels that need a tensor map are not used)
} ZseRowCache;
typedef struct ZseChunks {  // sequences [first, last) of a packed pass
  const void *cu_q, *q_pos0, *ctx_off;
  int32_t first, last, window;
} ZseChunks;
int zse_latent_mma_ok(int heads, int dim, int rot, int vdim, int kv_rank, int row);
int zse_latent_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, int M, const ZseRowCache* c,
                    const void* positions, const void* slots, const void* freqs, const void* norm_w, int heads, int dim,
                    int rot, int rot_dims, int kv_rank, int latent_col, int gate_col, int gate_w, float eps,
                    void* stream);
// tensor_cores: 0 the general kernel, 1 tcgen05 where the shape allows (else as 2), 2 mma.sync
int zse_latent_attn(int dtype, const void* q_lat, const ZseRowCache* c, const void* row_seq, const void* positions,
                    void* o_lat, void* scratch, int M, int heads, int used, int kv_rank, int window, float scale,
                    int num_splits, int tensor_cores, void* status, void* stream);
int zse_latent_absorb(const void* inp, int ld, const void* uk, void* q_lat, int M, int heads, int dim, int rot,
                      int kv_rank, int row, void* stream);
int zse_latent_unabsorb(const void* o_lat, const void* uv, const void* gate, int ldg, void* out, int ldo, int M,
                        int heads, int vdim, int kv_rank, void* stream);
int zse_latent_gather(const ZseRowCache* c, const ZseChunks* g, int rows, int kv_rank, int rot, void* c_out,
                      void* kr_out, void* stream);
int zse_latent_chunk(const void* inp, int ld, const void* kvx, int ldkv, int v_col, const void* kr_ctx,
                     const ZseRowCache* c, const ZseChunks* g, int max_q, void* out, int ldo, const void* gate, int heads,
                     int dim, int rot, int vdim, float scale, void* stream);

// ---- moe.cu -------------------------------------------------------------------------------------------------
int zse_moe_tile_rows(int M, int E, int top);
// router logits (fp32 planes) -> chosen experts, sorted rows, tile table; `counts` [E] must be zero and is zero afterwards
typedef struct ZseRouter {
  const void* planes;         // fp32 logits [n_planes][M][cols]; column `experts`, if there is one: the shared expert's gate
  int32_t n_planes, experts, cols, top;
  int32_t softmax;            // scores: 0 sigmoid, 1 softmax over the experts
  int32_t normalise;          // weights: the chosen scores divided by their sum
  float scale;                // ... times this
  int32_t groups, keep;       // equal groups of neighbouring experts; experts come from the `keep` best of them
} ZseRouter;
int zse_moe_route(int dtype, const ZseRouter* r, int M, int tile_rows, const void* x, int H, int out_per_token, void* counts,
                  void* slot_expert, void* slot_rank, void* slot_score, void* first_row, void* tiles, void* n_tiles,
                  void* xs, void* row_score, void* out_rows, void* shared_score, void* stream);
typedef struct ZseMoeGemm {
  const void *routed_w, *routed_x;
  void* routed_out;
  const void *shared_w, *shared_x;
  void* shared_out;
  const void *row_score, *out_rows, *tiles, *n_tiles;
  const void* shared_score;   // per token, or null
  int32_t routed_n, routed_k, routed_ldo, shared_n, shared_k, shared_ldo, shared_mul, shared_add, shared_x_rows;
  int32_t routed_cols, shared_cols;     // gated: output columns (weight rows: tiles of 64 gate rows and 64 up rows)
  float routed_limit, shared_limit;
  int32_t glu;                // which gated activation, see zse_glu
} ZseMoeGemm;
int zse_moe_gemm(const ZseMoeGemm* g, int M, int E, int max_rows, int tile_rows, int max_tiles, int epilogue,
                 void* status, void* stream);

// ---- heads.cu -----------------------------------------------------------------------------------------------
typedef struct ZseHeads {
  void *k, *v;                  // cached keys and values: element (block, kv head, token, d) at block * block_stride +
  int64_t block_stride;         //   (head * block_size + token) * dim_pad + d (values: vdim_pad)
  int32_t block_size, dim_pad, vdim_pad, max_blocks;
  const void* tables;           // block tables [sequences][max_blocks], -1: a hole
  int32_t heads, kv_heads, dim, vdim, chunk, window;
  float scale;
  int32_t num_blocks;           // blocks in the pool
  int32_t keep_first;           // first positions that are seen whatever the window
  float softcap;                // > 0: scores become softcap * tanh(score / softcap)
  int32_t gate_each;            // a gate per dimension of a head's result, not per head
  int32_t pool;                 // > 0, with a window: blocks of that many tokens that lie before it are seen as their means,
  int32_t means_at;             //   rows of the cache whose blocks stand from this column on in a row of the tables
  const void* sink;             // fp32 [heads]: one more score without a value, null: none
  float out_scale;              // factor of the result
} ZseHeads;
// 1 when the tensor-core kernels take this shape (bfloat16)
int zse_heads_mma_ok(int dim, int vdim, int block_size);
// columns of a projected row: q from 0, k from k_col, v from v_col (k_col: the values are the keys as projected), gate from
// gate_col (gate_w of them); own_kv 0: no keys and values of its own
typedef struct ZseHeadsPrep {
  const void *q_norm, *k_norm;  // weights of the norms over a head's dimensions, null: 1; `whole`: over all heads'
  const void* bias;             // of the columns before gate_col, null: none
  const void* turns;            // pairs that rotate: [rot_dims / 2] high and low parts of the turns per position
  const void* positions;
  int32_t k_col, v_col, gate_col, gate_w, own_kv, rot_dims;
  float temp_coef;              // queries are multiplied by 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1)
  int32_t temp_every;
  float eps;
  int32_t whole;                // one norm over all query (key) heads, before the rotation
  const void* head_temp;        // `whole`: fp32 [heads], factor of a head's queries, null: 1
  int32_t pool_rows;            // `whole`: rows are sequences of their own, and one that completes a block of tokens leaves
                                //   its mean in the cache
} ZseHeadsPrep;
int zse_heads_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, int M, const ZseHeads* h,
                   const void* slots, const ZseHeadsPrep* p, void* stream);
// means of the blocks of h->pool tokens that rows [0, M) complete, from the cache into the cache; row_seq null: row t is
// sequence t
int zse_heads_pool(int dtype, const ZseHeads* h, const void* row_seq, const void* positions, int M, void* stream);
// rows [0, M) one by one; gate: first element of the gates (row stride ld), or null
int zse_heads_attn(int dtype, const void* inp, int ld, const ZseHeads* h, const void* row_seq, const void* positions,
                   void* out, int ldo, const void* gate, void* scratch, int M, int num_splits, int tensor_cores,
                   void* stream);
// rows of the sequences [first, last) in tiles of queries (bfloat16); rows: rows of inp; form: 1 tcgen05 where it takes the
// shape, 2 mma.sync
int zse_heads_attn_chunks(const void* inp, int ld, int rows, const ZseHeads* h, const void* cu_q, const void* q_pos0,
                          int first, int last, int max_q, void* out, int ldo, const void* gate, int form, void* status,
                          void* stream);

// ---- memory.cu ----------------------------------------------------------------------------------------------
typedef struct ZseMemory {
  int32_t heads, dim, vdim;
  int32_t k_col, v_col, gate_col, if_col;   // columns of a projected row (q from 0); if_col: input gates, then forget gates
  void* states;                 // state rows, row_floats apart; this layer's part: memory at 0, key sum at sum_at, max at max_at
  int64_t row_floats;
  int32_t sum_at, max_at;
  const void* state_rows;       // [2][state_ld]: rows that sequences read and write (-1: none)
  int32_t state_ld;
  float gate_cap, eps;
  const void* head_norm;        // [heads * vdim], activations' type
} ZseMemory;
int zse_memory_chunk_ok(int dim, int vdim);
int zse_memory_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, const void* gate_planes,
                    int n_gate_planes, const void* if_bias, void* gates, const ZseMemory* m, int M, void* stream);
// sequences [0, S), token by token: update, read-out, head norm, output gate; cu_q null: a row each
int zse_memory_tokens(int dtype, const void* inp, int ld, const void* gates, const ZseMemory* m, const void* cu_q, int S,
                      void* out, int ldo, void* stream);
// sequences [first, last) chunkwise (bfloat16): read-outs to o [M, heads * vdim] fp32, then head norm and output gate
int zse_memory_chunks(const void* inp, int ld, const void* gates, const ZseMemory* m, const void* cu_q, int first, int last,
                      void* o, int M, int first_row_of_first, void* out, int ldo, void* stream);

// ---- state_space.cu -----------------------------------------------------------------------------------------
typedef struct ZseSpace {
  int32_t heads, vdim, state, groups, taps;
  int32_t x_col;                // columns of a projected row: z from 0, the channels x, B, C from x_col, step sizes from dt_col
  int32_t b_at, c_at, conv_width;   // the channels' layout, in a projected row from x_col on and in the convolution's output
  int32_t dt_col;
  void* states;                 // state rows, row_floats apart; this layer's part: S at 0, the convolution's inputs at conv_at
  int64_t row_floats;
  int32_t conv_at;
  const void* state_rows;       // [2][state_ld]: rows that sequences read and write (-1: none)
  int32_t state_ld;
  const void *conv_w, *conv_b;  // fp32 [taps][conv_width] (a row's own tap last), [conv_width]
  const void *dt_bias, *neg_a, *skip;   // fp32 [heads]
} ZseSpace;
int zse_space_chunk_ok(int state, int vdim);
// planes: of the input projection (0: inp is complete; side [M][side_ld]: its step sizes in fp32, or null); xbc
// [M][conv_width], dt fp32 [M][heads]; row_seq, cu_q null: every row is a sequence of its own
int zse_space_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, const void* side, int side_ld,
                   const ZseSpace* m, const void* row_seq, const void* cu_q, void* xbc, void* dt, int M, void* stream);
// sequences [0, S), token by token: update, read-out, gate silu(z); cu_q null: a row each
int zse_space_tokens(int dtype, const void* inp, int ld, const void* xbc, const void* dt, const ZseSpace* m,
                     const void* cu_q, int S, void* out, int ldo, void* stream);
// sequences [first, last) chunkwise (bfloat16)
int zse_space_chunks(const void* inp, int ld, const void* xbc, const void* dt, const ZseSpace* m, const void* cu_q, int first,
                     int last, void* out, int ldo, void* stream);
// rows [M][ld] in place: `parts` parts of `width` columns, each divided by its root mean square, times weight
int zse_group_norm(int dtype, void* x, int ld, int M, int parts, int width, const void* weight, float eps, void* stream);

// ---- gated_linear.cu ----------------------------------------------------------------------------------------
typedef struct ZseGatedLinear {
  int32_t heads, dim, vdim, rank;
  int32_t q_col, k_col, v_col, gate_col, rank_col;   // columns of a projected row; rank_col: the decays' inner vector
  void* states;                 // state rows, row_floats apart; this layer's part: [heads][dim][vdim]
  int64_t row_floats;
  const void* state_rows;       // [2][state_ld]: rows that sequences read and write (-1: none)
  int32_t state_ld;
  float tau, eps, out_scale;
  const void* head_norm;        // [vdim], shared by the heads
  const void *decay_w, *decay_b;   // fp32 [heads * dim][rank], [heads * dim]
} ZseGatedLinear;
int zse_gated_linear_chunk_ok(int dim, int vdim);
// split-K planes of its columns -> inp (n_planes 0: inp is complete; side [M][side_ld]: its inner vectors in fp32, or null);
// decays: fp32 [M][heads * dim], logarithms
int zse_gated_linear_prep(int dtype, void* inp, int ld, const void* planes, int n_planes, const void* side, int side_ld,
                          const ZseGatedLinear* z, void* decays, int M, void* stream);
// sequences [0, S), token by token: update, read-out, head norm, output gate; cu_q null: a row each; decays null: inp and the
// decays' inner vectors are in the planes
int zse_gated_linear_tokens(int dtype, const void* inp, int ld, const void* planes, int n_planes, int M, const void* decays,
                            const ZseGatedLinear* z, const void* cu_q, int S, void* out, int ldo, void* stream);
// sequences [first, last) chunkwise (bfloat16), whose rows are [row0, M); o: fp32 [M][heads * vdim] scratch
int zse_gated_linear_chunks(const void* inp, int ld, const void* decays, const ZseGatedLinear* z, const void* cu_q, int first,
                            int last, void* o, int M, int row0, void* out, int ldo, void* stream);

// ---- repack.cu ----------------------------------------------------------------------------------------------
// Row-major INT4 [N, K/2] + scales/zeros [N, K/128] -> tiled chunks.  interleave_rows > 0 builds a fused gate/up
// tensor: `packed` holds gate rows [0, interleave_rows) then up rows; output tile t = 64 gate rows + 64 up rows.
int64_t zse_w4_tiled_bytes(int N, int K);
int zse_repack_w4(const void* packed, const void* scales, const void* zeros, void* out_tiled, int N, int K,
                  int interleave_rows, void* stream);
int zse_dequant_w4(const void* packed, const void* scales, const void* zeros, void* out_f16, int64_t n_elements,
                   int group_size, void* stream);
int zse_dequant_w8(const void* q, const void* scales, void* out_f16, int64_t n_elements, int group_size, void* stream);
int zse_quantize_w4(const void* w_f16, void* packed, void* scales, void* zeros, int64_t n_groups, void* stream);

// ---- elementwise.cu -----------------------------------------------------------------------------------------
int zse_embedding(const void* table_f16, const void* ids_i32, void* out_f32, int M, int H, int vocab, float scale,
                  void* status, void* stream);
// residual[M,H] (fp32, in/out) += sum of n_partials fp32 planes (stride M*H) [+ add_f16]; out = rmsnorm(residual)*w
int zse_add_rmsnorm(void* residual, const void* partials, int n_partials, const void* add_f16, const void* weight,
                    void* out_f16, int M, int H, float eps, void* stream);
int zse_rmsnorm_f16(const void* x_f16, const void* weight, void* out_f16, int M, int H, float eps, void* stream);
// qkv fp16 [M, (nh+2nkv)*hd]; rotates q and k in place (rotate-half), writes k and v into the paged cache
// kv_layer: [num_blocks][2][nkv][block_size][hd] fp16; slot = block*block_size + offset, -1 = skip;
// inv_freq: fp32 [rotary_dim/2] (theta^(-2i/rotary_dim), with any rope scaling already applied by the host)
// planes != NULL: q/k/v are read as n_planes fp32 planes [n_planes][M][(nh+2nkv)*hd] plus bias_f16 (may be NULL)
// instead of from qkv, and qkv only receives the rotated q
int zse_rope_kv_write(void* qkv, void* kv_layer, const void* positions_i32, const void* slots_i64,
                      const void* inv_freq_f32, int M, int nh, int nkv, int hd, int rotary_dim, int block_size,
                      const void* planes_f32, int n_planes, const void* bias_f16, void* stream);
int zse_swiglu(const void* gate_up_f16, void* out_f16, int M, int I, int gelu, void* stream);
int zse_bias_add(void* x_f16, const void* bias_f16, int M, int N, void* stream);
// dst[r, :] = src[rows_i64[r], :] for r < n (fp16 rows of H elements, H and ld multiples of 8)
// Diagnostic: `ctas` CTAs read `bytes` of `buf` `repeats` times (16-byte loads past L1); the caller times the launch.
int zse_read_probe(const void* buf, long long bytes, int repeats, int ctas, void* sink_u32, void* stream);
int zse_gather_rows_f16(const void* src_f16, int ld, const void* rows_i64, void* dst_f16, int n, int H, int src_rows,
                        void* status, void* stream);

// ---- gemma.cu: Gemma-family layers ------------------------------------------------------------------------------
// qkv fp16 [M, ld]: q heads, k heads, v heads (no v columns when k_is_v: V is then the raw k projection).  Per head:
// RMSNorm (q, k with the given fp16 weights [hd], NULL = none; v without weight when norm_v), RoPE on pairs
// (i, i + hd/2) with freqs_f32[i] (0 = pair not rotated), q written back in place, k and v into the cache of this
// layer: element (block, half, kv_head, offset, d) at block*blk_stride + half*half_stride + (kv_head*block_size +
// offset)*hd + d.
int zse_headnorm_rope_kv_write(void* qkv, int ld, void* kv_layer, int64_t blk_stride, int64_t half_stride,
                               const void* positions_i32, const void* slots_i64, const void* freqs_f32,
                               const void* q_norm_w, const void* k_norm_w, int norm_v, int k_is_v, float eps, int M,
                               int nh, int nkv, int hd, int block_size, void* stream);
// paged attention for any even head_dim <= 512.  Decode: cu_q = q_pos0 = NULL, query t belongs to sequence t at
// position seq_lens[t]-1.  Prefill: queries packed by cu_q, first query of sequence s at position q_pos0[s].
// softcap > 0: scores = softcap*tanh(scores/softcap); window > 0: only the last `window` positions are seen.
int zse_attn_generic(const void* q, int ldq, const void* kv_layer, int64_t blk_stride, int64_t half_stride,
                     const void* block_tables_i32, int max_blocks, const void* seq_lens_i32, const void* cu_q_i32,
                     const void* q_pos0_i32, int num_seqs, void* out_f16, int ldo, int T, int nh, int nkv, int hd,
                     int block_size, float scale, float softcap, int window, void* stream);
// residual = (residual + RMSNorm(x)*w_post) * scalar_f16[0] (scalar may be NULL); out = RMSNorm(residual)*w_next
// (out may be NULL)
int zse_norm_add_rmsnorm(const void* x_f16, const void* w_post, void* residual_f32, const void* scalar_f16,
                         const void* w_next, void* out_f16, int M, int H, float eps, void* stream);
int zse_softcap_f16(void* x_f16, int ld, int M, int V, float cap, void* stream);

// ---- attention.cu -------------------------------------------------------------------------------------------
int64_t zse_attn_decode_scratch_floats(int num_seqs, int nh, int hd, int max_splits);
int zse_attn_decode(const void* q, int ldq, const void* kv_layer, const void* block_tables_i32, int max_blocks,
                    const void* seq_lens_i32, void* out_f16, int ldo, void* scratch_f32, int num_seqs, int nh, int nkv,
                    int hd, int block_size, int num_splits, float scale, void* stream);
// causal attention of `total_q` query tokens (several sequences packed) over the paged cache.
// cu_q: [num_seqs+1] prefix offsets of query tokens; q_pos0[s]: cache position of the first query token of seq s.
int zse_attn_prefill(const void* q, int ldq, const void* kv_layer, const void* block_tables_i32, int max_blocks,
                     const void* cu_q_i32, const void* q_pos0_i32, void* out_f16, int ldo, int num_seqs, int max_q_len,
                     int nh, int nkv, int hd, int block_size, float scale, void* stream);
// The same on the tcgen05 tensor cores (attention_tc.cu): head_dim 128, contiguous cache layer of `num_blocks` blocks,
// `total_rows` rows in q.  ZSE_ERR_SHAPE for shapes it does not cover.
int zse_attn_prefill_tc(const void* q, int ldq, int total_rows, const void* kv_layer, int num_blocks,
                        const void* block_tables, int max_blocks, const void* cu_q, const void* q_pos0, void* out,
                        int ldo, int num_seqs, int max_q_len, int nh, int nkv, int hd, int block_size, float scale,
                        int variant, void* status, void* stream);

// the same kernels with an explicit cache addressing (element (block, half, kv_head, offset, d) at block*blk_stride +
// half*half_stride + (kv_head*block_size + offset)*hd + d; strides in elements, multiples of 8), soft-capped scores
// (softcap > 0: cap*tanh(score/cap)) and a sliding window (window > 0: only the last `window` positions are seen).
// head_dim 64, 128 or 256.
int zse_attn_decode_ext(const void* q, int ldq, const void* kv_layer, int64_t blk_stride, int64_t half_stride,
                        const void* block_tables_i32, int max_blocks, const void* seq_lens_i32, void* out_f16, int ldo,
                        void* scratch_f32, int num_seqs, int nh, int nkv, int hd, int block_size, int num_splits,
                        float scale, float softcap, int window, void* stream);
int zse_attn_prefill_ext(const void* q, int ldq, const void* kv_layer, int64_t blk_stride, int64_t half_stride,
                         const void* block_tables_i32, int max_blocks, const void* cu_q_i32, const void* q_pos0_i32,
                         void* out_f16, int ldo, int num_seqs, int max_q_len, int nh, int nkv, int hd, int block_size,
                         float scale, float softcap, int window, void* stream);

// ---- sampling.cu --------------------------------------------------------------------------------------------
int zse_argmax(const void* logits_f16, int ld, void* out_i32, int M, int V, void* stream);
int zse_sample(const void* logits_f16, int ld, void* out_i32, int M, int V, const void* temperature_f32,
               const void* top_k_i32, const void* top_p_f32, const void* seeds_u64, uint64_t step, void* stream);
// sparse form: entry i scales logits[rows[i], tokens[i]] by penalty[rows[i]]^(1+log2(counts[i]))
int zse_apply_repetition_penalty(void* logits_f16, int ld, const void* rows_i32, const void* tokens_i32,
                                 const void* counts_i32, int n, const void* penalty_f32, int V, void* stream);

// ---- lora.cu ------------------------------------------------------------------------------------------------
// y[t, :] += scale[a] * B[a] (A[a] x[t, :]) with a = adapter_ids[t] (-1 = none); A: [n_adapters][r][K], B: [n_adapters][N][r]
int zse_lora_shrink(const void* x_f16, int ldx, const void* a_f16, const void* adapter_ids_i32, void* tmp_f32, int M,
                    int K, int rank, void* stream);
int zse_lora_expand(const void* tmp_f32, const void* b_f16, const void* adapter_ids_i32, const void* scales_f32,
                    void* y_f16, int ldy, int M, int N, int rank, void* stream);
// shrink + expand in one launch, the activation row read once per token (rank even, <= 64)
int zse_lora_apply(const void* x, int ldx, const void* a, const void* b, const void* ids, const void* scales, void* y,
                   int ldy, int M, int K, int N, int rank, void* stream);

// ---- comm.cu ------------------------------------------------------------------------------------------------
// Tensor-parallel context: peer-mapped symmetric buffers of every rank (row data [2][m_cap][H] fp16, flags
// [2][tp][m_cap] u32, exchange words [2][tp][m_cap] u64 + flags), optional multicast view of the row data.
void* zse_tp_ctx_create(int tp, int rank, int m_cap, int H, const uint64_t* data_ptrs, const uint64_t* flag_ptrs,
                        uint64_t mc_data, const uint64_t* xchg_ptrs, const uint64_t* xflag_ptrs);
void zse_tp_ctx_destroy(void* ctx);
int zse_tp_reduce_add_rmsnorm(void* ctx, void* residual, const void* partials, int n_planes, const void* weight,
                              void* out, int M, float eps, int slot, int use_multimem, void* status,
                              void* stream);
int zse_tp_reduce_add_rmsnorm_emulated(void* ctx, const uint64_t* residuals, const uint64_t* partials, int n_planes,
                                       const void* weight, const uint64_t* outs, int M, float eps,
                                       int slot, void* status, void* stream);
// Two-shot form for many rows (prefill): reduce-scatter by rows (row r is reduced by rank r % tp, which also keeps the
// only current copy of the fp32 residual row) + all-gather of the normalised rows, in one kernel.
int zse_tp_reduce_scatter_add_rmsnorm(void* ctx, void* residual, const void* partials, int n_planes,
                                      const void* weight, void* out, int M, float eps, int slot, int use_multimem,
                                      void* status, void* stream);
int zse_tp_reduce_scatter_add_rmsnorm_emulated(void* ctx, const uint64_t* residuals, const uint64_t* partials,
                                               int n_planes, const void* weight, const uint64_t* outs, int M,
                                               float eps, int slot, void* status, void* stream);
// Push exchange: the row-parallel INT4 GEMM sends its fp16 partial rows to every rank's inbox from its own epilogue
// (multimem.st through NVSwitch or one store per peer) and counts its CTAs in; the consumer waits for the counters,
// adds the tp rows of its own inbox in rank order, adds the residual and applies RMSNorm.
//   inbox_ptrs[r]  : rank r's inbox [2][tp][push_m_cap][H] fp16 as mapped into this process (symmetric memory)
//   arrive_ptrs[r] : rank r's counters [2][tp] u32 (symmetric memory, zero at start)
//   state_ptrs[r]  : 4 u32 of ordinary device memory of rank r (zero at start); only the own rank's is needed
int zse_tp_ctx_set_push(void* ctx, int push_m_cap, const uint64_t* inbox_ptrs, uint64_t mc_inbox,
                        const uint64_t* arrive_ptrs, uint64_t mc_arrive, const uint64_t* state_ptrs);
// returns the number of CTAs launched (what the consumer waits for from every rank) or a negative error
int zse_tp_gemm_w4_push(void* ctx, const void* w_tiled, const void* x, int x_rows_cap, int M, int N, int K, int slot,
                        int use_multimem, int rank_override, void* status, void* stream);
// Decode-sized passes (M <= 64): row-parallel projection (INT4 or INT8 tiles), the exchange of the partial rows, the
// residual add and the next RMSNorm in ONE kernel (gemm_w4_dec.cu).  tp = 1 contexts work too (nothing to exchange).
int zse_tp_gemm_dec_allreduce_norm(void* ctx, const void* w_tiled, int int8_weights, const void* x, int x_rows_cap,
                                   int M, int N, int K, int slot, int use_multimem, int rank_override, void* residual,
                                   const void* norm_w, void* xnorm, float eps, void* workspace, void* status,
                                   void* stream);
int zse_tp_sum_add_rmsnorm(void* ctx, void* residual, const void* weight, void* out, int M, float eps, int slot,
                           int expected_add, void* status, void* stream);
int zse_tp_sum_add_rmsnorm_emulated(void* ctx, const uint64_t* residuals, const void* weight, const uint64_t* outs,
                                    int M, float eps, int slot, int expected_add, void* status, void* stream);
// Sequence-parallel exchange for passes of more than 64 rows (prefill): token rows are owned in blocks of 64
// (block b -> rank b % tp).  The row-parallel GEMM scatters its fp16 partial tiles to the owners from its epilogue;
// the owner adds, applies residual + RMSNorm and stores the row into the gathered buffer of every rank; GEMMs that
// read the gathered buffer wait, in their prologue, for the row blocks of their own token tile.
//   inbox_ptrs[r]  : rank r's inbox [2][tp][own_cap][H] fp16   arrive_ptrs[r] : counters [2][tp][nblk_cap] u32
//   xg_ptrs[r]     : gathered activations [nblk_cap * 64][H]    gflag_ptrs[r]  : flags [nblk_cap] u32
//   state_ptrs[r]  : 4 + nblk_cap u32 of ordinary device memory of rank r (all zero at start)
int zse_tp_ctx_set_sp(void* ctx, int own_cap, int nblk_cap, const uint64_t* inbox_ptrs, const uint64_t* arrive_ptrs,
                      const uint64_t* xg_ptrs, uint64_t mc_xg, const uint64_t* gflag_ptrs, const uint64_t* state_ptrs);
int zse_tp_gemm_w4_scatter(void* ctx, const void* w_tiled, const void* x, int x_rows_cap, int M, int N, int K,
                           int slot, int rank_override, void* status, void* stream);
int zse_tp_gemm_w4_gathered(void* ctx, const void* w_tiled, const void* x, int x_rows_cap, const void* bias, void* out,
                            int M, int N, int K, int ldo, int epilogue, int k_split, int rank_override, void* status,
                            void* stream);
int zse_tp_sp_sum_norm_gather(void* ctx, void* residual, const void* weight, int M, float eps, int slot,
                              int use_multimem, void* status, void* stream);
int zse_tp_sp_sum_norm_gather_emulated(void* ctx, const uint64_t* residuals, const void* weight, int M, float eps,
                                       int slot, void* status, void* stream);
int zse_tp_sp_wait(void* ctx, int M, int rank_override, void* status, void* stream);
// All-gather of vocabulary-sharded logits rows over NVLink (peer stores + per-row flags): buf_ptrs[r] = rank r's gathered
// rows [2][rows_cap][tp * width] fp16, flag_ptrs[r] = its flags [2][tp][rows_cap] u32, both symmetric memory.
int zse_tp_ctx_set_gather(void* ctx, int rows_cap, int width, const uint64_t* buf_ptrs, const uint64_t* flag_ptrs);
int zse_tp_gather_rows(void* ctx, const void* logits, int ld, int M, int slot, void* status, void* stream);
int zse_tp_gather_rows_emulated(void* ctx, const uint64_t* logits, int ld, int M, int slot, void* status, void* stream);
int zse_tp_argmax(void* ctx, const void* logits, int ld, void* out, int M, int V_local, int vocab_stride,
                  int slot, void* status, void* stream);
int zse_tp_argmax_emulated(void* ctx, const uint64_t* logits, int ld, const uint64_t* outs, int M, int V_local,
                           int vocab_stride, int slot, void* status, void* stream);

// ---- runtime.cu ---------------------------------------------------------------------------------------------
int zse_status_read(const void* status_dev, uint32_t* out4);   // synchronous 16-byte copy
int zse_device_info(int* sm_count, int* cc_major, int* cc_minor, int64_t* total_mem, int64_t* free_mem);
const char* zse_build_info(void);

#ifdef __cplusplus
}
#endif
