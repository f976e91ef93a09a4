// Addressing of cached latent rows, and the tensor-core form of decode attention over them (latent_tc.cu).
#pragma once
#include "typed.cuh"

namespace zse {

struct RowCache {
  long long block_stride;       // elements between blocks
  int block_size, row;          // tokens per block, elements per row
  const int* tables;            // [sequences][max_blocks]
  int max_blocks;
};

bool latent_tc_ok(const RowCache& rc, int num_blocks, int used, int kv_rank);
int launch_latent_tc(const bf16* q_lat, const void* rows, const RowCache& rc, int num_blocks, const int* row_seq,
                     const int* positions, bf16* o_lat, float* scratch, int M, int heads, int used, int kv_rank, int window,
                     float scale, int num_splits, Status* status, cudaStream_t st);

}  // namespace zse
