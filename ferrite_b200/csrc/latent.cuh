// Arguments of fb_latent_attention as its kernels see them.
#pragma once
#include "common.cuh"

namespace fb {

struct LatentArgs {
  const void* q;  // [T, ld_q]: head h of a token at h * (rank + rot), its query in the latent's space and its rotated part
  int64_t T, ld_q;
  int heads, rank, rot;
  const void* cache;  // [cache_rows, rank + rot]
  int64_t cache_rows;
  const int32_t* base;  // [T] first cache row of each token's sequence, or null
  int64_t row0;         // added to it
  const int32_t* last;  // [T] token t sees the rows 0 .. last[t] of its sequence
  int64_t max_keys;     // an upper bound of last[t] + 1
  int window;           // 0: none; else only the last `window` of those
  int chunk;            // the tokens are one sequence's, in order (base null): they may share the rows read
  float scale;
  const float* sink;  // [heads] or null
  void* out;          // [T, ld_o]: head h at h * rank
  int64_t ld_o;
  void* workspace;
  size_t workspace_bytes;
};

// latent_tcgen05.cu: bf16 rows on the tensor cores
bool latent_tcgen05_supports(const LatentArgs& a);
size_t latent_tcgen05_workspace(int64_t T, int heads, int rank, int rot, int64_t max_keys, int chunk, int window);
int latent_tcgen05(const LatentArgs& a, cudaStream_t s);

}  // namespace fb
