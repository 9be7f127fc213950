// What the kernels of attention over cached rows (latent attention in its cached form, keys that are also the values)
// share; see latent_attn.cu.
#pragma once

#include "tcgen05.cuh"

namespace axb {

struct AttendParams {
  const void *q_lat;  // (rows, heads, kv_rank)
  const void *q;      // (rows, q_ld): the rotated part of head h starts at h * (dim + rot_dim) + dim
  int64_t q_ld;
  void *out;  // (rows, heads, kv_rank)
  const void *pages;
  const int32_t *block_table, *row_seq, *row_pos;
  int rows, heads, dim, kv_rank, rot_dim, page_tokens, max_blocks, num_pages, max_seqs, max_len;
  float scale;
  unsigned long long wait_ns;
  int kv_heads;       // a token caches kv_heads rows, each for heads / kv_heads query heads; in a page head by head
  int row_elems;      // of one such row: kv_rank + rot_dim
  int page_elems;     // elements from one page to the next
  int key_scale;      // whether a page ends, behind its rows, with an fp32 factor of the keys of each row
  int window;         // keys a row sees, itself included; 0: all
  const float *sink;  // (heads): logit that takes part in the softmax's denominator only, or null
};

// Keys row r may read: 0 .. row_pos[r], never beyond the block table's reach or the host's bound.
__device__ __forceinline__ int visible_keys(const AttendParams &p, int r) {
  const int seq = p.row_seq[r];
  if (seq < 0 || seq >= p.max_seqs) return 0;
  const int cover = min(p.max_blocks * p.page_tokens, p.max_len);
  return max(0, min(p.row_pos[r] + 1, cover));
}

// The first key row r sees.
__device__ __forceinline__ int first_key(const AttendParams &p, int r) {
  return p.window > 0 ? max(0, p.row_pos[r] + 1 - p.window) : 0;
}

// The factors of a page's rows (see shared_kv.cu).
template <typename T>
__device__ __forceinline__ const float *page_factors(const T *page, const AttendParams &p) {
  return reinterpret_cast<const float *>(page + (size_t)p.kv_heads * p.page_tokens * p.row_elems);
}

// tcgen05 form for bf16 (latent_umma.cu)
size_t latent_umma_workspace_bytes(int part_heads, int kv_rank, int rot_dim);
bool latent_umma_supported(const AttendParams &p);
int latent_umma(const AttendParams &p, void *workspace, cudaStream_t st);

}  // namespace axb
