// Differential attention over paged keys and values ("tiles" pages, see the cache module): shared declarations.
//
// Each head has two query / key maps of `dim` and one value of `vdim`; a map is a softmax attention of its own, and the head's
// output is rms(a1 - lam * a2) * post over its vdim values.  Query head h reads key/value head h / group.  A row sees the keys
// at most window - 1 positions before it (window 0: all of them).
// A page block (one page, one key/value head) is [K map 1 | K map 2 | V] of 16 tokens each, as 8 x 8 core matrices:
// element (token t, column j) of a part with D padded columns sits at (t / 8) * 8 D + (j / 8) * 64 + (t % 8) * 8 + j % 8.
#pragma once
#include "blaze/sm100.cuh"

namespace blz {

struct DiffParams {
  const void* qkv;             // [T, ld]: q [heads][2][dim] | k [kv_heads][2][dim] | v [kv_heads][vdim] of every row
  void* out;                   // [T, heads * vdim]
  void* pool;                  // page blocks
  long long ld, page_stride, head_stride;    // elements
  const int* block_table;
  const int* slots;            // [B]
  const int* q_start;          // [B + 1]
  const int* ctx_len;          // [B]
  const int* seq_of_row;       // [T], -1 = padding
  const int* slot_mapping;     // [T], -1 = padding
  float* part_o;               // partial outputs of split key ranges
  float* part_ml;
  int bt_stride, T, B, heads, kv_heads, dim, vdim, window;
  float scale, lam, post, eps;
  int max_rows;                // rows (new tokens * group) up to which a sequence belongs to the short-row kernel
  int row_blocks, splits, stages;
  int* status;

  __host__ __device__ int group() const { return heads / kv_heads; }
  __host__ __device__ int dp() const { return (dim + 15) / 16 * 16; }
  __host__ __device__ int vp() const { return (vdim + 15) / 16 * 16; }
  __host__ __device__ int block_elems() const { return 16 * (2 * dp() + vp()); }
};

// offset of (token, column) in a part with D padded columns
__host__ __device__ __forceinline__ int core_off(int t, int j, int D) { return (t >> 3) * 8 * D + (j >> 3) * 64 + (t & 7) * 8 + (j & 7); }

// first visible key position of a row at position `pos`
__device__ __forceinline__ int first_key(int pos, int window) { return window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0; }

}  // namespace blz
