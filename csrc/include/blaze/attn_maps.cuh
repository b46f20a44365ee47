// Softmax attention over paged bf16 / fp32 keys and values ("tiles" pages, see the cache module): shared declarations.
//
// A head has one or two query / key maps of `dim` and one value of `vdim`; a map is a softmax attention of its own.
//   two maps (differential attention): the head's output is rms(a1 - lam * a2) * post over its vdim values;
//   one map: a * sigmoid(gate) * post, where the softmax may have a sink: one more term exp(sink) in the denominator, without a
//   key and a value; sink and gate are optional;
//   sigmoid (one map): a key's weight is sigmoid(score + bias), not its share of a sum; the bias is a number per head and distance.
// Query head h reads key/value head h / group.  A row sees the keys at most window - 1 positions before it (window 0: all).
// A page block (one page, one key/value head) is [K map 1 | (K map 2) | V] of 16 tokens each, as 8 x 8 core matrices:
// element (token t, column j) of a part with D padded columns sits at (t / 8) * 8 D + (j / 8) * 64 + (t % 8) * 8 + j % 8.
#pragma once
#include "blaze/attn.cuh"
#include "blaze/sm100.cuh"

namespace blz {

static constexpr int kBiasPad = 128;

struct MapsParams {
  const void* q;               // [T, ld]: q [heads][maps][dim] of every row
  const void* kv;              // page write: the same rows from their keys on, k [kv_heads][maps][dim] | v [kv_heads][vdim]
  void* out;                   // [T, ld_out], heads * vdim columns
  void* pool;                  // page blocks
  const float* sink;           // [heads] or null
  const void* gate;            // [T, ld_gate], heads * vdim columns, or null
  long long ld, ld_out, ld_gate, page_stride, head_stride;    // elements
  const int* block_table;
  const int* slots;            // [B]
  const int* q_start;          // [B + 1]
  const int* ctx_len;          // [B]
  const int* seq_of_row;       // [T], -1 = padding
  const int* slot_mapping;     // [T], -1 = padding
  float* part_o;               // partial outputs of split key ranges
  float* part_ml;
  int bt_stride, T, B, heads, kv_heads, dim, vdim, window, maps;
  float scale, lam, post, eps;
  int max_rows;                // rows (new tokens * group) up to which a sequence belongs to the short-row kernel
  int row_blocks, splits, stages;
  int* status;
  const int* page_base;        // [B] or null: the pages of sequence b are page_base[b] + page index, not block_table's
  const float* bias;           // sigmoid: [heads][bias_len()], entry kBiasPad + distance, see bias_len
  int reach;                   // sigmoid: distances listed one by one; keys farther away have the last one's bias
  int shared_kv;               // one map: a block is its key part alone, whose first vdim columns are the values

  __host__ __device__ int group() const { return heads / kv_heads; }
  __host__ __device__ int dp() const { return (dim + 15) / 16 * 16; }
  __host__ __device__ int vp() const { return (vdim + 15) / 16 * 16; }
  // a row's entries around its own position can be read for a whole tile: those of keys that come later are -inf, those beyond
  // the last listed distance equal it.  The tensor-core kernels take the table times -log2(e).
  __host__ __device__ int bias_len() const { return reach + 2 * kBiasPad; }
  __host__ __device__ int block_elems() const { return 16 * (maps * dp() + vp()); }
};

// offset of (token, column) in a part with D padded columns
__host__ __device__ __forceinline__ int core_off(int t, int j, int D) { return (t >> 3) * 8 * D + (j >> 3) * 64 + (t & 7) * 8 + (j & 7); }

// first visible key position of a row at position `pos`
__device__ __forceinline__ int first_key(int pos, int window) { return window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0; }

static constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ad_ld(const float* p) { return *p; }
__device__ __forceinline__ float ad_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ad_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void ad_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// R rows (a multiple of 8) of dim columns -> shared memory as core matrices with D padded columns, by n threads with asynchronous copies of
// 16 bytes, all under way together; src(r): the row in memory, 16-byte aligned, or null (zeros).  dim % 8 == 0.  A warp reads 32 bytes of
// a row at a time and writes whole core matrices.  The caller waits (copies_wait) and fences.
template <typename F>
__device__ __forceinline__ void copy_rows(__nv_bfloat16* dst, int R, int D, int dim, int tid, int n, const void* any, F&& src) {
  for (int i = tid; i < R * (D / 8); i += n) {
    const int rest = i >> 4, r = (rest % (R / 8)) * 8 + (i & 7), j = ((rest / (R / 8)) * 2 + (i >> 3 & 1)) * 8;
    const __nv_bfloat16* row = src(r);
    const bool live = row != nullptr && j < dim;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + core_off(r, j, D))),
                 "l"(live ? (const void*)(row + j) : any), "r"(live ? 16 : 0) : "memory");
  }
}
__device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// 1 / (1 + 2^t): the sigmoid of a score s for t = -s log2(e)
__device__ __forceinline__ float sigmoid_ex2(float t) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + ex2(t)));
  return r;
}

// factor of output column e of (row t, head h): sigmoid(gate) * post
template <typename T>
__device__ __forceinline__ float gate_factor(const MapsParams& p, int t, int h, int e) {
  if (!p.gate) return p.post;
  const float g = ad_ld(reinterpret_cast<const T*>(p.gate) + (size_t)t * p.ld_gate + (size_t)h * p.vdim + e);
  return p.post / (1.f + (sizeof(T) == 4 ? expf(-g) : __expf(-g)));
}

}  // namespace blz
