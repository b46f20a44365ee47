// Residual streams with learned static mixes (hyper-connections whose weights do not depend on the input):
//   a sublayer reads u = sum_s in[s] x_s; afterwards, all streams at once from the old ones,
//   x_t <- sum_s mix[s, t] x_s + out[t] * y.
//
// One kernel does everything between two sublayers: it takes the sublayer's output y, rewrites the streams in place, forms
// the next sublayer's input from the new streams and RMS-normalises it, so that the fp32 streams make one trip through HBM
// per sublayer.  Before the first sublayer all streams equal the scaled embedding row, which is read from the table
// (`from_embed`) instead of being copied S times; after the last one only the sum of the streams is written.
// Beside them: the norm of fp32 rows, the residual sum of a post-norm decoder (residual_norm_kernel), the residual that takes
// normed branches (branch_norm_kernel), the residual that takes a mixer and a feed-forward side by side (branch_step_kernel), embedding
// rows with position vectors (embed_positions_kernel), and the causal convolution of a residual over time (input_conv_kernel).
// One CTA per row; the row's columns stay with their thread (float4 where the width allows), so the update is in place.
#include "blaze/host.h"
#include "blaze/sm100.cuh"

namespace blz {

struct StreamsParams {
  float* streams;              // [T, S, W]; read unless from_embed, written when write_streams
  const void* table;           // [vocab, W] (activation type)
  const int* tokens;           // [T]
  const void* y;               // [T, W] (activation type) or null (nothing to add: before the first sublayer)
  const float* mix;            // [S, S] from, to
  const float* w_out;          // [S], the residual multiplier included
  const float* w_in;           // [S] of the next sublayer, or null (no next one)
  const float* norm_w;         // [W]
  void* h;                     // [T, W] (activation type): the next sublayer's normed input
  float* sum;                  // [T, W] or null: sum of the new streams
  float embed_scale, eps;
  int S, W, vocab, from_embed, write_streams;
};

__device__ __forceinline__ float ld_act(const float* p) { return *p; }
__device__ __forceinline__ float ld_act(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st_act(float* p, float v) { *p = v; }
__device__ __forceinline__ void st_act(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <int VEC>
__device__ __forceinline__ void ld_vec(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = *p;
  }
}
template <int VEC>
__device__ __forceinline__ void ld_vec(const __nv_bfloat16* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = __bfloat162float(e[i]);
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int VEC>
__device__ __forceinline__ void st_vec(float* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int VEC>
__device__ __forceinline__ void st_vec(__nv_bfloat16* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  else *p = __float2bfloat16(v[0]);
}

__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float r = 0.f;
  for (int i = 0; i < nw; ++i) r += red[i];
  return r;
}

template <typename T, int SMAX, int VEC>
__global__ void __launch_bounds__(512) streams_kernel(StreamsParams p) {
  extern __shared__ float u_row[];                   // [W]
  __shared__ float s_mix[SMAX * SMAX], s_out[SMAX], s_in[SMAX], red[16];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, S = p.S, W = p.W;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) s_mix[i] = p.mix ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    s_out[i] = p.w_out ? p.w_out[i] : 0.f;
    s_in[i] = p.w_in ? p.w_in[i] : 0.f;
  }
  __syncthreads();
  float wm[SMAX <= 4 ? SMAX * SMAX : 1], wo[SMAX], wi[SMAX];
  if constexpr (SMAX <= 4) {
#pragma unroll
    for (int a = 0; a < SMAX; ++a)
#pragma unroll
      for (int b = 0; b < SMAX; ++b) wm[a * SMAX + b] = (a < S && b < S) ? s_mix[a * S + b] : 0.f;
  }
#pragma unroll
  for (int a = 0; a < SMAX; ++a) { wo[a] = a < S ? s_out[a] : 0.f; wi[a] = a < S ? s_in[a] : 0.f; }
  const T* erow = nullptr;
  if (p.from_embed) {
    int tok = p.tokens[t];
    tok = tok < 0 ? 0 : (tok >= p.vocab ? p.vocab - 1 : tok);
    erow = reinterpret_cast<const T*>(p.table) + (size_t)tok * W;
  }
  float* xrow = p.streams + (size_t)t * S * W;
  const T* yrow = p.y ? reinterpret_cast<const T*>(p.y) + (size_t)t * W : nullptr;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float x[SMAX][VEC];
    if (p.from_embed) {
      float e[VEC];
      ld_vec<VEC>(erow + c, e);
#pragma unroll
      for (int s = 0; s < SMAX; ++s)
#pragma unroll
        for (int j = 0; j < VEC; ++j) x[s][j] = e[j] * p.embed_scale;
    } else {
#pragma unroll
      for (int s = 0; s < SMAX; ++s)
        if (s < S) ld_vec<VEC>(xrow + (size_t)s * W + c, x[s]);
    }
    float u[VEC], sum[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = sum[j] = 0.f;
    if (yrow) {
      float y[VEC];
      ld_vec<VEC>(yrow + c, y);
#pragma unroll
      for (int b = 0; b < SMAX; ++b) {
        if (b >= S) break;
        float n[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) n[j] = wo[b] * y[j];
#pragma unroll
        for (int a = 0; a < SMAX; ++a) {
          if (a >= S) break;
          float m;
          if constexpr (SMAX <= 4) m = wm[a * SMAX + b];
          else m = s_mix[a * S + b];
#pragma unroll
          for (int j = 0; j < VEC; ++j) n[j] = fmaf(m, x[a][j], n[j]);
        }
        if (p.write_streams) st_vec<VEC>(xrow + (size_t)b * W + c, n);
#pragma unroll
        for (int j = 0; j < VEC; ++j) { u[j] = fmaf(wi[b], n[j], u[j]); sum[j] += n[j]; }
      }
    } else {
#pragma unroll
      for (int b = 0; b < SMAX; ++b) {
        if (b >= S) break;
#pragma unroll
        for (int j = 0; j < VEC; ++j) { u[j] = fmaf(wi[b], x[b][j], u[j]); sum[j] += x[b][j]; }
      }
    }
    if (p.sum) st_vec<VEC>(p.sum + (size_t)t * W + c, sum);
    if (p.w_in) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(u[j], u[j], ss);
      st_vec<VEC>(u_row + c, u);
    }
  }
  if (!p.w_in) return;
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)W + p.eps);
  T* hrow = reinterpret_cast<T*>(p.h) + (size_t)t * W;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC], w[VEC];
    ld_vec<VEC>(u_row + c, u);
    ld_vec<VEC>(p.norm_w + c, w);
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = u[j] * rs * w[j];
    st_vec<VEC>(hrow + c, u);
  }
}

// RMS norm (centre: layer norm) of fp32 rows (the rows named by `rows`, or all) to the activation type.
template <typename T, int VEC>
__global__ void __launch_bounds__(512) norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ rows,
                                                        const float* __restrict__ w, T* __restrict__ out, int W, float eps, int centre) {
  __shared__ float red[16], red1[16];
  pdl_trigger();
  pdl_wait();
  const float* xr = x + (size_t)(rows ? rows[blockIdx.x] : blockIdx.x) * W;
  float ss = 0.f, mean = 0.f;
  if (centre) {
    for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
      float v[VEC];
      ld_vec<VEC>(xr + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) mean += v[j];
    }
    mean = block_sum(mean, red1) / (float)W;
  }
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC];
    ld_vec<VEC>(xr + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(v[j] - mean, v[j] - mean, ss);
  }
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
  T* o = out + (size_t)blockIdx.x * W;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC], g[VEC];
    ld_vec<VEC>(xr + c, v);
    ld_vec<VEC>(w + c, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = (v[j] - mean) * rs * g[j];
    st_vec<VEC>(o + c, v);
  }
}

// The residual of a post-norm decoder: x <- norm(alpha * x + y), kept in fp32, with a copy in the activation type for the next
// sublayer.  `from` holds the old x: fp32 rows (may be x itself), or rows of the activation type.
template <typename T, typename X, int VEC>
__global__ void __launch_bounds__(512) residual_norm_kernel(const X* __restrict__ from, float alpha, const T* __restrict__ y,
                                                            const float* __restrict__ w, float eps, float* x, T* h, int W) {
  extern __shared__ float u_row[];                   // [W]
  __shared__ float red[16];
  pdl_trigger();
  pdl_wait();
  const size_t at = (size_t)blockIdx.x * W;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC], v[VEC];
    ld_vec<VEC>(from + at + c, u);
    ld_vec<VEC>(y + at + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      u[j] = fmaf(alpha, u[j], v[j]);
      ss = fmaf(u[j], u[j], ss);
    }
    st_vec<VEC>(u_row + c, u);
  }
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC], g[VEC];
    ld_vec<VEC>(u_row + c, u);
    ld_vec<VEC>(w + c, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = u[j] * rs * g[j];
    st_vec<VEC>(x + at + c, u);
    if (h) st_vec<VEC>(h + at + c, u);
  }
}

// A branch into an fp32 residual: x <- x + layer_norm(branch) * w, with a copy in the activation type (h, may be null).  The branch is
// a row of y; or (ROUTED) the weighted sum of the k rows of y that row_map names (-1: none) plus, if there is one, a row of `extra`;
// or (EMBED) the token's row of a table, and x is then the normed row alone.
enum BranchSrc { ROWS, ROUTED, EMBED };
struct BranchParams {
  const void* y;               // [.., ldy] activation type
  const void* extra;           // [T, W]
  const float* weights;        // [T, k]
  const int* row_map;          // [T, k], or (EMBED) tokens [T]
  const float* w;              // [W]
  float* x;                    // [T, W]
  void* h;
  long long ldy;
  int k, W, vocab;
  float eps;
};

template <typename T, int VEC, BranchSrc SRC>
__global__ void __launch_bounds__(512) branch_norm_kernel(BranchParams p) {
  extern __shared__ float u_row[];                   // [W]
  __shared__ float red0[16], red1[16], s_w[32];
  __shared__ int s_row[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, W = p.W;
  const size_t at = (size_t)t * W;
  const T* y = reinterpret_cast<const T*>(p.y);
  if constexpr (SRC == ROUTED) {
    if (threadIdx.x < p.k) {
      s_w[threadIdx.x] = p.weights[(size_t)t * p.k + threadIdx.x];
      s_row[threadIdx.x] = p.row_map[(size_t)t * p.k + threadIdx.x];
    }
    __syncthreads();
  } else if constexpr (SRC == EMBED) {
    const int tok = p.row_map[t];
    y += (size_t)(tok < 0 ? 0 : tok >= p.vocab ? p.vocab - 1 : tok) * p.ldy;
  } else {
    y += (size_t)t * p.ldy;
  }
  float sum = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC];
    if constexpr (SRC == ROUTED) {
      if (p.extra) {
        ld_vec<VEC>(reinterpret_cast<const T*>(p.extra) + at + c, u);
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = 0.f;
      }
      for (int i = 0; i < p.k; ++i) {
        if (s_row[i] < 0) continue;
        float v[VEC];
        ld_vec<VEC>(y + (size_t)s_row[i] * p.ldy + c, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = fmaf(s_w[i], v[j], u[j]);
      }
    } else {
      ld_vec<VEC>(y + c, u);
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) sum += u[j];
    st_vec<VEC>(u_row + c, u);
  }
  const float mean = block_sum(sum, red0) / (float)W;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC];
    ld_vec<VEC>(u_row + c, u);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(u[j] - mean, u[j] - mean, ss);
  }
  const float rs = 1.f / sqrtf(block_sum(ss, red1) / (float)W + p.eps);
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC], g[VEC], x[VEC];
    ld_vec<VEC>(u_row + c, u);
    ld_vec<VEC>(p.w + c, g);
    if constexpr (SRC != EMBED) ld_vec<VEC>(p.x + at + c, x);
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = SRC == EMBED ? (u[j] - mean) * rs * g[j] : fmaf((u[j] - mean) * rs, g[j], x[j]);
    st_vec<VEC>(p.x + at + c, u);
    if (p.h) st_vec<VEC>(reinterpret_cast<T*>(p.h) + at + c, u);
  }
}

// sums of two numbers over the block
__device__ __forceinline__ float2 block_sum2(float2 v, float2* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float2 r = make_float2(0.f, 0.f);
  for (int i = 0; i < nw; ++i) { r.x += red[i].x; r.y += red[i].y; }
  return r;
}

// What stands between two layers whose mixer and feed-forward read the same residual:
//   x <- x + mult * (mixer + ffn), in fp32; then up to two RMS norms of it, for the next mixer and feed-forward, and a copy (activation type).
// mixer: a row of y1, or (m1) the mean of the rows of y1 and y2, each RMS-normed with a weight; or nothing (y1 null: x stays as it is).
// ffn: the sum of the k rows of routed that row_map names (-1: none), times weights where there are any, and of a row of extra times
// sigmoid(gate) where there is a gate.
struct BranchStepParams {
  float* x;                    // [T, W]
  const void *y1, *y2;         // [T, W] activation type
  const float *m1, *m2;        // [W]
  const void* routed;          // [.., ld_routed]
  const float* weights;        // [T, k] or null
  const int* row_map;          // [T, k]
  const void* extra;           // [T, W] or null
  const float* gate;           // gate[t * ld_gate], or null
  const float *w1, *w2;        // [W] or null
  void *h1, *h2, *copy;        // [T, W], [T, W], [T, ld_copy] activation type, or null
  long long ld_routed, ld_gate, ld_copy;
  int k, W;
  float mult, eps;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(512) branch_step_kernel(BranchStepParams p) {
  extern __shared__ float u_row[];                   // [W]
  __shared__ float2 red0[16];
  __shared__ float red1[16], s_w[32];
  __shared__ int s_row[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, W = p.W;
  const size_t at = (size_t)t * W;
  const T *y1 = reinterpret_cast<const T*>(p.y1) + at, *y2 = reinterpret_cast<const T*>(p.y2) + at;
  const T *routed = reinterpret_cast<const T*>(p.routed), *extra = reinterpret_cast<const T*>(p.extra);
  const bool add = p.y1 != nullptr, normed = p.m1 != nullptr;
  float f1 = 1.f, f2 = 0.f, sg = 1.f;
  if (add) {
    if (threadIdx.x < p.k) {
      s_w[threadIdx.x] = p.weights ? p.weights[(size_t)t * p.k + threadIdx.x] : 1.f;
      s_row[threadIdx.x] = p.row_map[(size_t)t * p.k + threadIdx.x];
    }
    if (p.gate) sg = 1.f / (1.f + expf(-p.gate[(size_t)t * p.ld_gate]));
    float2 ss = make_float2(0.f, 0.f);
    if (normed) {
      for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
        float a[VEC], b[VEC];
        ld_vec<VEC>(y1 + c, a);
        ld_vec<VEC>(y2 + c, b);
#pragma unroll
        for (int j = 0; j < VEC; ++j) { ss.x = fmaf(a[j], a[j], ss.x); ss.y = fmaf(b[j], b[j], ss.y); }
      }
    }
    ss = block_sum2(ss, red0);                       // also makes s_w and s_row visible
    if (normed) {
      f1 = 0.5f / sqrtf(ss.x / (float)W + p.eps);
      f2 = 0.5f / sqrtf(ss.y / (float)W + p.eps);
    }
  }
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float x[VEC];
    ld_vec<VEC>(p.x + at + c, x);
    if (add) {
      float u[VEC], v[VEC];
      ld_vec<VEC>(y1 + c, u);
      if (normed) {
        float g[VEC], w[VEC];
        ld_vec<VEC>(y2 + c, v);
        ld_vec<VEC>(p.m1 + c, g);
        ld_vec<VEC>(p.m2 + c, w);
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = fmaf(u[j] * f1, g[j], v[j] * f2 * w[j]);
      }
      if (extra) {
        ld_vec<VEC>(extra + at + c, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = fmaf(sg, v[j], u[j]);
      }
      for (int i = 0; i < p.k; ++i) {
        if (s_row[i] < 0) continue;
        ld_vec<VEC>(routed + (size_t)s_row[i] * p.ld_routed + c, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = fmaf(s_w[i], v[j], u[j]);
      }
#pragma unroll
      for (int j = 0; j < VEC; ++j) x[j] = fmaf(p.mult, u[j], x[j]);
      st_vec<VEC>(p.x + at + c, x);
    }
    if (p.copy) st_vec<VEC>(reinterpret_cast<T*>(p.copy) + (size_t)t * p.ld_copy + c, x);
    if (p.w1 || p.w2) {
      st_vec<VEC>(u_row + c, x);
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(x[j], x[j], ss);
    }
  }
  if (!p.w1 && !p.w2) return;
  const float rs = 1.f / sqrtf(block_sum(ss, red1) / (float)W + p.eps);
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC], w[VEC], h[VEC];
    ld_vec<VEC>(u_row + c, u);
    if (p.w1) {
      ld_vec<VEC>(p.w1 + c, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) h[j] = u[j] * rs * w[j];
      st_vec<VEC>(reinterpret_cast<T*>(p.h1) + at + c, h);
    }
    if (p.w2) {
      ld_vec<VEC>(p.w2 + c, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) h[j] = u[j] * rs * w[j];
      st_vec<VEC>(reinterpret_cast<T*>(p.h2) + at + c, h);
    }
  }
}

// x = scale * table[token] + position vector: sine (even columns) and cosine (odd ones) of position * freq[column / 2], with freq given as
// two floats so that far positions keep their angle; copy (activation type, or null) gets the row too.
template <typename T>
__global__ void __launch_bounds__(256) embed_positions_kernel(const T* __restrict__ table, const int* __restrict__ tokens,
                                                              const int* __restrict__ positions, const float* __restrict__ freq, int vocab,
                                                              float scale, float* __restrict__ x, T* __restrict__ copy, long long ld_copy, int W) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, half = (W + 1) / 2;
  int tok = tokens[t];
  tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
  const T* row = table + (size_t)tok * W;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float hi = freq[i], ang = pos * hi, rest = fmaf(pos, hi, -ang) + pos * freq[half + i];
    float s, c;
    sincosf(ang, &s, &c);
    const float half_sq = 0.5f * rest * rest;        // the rest grows to hundredths of a radian at the farthest positions
    const float v[2] = {fmaf(rest, c, fmaf(-half_sq, s, s)), fmaf(-rest, s, fmaf(-half_sq, c, c))};
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int col = 2 * i + j;
      if (col >= W) break;
      const float y = fmaf(scale, ld_act(row + col), v[j]);
      x[(size_t)t * W + col] = y;
      if (copy) st_act(copy + (size_t)t * ld_copy + col, y);
    }
  }
}

// h = x + conv(x): a causal convolution of every column over a sequence's rows, whose earlier inputs are in the sequence's state row.
// A thread takes VEC columns of up to kConvSeg rows of one sequence; a longer run's state is written by a kernel of its own (its first
// segment reads the old one).  TAPS = 0: any number, read again for every row.
static constexpr int kConvSeg = 32;
struct InputConvParams {
  const float* x;              // [T, W]
  void* h;                     // [T, W] activation type, or null (the state only)
  float* state;                // [rows, taps - 1, W]
  const float* w;              // [taps, W]
  const int *slots, *q_start, *ctx_len, *no_store;
  int W, taps;
};

template <typename T, int TAPS, int VEC>
__global__ void __launch_bounds__(128) input_conv_kernel(InputConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC, b = blockIdx.y, W = p.W, taps = TAPS ? TAPS : p.taps;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, t0 = blockIdx.z * kConvSeg, t1 = min(n, t0 + kConvSeg);
  if (c >= W || t0 >= n) return;
  const bool fresh = p.ctx_len[b] == n;
  float* st = p.state + (size_t)p.slots[b] * (taps - 1) * W + c;
  const float* x = p.x + (size_t)r0 * W + c;
  auto input = [&](int t, float (&v)[VEC]) {         // input of position t of this run (negative: before it)
    if (t >= 0) {
      ld_vec<VEC>(x + (size_t)t * W, v);
    } else if (!fresh) {
      ld_vec<VEC>(st + (size_t)(taps - 1 + t) * W, v);
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = 0.f;
    }
  };
  T* h = reinterpret_cast<T*>(p.h) + (size_t)r0 * W + c;
  if constexpr (TAPS == 0) {
    for (int t = t0; t < t1 && p.h; ++t) {
      float y[VEC], v[VEC], g[VEC];
      input(t, y);
      for (int i = 0; i < taps; ++i) {
        input(t - taps + 1 + i, v);
        ld_vec<VEC>(p.w + (size_t)i * W + c, g);
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] = fmaf(g[j], v[j], y[j]);
      }
      st_vec<VEC>(h + (size_t)t * W, y);
    }
  } else {
    float v[TAPS][VEC], g[TAPS][VEC];
#pragma unroll
    for (int i = 0; i < TAPS; ++i) ld_vec<VEC>(p.w + (size_t)i * W + c, g[i]);
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) input(t0 - TAPS + 1 + i, v[i]);
    constexpr int AHEAD = 4;                         // rows in flight
    for (int t = t0; t < t1; t += AHEAD) {
      float in[AHEAD][VEC];
#pragma unroll
      for (int k = 0; k < AHEAD; ++k)
        if (t + k < t1) ld_vec<VEC>(x + (size_t)(t + k) * W, in[k]);
#pragma unroll
      for (int k = 0; k < AHEAD; ++k) {
        if (t + k >= t1) break;
        float y[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          v[TAPS - 1][j] = y[j] = in[k][j];
#pragma unroll
          for (int i = 0; i < TAPS; ++i) y[j] = fmaf(g[i][j], v[i][j], y[j]);
#pragma unroll
          for (int i = 0; i < TAPS - 1; ++i) v[i][j] = v[i + 1][j];
        }
        if (p.h) st_vec<VEC>(h + (size_t)(t + k) * W, y);
      }
    }
    if (n > kConvSeg || (p.no_store != nullptr && p.no_store[b])) return;
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) st_vec<VEC>(st + (size_t)i * W, v[i]);
  }
}

// the state after a run of more than min_rows rows
template <int VEC>
__global__ void __launch_bounds__(128) input_conv_state_kernel(InputConvParams p, int min_rows) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC, b = blockIdx.y, W = p.W;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0;
  if (c >= W || n <= min_rows || (p.no_store != nullptr && p.no_store[b])) return;
  const bool fresh = p.ctx_len[b] == n;
  float* st = p.state + (size_t)p.slots[b] * (p.taps - 1) * W + c;
  for (int i = 0; i < p.taps - 1; ++i) {             // entry i: input n - (taps - 1) + i, an older entry where the run is shorter
    const int t = n - p.taps + 1 + i;
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = 0.f;
    if (t >= 0) ld_vec<VEC>(p.x + (size_t)(r0 + t) * W + c, v);
    else if (!fresh) ld_vec<VEC>(st + (size_t)(i + n) * W, v);
    st_vec<VEC>(st + (size_t)i * W, v);
  }
}

template <typename T, int VEC>
static int launch_input_conv(const InputConvParams& p, int B, int max_q, cudaStream_t s) {
  const dim3 grid((p.W + 128 * VEC - 1) / (128 * VEC), B, (max_q + kConvSeg - 1) / kConvSeg);
  cudaError_t e;
  switch (p.taps) {
#define BLZ_IC(K) case K: e = launch_pdl(input_conv_kernel<T, K, VEC>, grid, dim3(128), 0, s, p); break
    BLZ_IC(1); BLZ_IC(2); BLZ_IC(3); BLZ_IC(4); BLZ_IC(5); BLZ_IC(6); BLZ_IC(7); BLZ_IC(8);
    default: e = launch_pdl(input_conv_kernel<T, 0, VEC>, grid, dim3(128), 0, s, p);
#undef BLZ_IC
  }
  if (e != cudaSuccess) return (int)e;
  const int min_rows = p.taps > 8 ? 0 : kConvSeg;
  if (p.taps > 1 && max_q > min_rows) input_conv_state_kernel<VEC><<<dim3(grid.x, B), 128, 0, s>>>(p, min_rows);
  return (int)cudaGetLastError();
}

static int row_threads(int W, int vec);
template <BranchSrc SRC>
static int launch_branch(const BranchParams& p, int T, int f32, int vec, cudaStream_t s) {
  const dim3 block(row_threads(p.W, vec ? 4 : 1));
  const size_t sm = (size_t)p.W * 4;
#define BLZ_BN(TT, V)                                                                   \
  do {                                                                                  \
    static PerDeviceOnce once;                                                          \
    const cudaError_t e = once.smem_limit(branch_norm_kernel<TT, V, SRC>, 200 * 1024);  \
    if (e != cudaSuccess) return (int)e;                                                \
    return (int)launch_pdl(branch_norm_kernel<TT, V, SRC>, dim3(T), block, sm, s, p);   \
  } while (0)
  if (f32) { if (vec) BLZ_BN(float, 4); BLZ_BN(float, 1); }
  if (vec) BLZ_BN(__nv_bfloat16, 4);
  BLZ_BN(__nv_bfloat16, 1);
#undef BLZ_BN
}

static int row_threads(int W, int vec) {
  int n = (W / vec + 1) / 2;
  n = (n + 31) / 32 * 32;
  return n < 64 ? 64 : (n > 512 ? 512 : n);
}

template <typename T, int SMAX, int VEC>
static cudaError_t launch_streams(const StreamsParams& p, int rows, cudaStream_t s) {
  auto kern = streams_kernel<T, SMAX, VEC>;
  static PerDeviceOnce once;
  cudaError_t e = once.smem_limit(kern, 200 * 1024);
  if (e != cudaSuccess) return e;
  return launch_pdl(kern, dim3(rows), dim3(row_threads(p.W, VEC)), (size_t)p.W * 4, s, p);
}

template <typename T>
static cudaError_t pick_streams(const StreamsParams& p, int rows, cudaStream_t s) {
  const bool v4 = p.W % 4 == 0;
#define BLZ_STREAMS(N) return v4 ? launch_streams<T, N, 4>(p, rows, s) : launch_streams<T, N, 1>(p, rows, s)
  if (p.S <= 1) { BLZ_STREAMS(1); }
  if (p.S == 2) { BLZ_STREAMS(2); }
  if (p.S <= 4) { BLZ_STREAMS(4); }
  if (p.S <= 8) { BLZ_STREAMS(8); }
  BLZ_STREAMS(16);
#undef BLZ_STREAMS
}

template <typename T, typename X, int VEC>
static cudaError_t launch_residual(const void* from, float alpha, const void* y, const float* w, float eps, float* x, void* h, int rows,
                                   int W, cudaStream_t s) {
  auto kern = residual_norm_kernel<T, X, VEC>;
  static PerDeviceOnce once;
  cudaError_t e = once.smem_limit(kern, 200 * 1024);
  if (e != cudaSuccess) return e;
  return launch_pdl(kern, dim3(rows), dim3(row_threads(W, VEC)), (size_t)W * 4, s, (const X*)from, alpha, (const T*)y, w, eps, x, (T*)h, W);
}

}  // namespace blz

// See StreamsParams; f32 = 1: activations (table, y, h) are fp32, else bf16.  1 <= S <= 16, W <= 51200.
BLZ_API int blz_streams(float* streams, const void* table, const int* tokens, int vocab, float embed_scale, const void* y,
                        const float* mix, const float* w_out, const float* w_in, const float* norm_w, float eps, void* h, float* sum,
                        int T, int S, int W, int from_embed, int write_streams, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || S < 1 || S > 16 || W < 1 || W > 51200) return (int)cudaErrorInvalidValue;
  if (from_embed && (!table || !tokens)) return (int)cudaErrorInvalidValue;
  if ((!from_embed || write_streams) && !streams) return (int)cudaErrorInvalidValue;
  if (y && (!mix || !w_out)) return (int)cudaErrorInvalidValue;
  if (w_in && (!norm_w || !h)) return (int)cudaErrorInvalidValue;
  StreamsParams p;
  p.streams = streams; p.table = table; p.tokens = tokens; p.y = y; p.mix = mix; p.w_out = w_out; p.w_in = w_in; p.norm_w = norm_w;
  p.h = h; p.sum = sum; p.embed_scale = embed_scale; p.eps = eps; p.S = S; p.W = W; p.vocab = vocab; p.from_embed = from_embed;
  p.write_streams = write_streams;
  return (int)(f32 ? pick_streams<float>(p, T, s) : pick_streams<__nv_bfloat16>(p, T, s));
}

BLZ_API int blz_norm_rows(const float* x, const int* rows, const float* w, void* out, int R, int W, float eps, int centre, int f32,
                          cudaStream_t s) {
  using namespace blz;
  if (R <= 0 || W < 1) return (int)cudaErrorInvalidValue;
  const bool v4 = W % 4 == 0;
  const dim3 g(R), b(row_threads(W, v4 ? 4 : 1));
  if (f32) return (int)(v4 ? launch_pdl(norm_rows_kernel<float, 4>, g, b, 0, s, x, rows, w, (float*)out, W, eps, centre)
                           : launch_pdl(norm_rows_kernel<float, 1>, g, b, 0, s, x, rows, w, (float*)out, W, eps, centre));
  return (int)(v4 ? launch_pdl(norm_rows_kernel<__nv_bfloat16, 4>, g, b, 0, s, x, rows, w, (__nv_bfloat16*)out, W, eps, centre)
                  : launch_pdl(norm_rows_kernel<__nv_bfloat16, 1>, g, b, 0, s, x, rows, w, (__nv_bfloat16*)out, W, eps, centre));
}

// x [T, W] fp32 <- norm(alpha * from + y) with the norm's weight w; h [T, W] (activation type, or null) gets a copy.  from_act: `from`
// is of the activation type (else fp32; x itself may stand there).  f32 = 1: the activation type is fp32.  W <= 51200.
BLZ_API int blz_residual_norm(const void* from, int from_act, float alpha, const void* y, const float* w, float eps, float* x, void* h,
                              int T, int W, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || W < 1 || W > 51200 || !from || !y || !w || !x) return (int)cudaErrorInvalidValue;
  const bool v4 = W % 4 == 0;
#define BLZ_RN(TT, XX) return (int)(v4 ? launch_residual<TT, XX, 4>(from, alpha, y, w, eps, x, h, T, W, s) \
                                       : launch_residual<TT, XX, 1>(from, alpha, y, w, eps, x, h, T, W, s))
  if (f32) { BLZ_RN(float, float); }
  if (from_act) { BLZ_RN(__nv_bfloat16, __nv_bfloat16); }
  BLZ_RN(__nv_bfloat16, float);
#undef BLZ_RN
}

// x [T, W] fp32 <- x + layer_norm(branch) * w, h (activation type, or null) a copy; the branch: rows of y [T, ldy], or (row_map) the sums
// of weights[t, i] * y[row_map[t, i]], i < k <= 32, and of extra [T, W] (or null).  W <= 51200.
BLZ_API int blz_branch_norm(const void* y, long long ldy, const float* weights, const int* row_map, int k, const void* extra, const float* w,
                            float eps, float* x, void* h, int T, int W, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || W < 1 || W > 51200 || !y || !w || !x || (row_map && (!weights || k < 1 || k > 32))) return (int)cudaErrorInvalidValue;
  BranchParams p = {y, extra, weights, row_map, w, x, h, ldy, k, W, 0, eps};
  const int vec = W % 4 == 0 && ldy % 4 == 0;
  return row_map ? launch_branch<ROUTED>(p, T, f32, vec, s) : launch_branch<ROWS>(p, T, f32, vec, s);
}

// x [T, W] fp32 = layer_norm(table[token]) * w.
BLZ_API int blz_embed_norm(const void* table, const int* tokens, int vocab, const float* w, float eps, float* x, int T, int W, int f32,
                           cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || W < 1 || W > 51200 || vocab < 1 || !table || !tokens || !w || !x) return (int)cudaErrorInvalidValue;
  const BranchParams p = {table, nullptr, nullptr, tokens, w, x, nullptr, W, 0, W, vocab, eps};
  return launch_branch<EMBED>(p, T, f32, W % 4 == 0, s);
}

// See BranchStepParams; f32 = 1: the activation type is fp32.  k <= 32, W <= 51200.
BLZ_API int blz_branch_step(float* x, const void* y1, const void* y2, const float* m1, const float* m2, const void* routed, long long ld_routed,
                            const float* weights, const int* row_map, int k, const void* extra, const float* gate, long long ld_gate,
                            const float* w1, const float* w2, void* h1, void* h2, void* copy, long long ld_copy, float mult, float eps, int T,
                            int W, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || W < 1 || W > 51200 || !x || k < 0 || k > 32 || (k && (!routed || !row_map)) || (m1 && (!m2 || !y1 || !y2)) ||
      (w1 && !h1) || (w2 && !h2))
    return (int)cudaErrorInvalidValue;
  const BranchStepParams p = {x, y1, y2, m1, m2, routed, weights, row_map, extra, gate, w1, w2, h1, h2, copy, ld_routed, ld_gate, ld_copy,
                              k, W, mult, eps};
  const bool vec = W % 4 == 0 && ld_routed % 4 == 0 && ld_copy % 4 == 0;
  const dim3 block(row_threads(W, vec ? 4 : 1));
#define BLZ_BS(TT, V)                                                                                \
  do {                                                                                               \
    static PerDeviceOnce once;                                                                       \
    const cudaError_t e = once.smem_limit(branch_step_kernel<TT, V>, 200 * 1024);                    \
    if (e != cudaSuccess) return (int)e;                                                             \
    return (int)launch_pdl(branch_step_kernel<TT, V>, dim3(T), block, (size_t)W * 4, s, p);          \
  } while (0)
  if (f32) { if (vec) BLZ_BS(float, 4); BLZ_BS(float, 1); }
  if (vec) BLZ_BS(__nv_bfloat16, 4);
  BLZ_BS(__nv_bfloat16, 1);
#undef BLZ_BS
}

// x [T, W] fp32 = scale * table[token] + sines and cosines (embed_positions_kernel); freq [2][(W + 1) / 2].
BLZ_API int blz_embed_positions(const void* table, const int* tokens, const int* positions, const float* freq, int vocab, float scale, float* x,
                                void* copy, long long ld_copy, int T, int W, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || W < 1 || vocab < 1 || !table || !tokens || !positions || !freq || !x) return (int)cudaErrorInvalidValue;
  if (f32)
    return (int)launch_pdl(embed_positions_kernel<float>, dim3(T), dim3(256), 0, s, (const float*)table, tokens, positions, freq, vocab, scale, x,
                           (float*)copy, ld_copy, W);
  return (int)launch_pdl(embed_positions_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, (const __nv_bfloat16*)table, tokens, positions, freq,
                         vocab, scale, x, (__nv_bfloat16*)copy, ld_copy, W);
}

// See InputConvParams; max_q: the longest run of the batch.  no_store: optional [B], 1 = leave the sequence's state as it was.
BLZ_API int blz_input_conv(const float* x, void* h, float* state, const float* w, const int* slots, const int* q_start, const int* ctx_len,
                           const int* no_store, int B, int W, int taps, int max_q, int f32, cudaStream_t s) {
  using namespace blz;
  if (B < 1 || B > 65535 || W < 1 || taps < 1 || max_q < 1 || !x || !w || (taps > 1 && !state)) return (int)cudaErrorInvalidValue;
  const InputConvParams p = {x, h, state, w, slots, q_start, ctx_len, no_store, W, taps};
  if (f32) return W % 4 == 0 ? launch_input_conv<float, 4>(p, B, max_q, s) : launch_input_conv<float, 1>(p, B, max_q, s);
  return W % 4 == 0 ? launch_input_conv<__nv_bfloat16, 4>(p, B, max_q, s) : launch_input_conv<__nv_bfloat16, 1>(p, B, max_q, s);
}
