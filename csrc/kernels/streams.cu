// Residual streams with learned static mixes (hyper-connections whose weights do not depend on the input):
//   a sublayer reads u = sum_s in[s] x_s; afterwards, all streams at once from the old ones,
//   x_t <- sum_s mix[s, t] x_s + out[t] * y.
//
// One kernel does everything between two sublayers: it takes the sublayer's output y, rewrites the streams in place, forms
// the next sublayer's input from the new streams and RMS-normalises it, so that the fp32 streams make one trip through HBM
// per sublayer.  Before the first sublayer all streams equal the scaled embedding row, which is read from the table
// (`from_embed`) instead of being copied S times; after the last one only the sum of the streams is written.
// Beside them: the norm of fp32 rows, and the residual sum of a post-norm decoder (residual_norm_kernel).
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

// RMS norm of fp32 rows (the rows named by `rows`, or all) to the activation type.
template <typename T, int VEC>
__global__ void __launch_bounds__(512) norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ rows,
                                                        const float* __restrict__ w, T* __restrict__ out, int W, float eps) {
  __shared__ float red[16];
  pdl_trigger();
  pdl_wait();
  const float* xr = x + (size_t)(rows ? rows[blockIdx.x] : blockIdx.x) * W;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC];
    ld_vec<VEC>(xr + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
  }
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
  T* o = out + (size_t)blockIdx.x * W;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC], g[VEC];
    ld_vec<VEC>(xr + c, v);
    ld_vec<VEC>(w + c, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = v[j] * rs * g[j];
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

BLZ_API int blz_norm_rows(const float* x, const int* rows, const float* w, void* out, int R, int W, float eps, int f32, cudaStream_t s) {
  using namespace blz;
  if (R <= 0 || W < 1) return (int)cudaErrorInvalidValue;
  const bool v4 = W % 4 == 0;
  const dim3 g(R), b(row_threads(W, v4 ? 4 : 1));
  if (f32) return (int)(v4 ? launch_pdl(norm_rows_kernel<float, 4>, g, b, 0, s, x, rows, w, (float*)out, W, eps)
                           : launch_pdl(norm_rows_kernel<float, 1>, g, b, 0, s, x, rows, w, (float*)out, W, eps));
  return (int)(v4 ? launch_pdl(norm_rows_kernel<__nv_bfloat16, 4>, g, b, 0, s, x, rows, w, (__nv_bfloat16*)out, W, eps)
                  : launch_pdl(norm_rows_kernel<__nv_bfloat16, 1>, g, b, 0, s, x, rows, w, (__nv_bfloat16*)out, W, eps));
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
