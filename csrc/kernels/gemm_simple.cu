// Matrix products on the CUDA cores: C[M,N] = A[M,K] B[N,K]^T (+ bias) for fp32 operands (a model served in true 32-bit; the
// tensor cores have no such mode) and for bf16 shapes that the TMA kernels do not take (a row length that is not a multiple
// of 16).  fp32 accumulation, no reduced-precision mode.  Also the expert product over rows sorted by expert, and activations as ops
// of their own: the gated ones, the squared ReLU and the sum of normed powers.
#include "blaze/glu.cuh"
#include "blaze/host.h"
#include "blaze/sm100.cuh"

namespace blz {

__device__ __forceinline__ float gs_ld(const float* p) { return *p; }
__device__ __forceinline__ float gs_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void gs_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void gs_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// 64 x 64 output tile per 256-thread CTA, 16-deep K steps, 4 x 4 outputs per thread
// tile_expert (or null): expert of each 128 rows of A (-1: none), whose weight is B + expert * N * ldb, and its live rows
template <typename T, typename O>
__global__ void __launch_bounds__(256) gemm_simple_kernel(const T* __restrict__ A, long long lda, const T* __restrict__ B,
                                                          long long ldb, O* __restrict__ C, long long ldc,
                                                          const float* __restrict__ bias, int M, int N, int K,
                                                          const int* __restrict__ tile_expert, const int* __restrict__ tile_rows) {
  __shared__ float sa[16][68], sb[16][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  if (tile_expert) {
    const int e = tile_expert[m0 >> 7];
    if (e < 0) return;
    B += (size_t)e * N * ldb;
    M = (m0 & ~127) + tile_rows[m0 >> 7];
    if (m0 >= M) return;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = threadIdx.x + i * 256, r = e >> 4, k = e & 15;
      sa[k][r] = (m0 + r < M && k0 + k < K) ? gs_ld(A + (size_t)(m0 + r) * lda + k0 + k) : 0.f;
      sb[k][r] = (n0 + r < N && k0 + k < K) ? gs_ld(B + (size_t)(n0 + r) * ldb + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sa[k][ty * 4 + i]; b[i] = sb[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) gs_st(C + (size_t)m * ldc + n, acc[i][j] + (bias ? bias[n] : 0.f));
    }
  }
}

// gu [T, 2I] = [gate | up] -> out [T, I]; limit < 0: silu(gate) * up, else the clamped activation
template <typename T>
__global__ void glu_kernel(const T* __restrict__ gu, T* __restrict__ out, long long total, int I, float limit) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / I;
    const int c = (int)(i - t * I);
    const float g = gs_ld(gu + t * 2 * I + c), u = gs_ld(gu + t * 2 * I + I + c);
    gs_st(out + i, limit < 0.f ? g / (1.f + expf(-g)) * u : clamped_glu(g, u, limit));
  }
}

template <typename T, typename O>
static cudaError_t launch_simple(const void* A, long long lda, const void* B, long long ldb, void* C, long long ldc, const float* bias,
                                 int M, int N, int K, cudaStream_t s, const int* tile_expert = nullptr, const int* tile_rows = nullptr) {
  gemm_simple_kernel<T, O><<<dim3((N + 63) / 64, (M + 63) / 64), 256, 0, s>>>((const T*)A, lda, (const T*)B, ldb, (O*)C, ldc, bias, M, N, K,
                                                                              tile_expert, tile_rows);
  return cudaGetLastError();
}

// relu(z)^2 of the rows of z [.., I], in place; row_list (or null: all n) names n rows, -1 = none
template <typename T>
__global__ void __launch_bounds__(256) relu2_kernel(T* z, int I, const int* __restrict__ row_list, long long n, int vec) {
  pdl_trigger();
  pdl_wait();
  const int per = vec ? I / 8 : I;                   // units per row: 8 bf16 or one element
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n * per; i += (long long)gridDim.x * 256) {
    long long r = i / per;
    const int c = (int)(i - r * per);
    if (row_list) r = row_list[r];
    if (r < 0) continue;
    if constexpr (sizeof(T) == 2) {
      if (vec) {
        uint4* at = reinterpret_cast<uint4*>(z + r * I) + c;
        uint4 u = *at;
        __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&u);
#pragma unroll
        for (int k = 0; k < 8; ++k) { const float v = fmaxf(__bfloat162float(e[k]), 0.f); e[k] = __float2bfloat16(v * v); }
        *at = u;
        continue;
      }
    }
    const float v = fmaxf(gs_ld(z + r * I + c), 0.f);
    gs_st(z + r * I + c, v * v);
  }
}

// out[t] = a N(z) + b N(z^2) + c N(z^3) + e with N(v) = v / sqrt(mean(v^2) + eps) over the row; act = {a, b, c, e}.  A block per row.
template <typename T>
__global__ void __launch_bounds__(256) poly_norm_kernel(const T* __restrict__ z, const float* __restrict__ act, T* __restrict__ out, int I,
                                                        float eps, int vec) {
  __shared__ float red[3][8];
  pdl_trigger();
  pdl_wait();
  const T* zr = z + (size_t)blockIdx.x * I;
  T* o = out + (size_t)blockIdx.x * I;
  float s[3] = {0.f, 0.f, 0.f};
  constexpr int V = 16 / sizeof(T);
  const int step = vec ? V : 1;
  for (int c = threadIdx.x * step; c < I; c += 256 * step) {
    alignas(16) T e[V];
    if (vec) *reinterpret_cast<uint4*>(e) = *reinterpret_cast<const uint4*>(zr + c);
    else e[0] = zr[c];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      if (k >= step) break;
      const float v = gs_ld(e + k), q = v * v;
      s[0] += q; s[1] = fmaf(q, q, s[1]); s[2] = fmaf(q * q, q, s[2]);
    }
  }
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    s[i] = warp_sum(s[i]);
    if ((threadIdx.x & 31) == 0) red[i][threadIdx.x >> 5] = s[i];
  }
  __syncthreads();
  float f[3];
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) v += red[i][w];
    f[i] = act[i] / sqrtf(v / (float)I + eps);
  }
  const float last = act[3];
  for (int c = threadIdx.x * step; c < I; c += 256 * step) {
    alignas(16) T e[V];
    if (vec) *reinterpret_cast<uint4*>(e) = *reinterpret_cast<const uint4*>(zr + c);
    else e[0] = zr[c];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      if (k >= step) break;
      const float v = gs_ld(e + k);
      gs_st(e + k, fmaf(fmaf(fmaf(f[2], v, f[1]), v, f[0]), v, last));
    }
    if (vec) *reinterpret_cast<uint4*>(o + c) = *reinterpret_cast<uint4*>(e);
    else o[c] = e[0];
  }
}

}  // namespace blz

// in_f32: A and B are fp32 (C too); else A and B are bf16 and C is fp32 (out_f32) or bf16.  Leading dimensions in elements.
BLZ_API int blz_gemm_simple(const void* A, long long lda, const void* B, long long ldb, void* C, long long ldc, const float* bias,
                            int M, int N, int K, int in_f32, int out_f32, cudaStream_t s) {
  using namespace blz;
  if (M <= 0 || N <= 0 || K <= 0 || (M + 63) / 64 > 65535) return (int)cudaErrorInvalidValue;
  if (in_f32) return (int)launch_simple<float, float>(A, lda, B, ldb, C, ldc, bias, M, N, K, s);
  if (out_f32) return (int)launch_simple<__nv_bfloat16, float>(A, lda, B, ldb, C, ldc, bias, M, N, K, s);
  return (int)launch_simple<__nv_bfloat16, __nv_bfloat16>(A, lda, B, ldb, C, ldc, bias, M, N, K, s);
}

// The product over the padded row space of routed rows (blz_moe_plan): 128 rows of A per tile, B [experts][N][K]; types as A's.
BLZ_API int blz_gemm_simple_experts(const void* A, long long lda, const void* B, void* C, long long ldc, int tiles, int N, int K,
                                    const int* tile_expert, const int* tile_rows, int in_f32, cudaStream_t s) {
  using namespace blz;
  if (tiles <= 0 || N <= 0 || K <= 0 || tiles > 32767 || !tile_expert || !tile_rows) return (int)cudaErrorInvalidValue;
  const int M = tiles * 128;
  if (in_f32) return (int)launch_simple<float, float>(A, lda, B, K, C, ldc, nullptr, M, N, K, s, tile_expert, tile_rows);
  return (int)launch_simple<__nv_bfloat16, __nv_bfloat16>(A, lda, B, K, C, ldc, nullptr, M, N, K, s, tile_expert, tile_rows);
}

// relu(z)^2 in place: all n rows of z [n, I], or the n rows that row_list names (-1: none)
BLZ_API int blz_relu2(void* z, int I, const int* row_list, long long n, int f32, cudaStream_t s) {
  using namespace blz;
  if (n <= 0 || I <= 0) return (int)cudaErrorInvalidValue;
  const int vec = !f32 && I % 8 == 0 && (reinterpret_cast<uintptr_t>(z) & 15) == 0;
  const long long units = (n * (vec ? I / 8 : I) + 255) / 256;
  const dim3 grid((unsigned)(units < 16LL * sm_count() ? units : 16LL * sm_count()));
  if (f32) return (int)launch_pdl(relu2_kernel<float>, grid, dim3(256), 0, s, (float*)z, I, row_list, n, 0);
  return (int)launch_pdl(relu2_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (__nv_bfloat16*)z, I, row_list, n, vec);
}

// See poly_norm_kernel; z and out [T, I], act four floats.
BLZ_API int blz_poly_norm(const void* z, const float* act, void* out, int T, int I, float eps, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || I <= 0 || !act) return (int)cudaErrorInvalidValue;
  const int vec = I % (f32 ? 4 : 8) == 0 && ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  if (f32) return (int)launch_pdl(poly_norm_kernel<float>, dim3(T), dim3(256), 0, s, (const float*)z, act, (float*)out, I, eps, vec);
  return (int)launch_pdl(poly_norm_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, (const __nv_bfloat16*)z, act, (__nv_bfloat16*)out, I, eps, vec);
}

// limit < 0: silu(gate) * up
BLZ_API int blz_clamped_glu(const void* gu, void* out, int T, int I, float limit, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || I <= 0) return (int)cudaErrorInvalidValue;
  const long long total = (long long)T * I;
  const int blocks = (int)((total + 1023) / 1024 < 4LL * sm_count() ? (total + 1023) / 1024 : 4LL * sm_count());
  if (f32) return (int)launch_pdl(glu_kernel<float>, dim3(blocks), dim3(256), 0, s, (const float*)gu, (float*)out, total, I, limit);
  return (int)launch_pdl(glu_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, s, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out,
                         total, I, limit);
}
