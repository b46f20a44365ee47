// Matrix products on the CUDA cores: C[M,N] = A[M,K] B[N,K]^T (+ bias) for fp32 operands (a model served in true 32-bit; the
// tensor cores have no such mode) and for bf16 shapes that the TMA kernels do not take (a row length that is not a multiple
// of 16).  fp32 accumulation, no reduced-precision mode.  Also the gated activations as ops of their own.
#include "blaze/glu.cuh"
#include "blaze/host.h"
#include "blaze/sm100.cuh"

namespace blz {

__device__ __forceinline__ float gs_ld(const float* p) { return *p; }
__device__ __forceinline__ float gs_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void gs_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void gs_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// 64 x 64 output tile per 256-thread CTA, 16-deep K steps, 4 x 4 outputs per thread
template <typename T, typename O>
__global__ void __launch_bounds__(256) gemm_simple_kernel(const T* __restrict__ A, long long lda, const T* __restrict__ B,
                                                          long long ldb, O* __restrict__ C, long long ldc,
                                                          const float* __restrict__ bias, int M, int N, int K) {
  __shared__ float sa[16][68], sb[16][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
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
                                 int M, int N, int K, cudaStream_t s) {
  gemm_simple_kernel<T, O><<<dim3((N + 63) / 64, (M + 63) / 64), 256, 0, s>>>((const T*)A, lda, (const T*)B, ldb, (O*)C, ldc, bias, M, N, K);
  return cudaGetLastError();
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
