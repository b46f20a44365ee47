// Latent attention: softmax attention whose keys and values are linear maps of one cached vector per token.  A page block ("tiles" pages,
// one key/value head) holds 16 tokens of [latent (rank) | rotated key part (rot)], each part padded to 16 columns, as 8 x 8 core matrices
// (attn_maps.cuh): keys and values are read from the same bytes.
//   score(t, h, j) = (q_nope . uk_h c_j + rot(q_rot) . kr_j) * scale,   out(t, h) = uv_h (sum_j softmax(score)_j c_j), with a sink
//
// Two ways, by the number of a sequence's new tokens:
//   few (decode, verify rows, short portions): the maps are moved to the other side, q' = [uk_h^T q_nope | rot(q_rot)] against the cached
//     vectors themselves and uv_h on the weighted sum, so that all heads share every byte read (latent_rows_kernel, tcgen05);
//   many (prompt portions): the keys and values of the visible tokens are written out by head into scratch pages (gather, one product,
//     expand_store_kernel) for the prompt attention of attn_maps_tc.cu, which costs fewer products per score.
// 32-bit serving and sizes beyond these kernels take the first way with the plain kernel of attn_maps.cu.
#include "blaze/attn.cuh"
#include "blaze/attn_maps.cuh"
#include "blaze/host.h"

namespace blz {

__host__ __device__ __forceinline__ int up16(int n) { return (n + 15) / 16 * 16; }

// rows of sequences with at most max_tokens new tokens
struct RowFilter {
  const int* seq_of_row;       // [T], -1 = padding
  const int* q_start;
  int max_tokens;
  __device__ __forceinline__ int len(int t) const {            // new tokens of the row's sequence, 0 = padding
    const int b = seq_of_row[t];
    return b < 0 ? 0 : q_start[b + 1] - q_start[b];
  }
  __device__ __forceinline__ bool has(int t) const { const int n = len(t); return n > 0 && n <= max_tokens; }
};

// cos and sin of position * frequency i; freq holds the frequencies and what rounding them to 32 bits left over
__device__ __forceinline__ void turn_of(const float* freq, int half, int i, float pos, float& c, float& s) {
  const float hi = freq[i], ang = pos * hi, rest = fmaf(pos, hi, -ang) + pos * freq[half + i];
  float s0, c0;
  sincosf(ang, &s0, &c0);
  c = fmaf(-rest, s0, c0);
  s = fmaf(rest, c0, s0);
}

// ------------------------------------------------------------------------------------------ latents of new tokens
struct LatentPrepParams {
  const void* proj;            // [T, ld]: the queries' latent from q_off on, the keys' latent and rotated part from kv_off
  void* q_lat;                 // [T, q_rank]
  void* pool;
  const float *q_norm, *c_norm, *freq;
  const int *positions, *slot_mapping;
  long long ld, q_off, kv_off, page_stride;
  int q_rank, rank, rot, rot_dims;
  float eps;
};

// block (row, 0): the queries' latent, normed; block (row, 1): the keys' latent, normed, and the rotated part, into their page slot.
// VEC columns per thread and turn; the first KEEP turns stay in registers between the sum of squares and the result.
template <typename T, int VEC>
__global__ void __launch_bounds__(128) latent_prep_kernel(LatentPrepParams p) {
  constexpr int KEEP = VEC == 8 ? 2 : 1;
  __shared__ float red[4];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const bool keys = blockIdx.y == 1;
  const int slot = keys ? p.slot_mapping[t] : 0;
  if (slot < 0) return;
  const T* src = reinterpret_cast<const T*>(p.proj) + (size_t)t * p.ld + (keys ? p.kv_off : p.q_off);
  const int n = keys ? p.rank : p.q_rank;
  const float* w = keys ? p.c_norm : p.q_norm;
  auto load = [&](int j, float (&v)[VEC]) {
    if constexpr (VEC == 8) {
      const uint4 u = *reinterpret_cast<const uint4*>(src + j);
      const uint32_t x[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
      for (int k = 0; k < 4; ++k) { v[2 * k] = __uint_as_float(x[k] << 16); v[2 * k + 1] = __uint_as_float(x[k] & 0xffff0000u); }
    } else {
      v[0] = ad_ld(src + j);
    }
  };
  float ss = 0.f, kept[KEEP][VEC];
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int j = (i * 128 + tid) * VEC;
    if (j < n) {
      load(j, kept[i]);
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(kept[i][k], kept[i][k], ss);
    }
  }
  for (int j = (KEEP * 128 + tid) * VEC; j < n; j += 128 * VEC) {
    float v[VEC];
    load(j, v);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss = fmaf(v[k], v[k], ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  const float f = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)n + p.eps);
  const int rp = up16(p.rank), tp = up16(p.rot), D = rp + tp, half = p.rot_dims / 2, tok = slot & 15;
  T* q_lat = reinterpret_cast<T*>(p.q_lat) + (size_t)t * p.q_rank;
  T* page = reinterpret_cast<T*>(p.pool) + (size_t)(slot >> 4) * p.page_stride;
  auto put = [&](int j, const float (&v)[VEC]) {
    T* dst = keys ? page + core_off(tok, j, D) : q_lat + j;
    if constexpr (VEC == 8) {
      float y[8];
      const float4 a = *reinterpret_cast<const float4*>(w + j), b = *reinterpret_cast<const float4*>(w + j + 4);
      const float g[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
      for (int k = 0; k < 8; ++k) y[k] = v[k] * f * g[k];
      *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]), pack_bf16x2(y[4], y[5]), pack_bf16x2(y[6], y[7]));
    } else {
      ad_st(dst, v[0] * f * w[j]);
    }
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
    if ((i * 128 + tid) * VEC < n) put((i * 128 + tid) * VEC, kept[i]);
  for (int j = (KEEP * 128 + tid) * VEC; j < n; j += 128 * VEC) {
    float v[VEC];
    load(j, v);
    put(j, v);
  }
  if (!keys) return;
  for (int j = n + tid; j < rp; j += 128) ad_st(page + core_off(tok, j, D), 0.f);
  const float pos = (float)p.positions[t];
  for (int j = 127 - tid; j < tp; j += 128) {          // the threads with the least of the latent
    float v = j < p.rot ? ad_ld(src + n + j) : 0.f;
    if (j < 2 * half) {
      const bool low = j < half;
      const float other = ad_ld(src + n + (low ? j + half : j - half));
      float c, s;
      turn_of(p.freq, half, low ? j : j - half, pos, c, s);
      v = low ? v * c - other * s : v * c + other * s;
    }
    ad_st(page + core_off(tok, rp + j, D), v);
  }
}

// ------------------------------------------------------------------------------------------ query rotation
// The rotated part of the queries q [T, heads, dim + rot]: turned in place for the rows of long portions (a block per row), or, beside
// the product that maps a query to the latents, behind the mapped query in q_eff [T, heads, D] (pads zeroed).
struct LatentRotParams {
  void* q;
  void* q_eff;
  const float* freq;
  const int* positions;
  RowFilter rows;              // which rows are mapped; the others are turned in place
  int heads, dim, rot, rot_dims, rank;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_rot_kernel(LatentRotParams p) {
  extern __shared__ float cs[];                      // [rot_dims / 2][cos, sin]
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, half = p.rot_dims / 2;
  if (p.rows.len(t) <= p.rows.max_tokens) return;
  const float pos = (float)p.positions[t];
  for (int i = threadIdx.x; i < half; i += 128) turn_of(p.freq, half, i, pos, cs[2 * i], cs[2 * i + 1]);
  __syncthreads();
  T* q = reinterpret_cast<T*>(p.q) + (size_t)t * p.heads * (p.dim + p.rot);
  for (int i = threadIdx.x; i < p.heads * half; i += 128) {
    T* x = q + (size_t)(i / half) * (p.dim + p.rot) + p.dim + i % half;
    const float c = cs[2 * (i % half)], s = cs[2 * (i % half) + 1], u = ad_ld(x), v = ad_ld(x + half);
    ad_st(x, u * c - v * s);
    ad_st(x + half, v * c + u * s);
  }
}

// rows [m0, m0 + 64) of head h, by n threads: columns rank .. D of q_eff
template <typename T>
__device__ __forceinline__ void place_rotated(const LatentRotParams& p, int m0, int M, int h, int n) {
  const int half = p.rot_dims / 2, rp = up16(p.rank), D = rp + up16(p.rot), zeros = D - p.rank - 2 * half, per = half + zeros;
  for (int i = threadIdx.x; i < 64 * per; i += n) {
    const int m = m0 + i / per, k = i % per;
    if (m >= M || !p.rows.has(m)) continue;
    const T* x = reinterpret_cast<const T*>(p.q) + ((size_t)m * p.heads + h) * (p.dim + p.rot) + p.dim;
    T* e = reinterpret_cast<T*>(p.q_eff) + ((size_t)m * p.heads + h) * D;
    if (k < half) {
      float c, s;
      turn_of(p.freq, half, k, (float)p.positions[m], c, s);
      const float u = ad_ld(x + k), v = ad_ld(x + k + half);
      ad_st(e + rp + k, u * c - v * s);
      ad_st(e + rp + k + half, v * c + u * s);
    } else {                                         // the pad of the latent, what is not turned, the pad behind it
      const int z = k - half, col = z < rp - p.rank ? p.rank + z : z + p.rank + 2 * half, j = col - rp;
      ad_st(e + col, j >= 0 && j < p.rot ? ad_ld(x + j) : 0.f);
    }
  }
}

// ------------------------------------------------------------------------------------------ products by head
// C[t, h, :] = A[t, h, :] B[h]^T for the rows the filter has; B [heads][N][K].  64 x 64 outputs per block, grid (N, M, heads).
struct HeadGemmParams {
  const void *a, *b;
  void* c;
  long long lda, sa, ldc, sc;  // elements: row and head strides
  int M, N, K;
  RowFilter rows;
  LatentRotParams rot;         // q_eff not null: one block more along N places the rotated parts
};
static constexpr int kHgStages = 4, kHgPitch = 72;             // tiles of 64 columns under way; row pitch: 8 rows cover all banks

__global__ void __launch_bounds__(256) head_gemm_f32_kernel(HeadGemmParams p) {
  __shared__ float sa[16][68], sb[16][68];
  __shared__ int any;
  pdl_trigger();
  pdl_wait();
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, h = blockIdx.z, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  if (threadIdx.x == 0) any = 0;
  __syncthreads();
  if (threadIdx.x < 64 && m0 + threadIdx.x < p.M && p.rows.has(m0 + threadIdx.x)) any = 1;
  __syncthreads();
  if (!any) return;
  if (n0 >= p.N) return place_rotated<float>(p.rot, m0, p.M, h, 256);
  const float* A = reinterpret_cast<const float*>(p.a) + h * p.sa;
  const float* B = reinterpret_cast<const float*>(p.b) + (size_t)h * p.N * p.K;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = threadIdx.x + i * 256, r = e >> 4, k = e & 15;
      sa[k][r] = (m0 + r < p.M && k0 + k < p.K) ? A[(size_t)(m0 + r) * p.lda + k0 + k] : 0.f;
      sb[k][r] = (n0 + r < p.N && k0 + k < p.K) ? B[(size_t)(n0 + r) * p.K + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(sa[k][ty * 4 + i], sb[k][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= p.M || !p.rows.has(m)) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n0 + tx * 4 + j < p.N) reinterpret_cast<float*>(p.c)[(size_t)m * p.ldc + h * p.sc + n0 + tx * 4 + j] = acc[i][j];
  }
}

__device__ __forceinline__ void lt_ldm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lt_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// bf16: few rows against many small weights, so the products ride on the reads (warp-level MMAs); 4 warps of 32 x 32 outputs, the next
// tiles of both operands on their way as asynchronous copies
__global__ void __launch_bounds__(128) head_gemm_kernel(HeadGemmParams p, int vec) {
  constexpr int LD = kHgPitch;
  extern __shared__ __align__(16) __nv_bfloat16 ring[];          // [stages][A 64 x LD | B 64 x LD]
  __shared__ uint8_t live[64];                       // rows the filter has
  pdl_trigger();
  pdl_wait();
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, h = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (n0 >= p.N) return place_rotated<__nv_bfloat16>(p.rot, m0, p.M, h, 128);
  const __nv_bfloat16* A = reinterpret_cast<const __nv_bfloat16*>(p.a) + h * p.sa;
  const __nv_bfloat16* B = reinterpret_cast<const __nv_bfloat16*>(p.b) + (size_t)h * p.N * p.K;
  const int wm = (warp & 1) * 32, wn = (warp >> 1) * 32, tiles = (p.K + 63) / 64;
  const bool upper = m0 + 32 < p.M;                  // the second half of the rows exists
  auto send = [&](int t) {
    __nv_bfloat16* dst = ring + (t % kHgStages) * 128 * LD;
    for (int i = tid; t < tiles && i < 1024; i += 128) {
      const int which = i >> 9, r = i >> 3 & 63, c = t * 64 + (i & 7) * 8, row = (which ? n0 : m0) + r, lim = which ? p.N : p.M;
      const __nv_bfloat16* src = (which ? B + (size_t)row * p.K : A + (size_t)row * p.lda) + c;
      __nv_bfloat16* to = dst + (which * 64 + r) * LD + (i & 7) * 8;
      const bool live = row < lim && c < p.K;
      if (vec) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(to)), "l"(live ? src : A), "r"(live ? 16 : 0) : "memory");
      } else {
        for (int k = 0; k < 8; ++k) to[k] = live && c + k < p.K ? src[k] : __float2bfloat16(0.f);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float acc[2][4][4] = {};
  for (int t = 0; t < kHgStages - 1; ++t) send(t);
  const bool mine = tid < 64 && m0 + tid < p.M && p.rows.has(m0 + tid);
  if (tid < 64) live[tid] = mine;
  if (!__syncthreads_or(mine)) {                     // none of them
    asm volatile("cp.async.wait_all;" ::: "memory");
    return;
  }
  for (int t = 0; t < tiles; ++t) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kHgStages - 2) : "memory");
    __syncthreads();                                 // tile t is there, and everyone is done with the slot that is filled next
    send(t + kHgStages - 1);
    const __nv_bfloat16 *sa = ring + (t % kHgStages) * 128 * LD, *sb = sa + 64 * LD;
    if (wm == 0 || upper) {
      const int ks = min(64, p.K - t * 64);
      for (int k = 0; k < ks; k += 16) {
        uint32_t a[2][4], bq[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          lt_ldm4(a[i], smem_u32(sa + (wm + i * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8));
          lt_ldm4(bq[i], smem_u32(sb + (wn + i * 16 + (lane >> 4) * 8 + (lane & 7)) * LD + k + (lane >> 3 & 1) * 8));
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) lt_mma(acc[i][j], a[i], bq[j >> 1][(j & 1) * 2], bq[j >> 1][(j & 1) * 2 + 1]);
      }
    }
  }
  __nv_bfloat16* C = reinterpret_cast<__nv_bfloat16*>(p.c) + h * p.sc;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int m = m0 + wm + i * 16 + (lane >> 2) + half * 8;
      if (!live[m - m0]) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + wn + j * 8 + (lane & 3) * 2;
        const float x = acc[i][j][half * 2], y = acc[i][j][half * 2 + 1];
        __nv_bfloat16* dst = C + (size_t)m * p.ldc + n;
        if (vec && n + 1 < p.N) *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(x, y);
        else {
          if (n < p.N) dst[0] = __float2bfloat16(x);
          if (n + 1 < p.N) dst[1] = __float2bfloat16(y);
        }
      }
    }
}

// ------------------------------------------------------------------------------------------ few new tokens
// A CTA takes R rows (new tokens x heads) of one sequence and a range of its pages, 128 keys (8 pages) at a time:
//   S^T = C Q'^T     A = the 128 cached vectors (K-major), B = the R queries; 128 keys on the lanes, R columns, two buffers
//   O^T += C^T P^T   A = 128 latent columns of the same block (MN-major), B = the weights [keys x R]; one accumulator per 128 columns
// so that with few rows the tensor core spends N = R columns per key and not 128.  A weight enters as two bf16 numbers, value and
// remainder, so it is not rounded to 8 bits: they are columns of their own (N = 2 R), since with few columns an MMA costs what its A
// operand costs, and the two sums of a row meet at the end.  Scores, weights and sums are fp32; a row's running maximum moves only when its scores
// outgrow it by 2^8, and then the accumulators are rescaled in tensor memory.
// Softmax warps: a key per thread, R / 2 columns (16 rows: all) in each of the two warpgroups; then a page loader and an MMA issuer.
struct LatentRowsParams {
  const void* q;               // [T, heads, D]
  void* out;                   // [T, heads, rank]
  const void* pool;
  const float* sink;           // [heads] or null
  const int *block_table, *slots, *q_start, *ctx_len;
  float *part_o, *part_ml;
  long long page_stride;
  int bt_stride, heads, rank, D, window, max_tokens, row_blocks, splits, stages;
  float scale;
  int* status;
};

__host__ __device__ constexpr int lr_groups(int R) { return R >= 32 ? 2 : 1; }      // softmax warpgroups
__host__ __device__ constexpr int lr_threads(int R) { return lr_groups(R) * 128 + 64; }
static constexpr float kLrLazy = 8.f;
static constexpr int kLrRowBytes = 48;         // shared memory per row besides the operands, a multiple of 16
static constexpr float kLrNone = -1e30f;       // the maximum of a row that has seen no key

template <bool MAX>
__device__ __forceinline__ float lr_op(float a, float b) { return MAX ? fmaxf(a, b) : a + b; }
// maxima (or sums) of every column over the 32 lanes -> dst[R]
template <int R, bool MAX>
__device__ __forceinline__ void reduce_lanes(const float (&v)[R], int lane, float* dst) {
#pragma unroll
  for (int base = 0; base + 32 <= R; base += 32) {
    float a[16];
#pragma unroll
    for (int w = 16; w >= 1; w >>= 1) {
      const bool up = lane & w;
#pragma unroll
      for (int j = 0; j < w; ++j) {
        const float lo = w == 16 ? v[base + j] : a[j], hi = w == 16 ? v[base + (j + w) % 32] : a[(j + w) % 16];
        a[j] = lr_op<MAX>(up ? hi : lo, __shfl_xor_sync(0xffffffffu, up ? lo : hi, w));
      }
    }
    dst[base + lane] = a[0];
  }
  if constexpr (R % 32 == 16) {
    constexpr int base = R - 16;
    float a[8];
#pragma unroll
    for (int w = 8; w >= 1; w >>= 1) {
      const bool up = lane & (2 * w);
#pragma unroll
      for (int j = 0; j < w; ++j) {
        const float lo = w == 8 ? v[base + j] : a[j], hi = w == 8 ? v[base + j + w] : a[(j + w) % 8];
        a[j] = lr_op<MAX>(up ? hi : lo, __shfl_xor_sync(0xffffffffu, up ? lo : hi, 2 * w));
      }
    }
    a[0] = lr_op<MAX>(a[0], __shfl_xor_sync(0xffffffffu, a[0], 1));
    if ((lane & 1) == 0) dst[base + (lane >> 1)] = a[0];
  }
}

template <int R>
__global__ void __launch_bounds__(lr_threads(R), R <= 32 ? 2 : 1) latent_rows_kernel(LatentRowsParams p) {
  constexpr int WG = lr_groups(R), RC = R / WG, NT = WG * 128, kLoader = WG * 4, kIssuer = kLoader + 1;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~uintptr_t(127));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, H = p.heads, D = p.D, ST = p.stages;
  const int b = blockIdx.y, rb = blockIdx.x / p.splits, split = blockIdx.x % p.splits;
  pdl_trigger();
  pdl_wait();
  const int r0 = p.q_start[b], qlen = p.q_start[b + 1] - r0, rows = qlen * H;
  if (qlen <= 0 || qlen > p.max_tokens || rb * R >= rows) return;
  const int pos0 = p.ctx_len[b] - qlen, tok_lo = rb * R / H, tok_hi = (min(rb * R + R, rows) - 1) / H;
  const int pg_lo = first_key(pos0 + tok_lo, p.window) >> 4, pages = ((pos0 + tok_hi) >> 4) - pg_lo + 1, per = (pages + p.splits - 1) / p.splits;
  const int s_lo = pg_lo + split * per, s_n = min(per, pg_lo + pages - s_lo), n = s_n > 0 ? (s_n + 7) / 8 : 0;
  const size_t w0 = (((size_t)b * p.row_blocks + rb) * p.splits + split) * R;        // this CTA's rows in the workspace
  if (n == 0) {
    for (int r = threadIdx.x; r < R; r += lr_threads(R)) { p.part_ml[(w0 + r) * 2] = kLrNone; p.part_ml[(w0 + r) * 2 + 1] = 0.f; }
    return;
  }
  const int nvb = (p.rank + 127) / 128, tile = 256 * D;                            // accumulators; bytes of 128 cached vectors
  const int* bt = p.block_table + (size_t)p.slots[b] * p.bt_stride;
  auto page_of = [&](int i) { return lane < 8 ? bt[min(s_lo + i * 8 + lane, s_lo + s_n - 1)] : 0; };      // beyond the range: the last page again, masked
  int page = warp == kLoader ? page_of(0) : 0;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem);
  uint64_t *k_full = bars, *k_empty = bars + 4, *s_full = bars + 8, *p_full = bars + 10, *pv_done = bars + 11, *q_full = bars + 12;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 13);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_red = reinterpret_cast<float*>(smem + 128);         // [4][R]
  float* s_m = s_red + 4 * R;
  float* s_f = s_m + R;
  float* s_t = s_f + R;                                        // products above which a row's maximum moves
  int2* s_vis = reinterpret_cast<int2*>(s_t + R);              // first and last visible key of a row
  uint8_t* sQ = smem + 128 + kLrRowBytes * R;
  uint8_t* sP = sQ + 2 * R * D;
  uint8_t* ring = sP + 512 * R;
  uint32_t cols = 32;
  while (cols < (uint32_t)((2 + 2 * nvb) * R)) cols *= 2;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 4; ++i) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); }
    for (int i = 0; i < 2; ++i) mbar_init(&s_full[i], 1);
    mbar_init(p_full, WG * 4);
    mbar_init(pv_done, 1);
    mbar_init(q_full, WG * 4);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == kIssuer) tmem_alloc(tmem_slot, cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  if (warp == kLoader) {
    // -------------------------------------------------------------- page loader
    int i = 0;
    for (; i < n; ++i) {
      const int st = i % ST, next = i + 1 < n ? page_of(i + 1) : 0;
      if (!__all_sync(0xffffffffu, mbar_wait(&k_empty[st], (uint32_t)(((i / ST) & 1) ^ 1), abort_flag, p.status))) break;
      if (lane == 0) mbar_expect_tx(&k_full[st], tile);
      __syncwarp();
      if (lane < 8)
        bulk_load(ring + st * tile + lane * 32 * D, reinterpret_cast<const __nv_bfloat16*>(p.pool) + (size_t)page * p.page_stride, 32 * D, &k_full[st]);
      __syncwarp();
      page = next;
    }
    if (i < n)                               // given up: what was sent lands before the block may end
      for (int k = max(i - ST, 0); k < i; ++k) {
        const long long t0 = clock64();
        while (!mbar_try_sleep(&k_full[k % ST], (uint32_t)((k / ST) & 1), 20000u) && clock64() - t0 < kSpinLimit) {}
      }
  } else if (warp == kIssuer) {
    // -------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      const uint32_t id_s = make_idesc(1, 1, 128, R), id_o = make_idesc(1, 1, 128, 2 * R, 1, 1);
      // descriptors once, then steps of their address field (16 bytes): an MMA with few columns takes less time than its descriptors
      const uint64_t q_desc = make_smem_desc(smem_u32(sQ), 128, D * 16, kSwzNone), p_desc = make_smem_desc(smem_u32(sP), 32 * R, 128, kSwzNone);
      const uint32_t ra = smem_u32(ring);
      auto qk = [&](int i) {
        const uint64_t k_desc = make_smem_desc(ra + (i % ST) * tile, 128, D * 16, kSwzNone);
        const uint32_t d = tmem + (i & 1) * R;
#pragma unroll 6
        for (int s = 0; s < D / 16; ++s) mma_f16(d, k_desc + s * 16, q_desc + s * 16, id_s, s > 0);
        mma_commit(&s_full[i & 1]);
      };
      auto pv = [&](int i) {
        uint64_t v_desc = make_smem_desc(ra + (i % ST) * tile, D * 16, 128, kSwzNone);
        const uint32_t acc = i > 0;
        for (int v = 0; v < nvb; ++v, v_desc += 128) {
          const uint32_t d = tmem + (2 + 2 * v) * R;
#pragma unroll
          for (int s = 0; s < 8; ++s)        // a page of 16 keys per MMA
            mma_f16(d, v_desc + s * 2 * D, p_desc + s * 4 * R, id_o, s > 0 ? 1u : acc);
        }
        mma_commit(pv_done);
        mma_commit(&k_empty[i % ST]);
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status);
      tc_fence_after();
      // whichever is ready: the value product of tile j, or the scores of tile i, at most two tiles ahead of it (two score buffers)
      long long t0 = clock64();
      for (int i = 0, j = 0; ok && j < n;) {
        if (i > j && mbar_try(p_full, (uint32_t)(j & 1))) {
          tc_fence_after();
          pv(j++);
        } else if (i < n && i < j + 2 && mbar_try(&k_full[i % ST], (uint32_t)((i / ST) & 1))) {
          qk(i++);
        } else {
          if (*abort_flag) ok = false;
          else if (clock64() - t0 > kSpinLimit) {
            *abort_flag = 1;
            if (p.status) atomicCAS(p.status, kOk, kErrMbarTimeout);
            ok = false;
          }
          continue;
        }
        t0 = clock64();
      }
    }
  } else {
    // -------------------------------------------------------------- softmax: this thread's key of every tile
    const int tid = threadIdx.x;
    const int quad = warp & 3, c0 = (warp >> 2) * RC, key_of = tid & 127;        // this thread's lane quadrant, first column and key
    const uint32_t lanes = (uint32_t)(quad * 32) << 16;
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + ((size_t)r0 * H + (size_t)rb * R) * D;
    const int live = min(R, rows - rb * R);
    copy_rows(reinterpret_cast<__nv_bfloat16*>(sQ), R, D, D, tid, NT, q, [&](int r) { return r < live ? q + (size_t)r * D : nullptr; });
    const int end = (s_lo + s_n) * 16 - 1;
    if (tid < R) {
      const int pos = tid < live ? pos0 + (rb * R + tid) / H : -1;
      s_vis[tid] = make_int2(first_key(pos, p.window), min(pos, end));
      s_m[tid] = s_t[tid] = kLrNone;
    }
    copies_wait();
    fence_async_smem();
    __syncwarp();
    if (lane == 0) mbar_arrive(q_full);
    bar_sync(1, NT);
    const int all_lo = first_key(pos0 + tok_hi, p.window), all_hi = min(pos0 + tok_lo, end);        // what every row sees
    const float sc = p.scale * kLog2e;
    float l[RC];
#pragma unroll
    for (int r = 0; r < RC; ++r) l[r] = 0.f;
    bool ok = true;                          // once a wait has run out the others return at once; the barriers stay matched
    for (int i = 0; i < n; ++i) {
      ok = __all_sync(0xffffffffu, mbar_wait(&s_full[i & 1], (uint32_t)((i >> 1) & 1), abort_flag, p.status)) && ok;
      tc_fence_after();
      float v[RC];
      {
        uint32_t x[RC / 16][16];
#pragma unroll
        for (int k = 0; k < RC / 16; ++k) tmem_ld16(tmem + (i & 1) * R + lanes + c0 + k * 16, x[k]);
        tmem_ld_wait();
#pragma unroll
        for (int r = 0; r < RC; ++r) v[r] = __uint_as_float(x[r / 16][r % 16]);
      }
      const int k0 = (s_lo + i * 8) * 16, key = k0 + key_of;
      if (k0 < all_lo || k0 + 127 > all_hi) {
#pragma unroll
        for (int r = 0; r < RC; ++r) {
          const int2 vis = s_vis[c0 + r];
          if (key < vis.x || key > vis.y) v[r] = -INFINITY;
        }
      }
      // most tiles outgrow no row's maximum: one vote, and the columns are reduced only where it says so
      bool grow = false;
#pragma unroll
      for (int r = 0; r < RC; r += 4) {
        const float4 t = *reinterpret_cast<const float4*>(s_t + c0 + r);
        grow |= v[r] > t.x || v[r + 1] > t.y || v[r + 2] > t.z || v[r + 3] > t.w;
      }
      const bool calm = bar_red_and(2, NT, !grow);
      if (!calm) {
        reduce_lanes<RC, true>(v, lane, s_red + quad * R + c0);
        bar_sync(1, NT);
        if (tid < R) {
          const float t = fmaxf(fmaxf(s_red[tid], s_red[R + tid]), fmaxf(s_red[2 * R + tid], s_red[3 * R + tid])) * sc, m = s_m[tid];
          s_f[tid] = t > m + kLrLazy ? ex2(m - t) : 1.f;
          if (t > m + kLrLazy) { s_m[tid] = t; s_t[tid] = (t + kLrLazy) / sc; }
        }
        bar_sync(1, NT);
      }
      if (i > 0) ok = __all_sync(0xffffffffu, mbar_wait(pv_done, (uint32_t)((i - 1) & 1), abort_flag, p.status)) && ok;
      if (!calm) {
        tc_fence_after();
#pragma unroll
        for (int r = 0; r < RC; ++r) l[r] *= s_f[c0 + r];
        if (i > 0) {
#pragma unroll 1
          for (int k = 0; k < 2 * nvb * RC; k += 16) {
            const int at = (2 + k / RC) * R + c0 + k % RC;
            uint32_t x[16];
            tmem_ld16(tmem + at + lanes, x);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) x[j] = __float_as_uint(__uint_as_float(x[j]) * s_f[c0 + k % RC + j]);
            tmem_st16(tmem + at + lanes, x);
          }
          tmem_st_wait();
        }
      }
      uint8_t* dst = sP + (key_of >> 3) * 32 * R + (key_of & 7) * 16 + c0 * 16;
#pragma unroll
      for (int g = 0; g < RC / 8; ++g) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = g * 8 + j * 2;
          const float2 m = *reinterpret_cast<const float2*>(s_m + c0 + r);
          const float a = ex2(fmaf(v[r], sc, -m.x)), c = ex2(fmaf(v[r + 1], sc, -m.y));
          l[r] += a;
          l[r + 1] += c;
          hi[j] = pack_bf16x2(a, c);
          lo[j] = pack_bf16x2(a - __uint_as_float(hi[j] << 16), c - __uint_as_float(hi[j] & 0xffff0000u));
        }
        *reinterpret_cast<uint4*>(dst + g * 128) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(dst + 16 * R + g * 128) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      fence_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    ok = __all_sync(0xffffffffu, mbar_wait(pv_done, (uint32_t)((n - 1) & 1), abort_flag, p.status)) && ok;
    tc_fence_after();
    reduce_lanes<RC, false>(l, lane, s_red + quad * R + c0);
    bar_sync(1, NT);
    if (tid < R) {
      const float sum = s_red[tid] + s_red[R + tid] + s_red[2 * R + tid] + s_red[3 * R + tid], m = s_m[tid];
      if (p.splits > 1) {
        p.part_ml[(w0 + tid) * 2] = m;
        p.part_ml[(w0 + tid) * 2 + 1] = sum;
        s_f[tid] = 1.f;
      } else {
        s_f[tid] = 1.f / (sum + (p.sink && tid < live ? ex2(p.sink[(rb * R + tid) % H] * kLog2e - m) : 0.f));
      }
    }
    bar_sync(1, NT);
    __nv_bfloat16* s_out = reinterpret_cast<__nv_bfloat16*>(ring);         // [R][128]: the tiles have been used
    float* part = p.part_o + w0 * p.rank;
    for (int c = 0; c < nvb; ++c) {
      const int at = c * 128, width = min(128, p.rank - at);
#pragma unroll 1
      for (int k = c0; k < c0 + RC; k += 16) {           // (loops that run once per CTA are kept short: their code is not in the cache)
        uint32_t x[16], y[16];
        tmem_ld16(tmem + (2 + 2 * c) * R + lanes + k, x);
        tmem_ld16(tmem + (3 + 2 * c) * R + lanes + k, y);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; ++j) x[j] = __float_as_uint((__uint_as_float(x[j]) + __uint_as_float(y[j])) * s_f[k + j]);
        if (p.splits == 1) {
#pragma unroll
          for (int j = 0; j < 16; ++j) s_out[(k + j) * 128 + key_of] = __float2bfloat16(__uint_as_float(x[j]));
        } else if (key_of < width) {
          float* dst = part + (size_t)k * p.rank + at + key_of;             // rows beyond the live ones have a place too
#pragma unroll
          for (int j = 0; j < 16; ++j) dst[j * p.rank] = __uint_as_float(x[j]);
        }
      }
      if (p.splits > 1) continue;
      bar_sync(1, NT);
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + ((size_t)r0 * H + (size_t)rb * R) * p.rank + at;
      if (ok && p.rank % 8 == 0) {
        for (int i = tid; i < live * 16; i += NT) {
          const int r = i >> 4, j = (i & 15) * 8;
          if (j < width) *reinterpret_cast<uint4*>(out + (size_t)r * p.rank + j) = *reinterpret_cast<const uint4*>(s_out + r * 128 + j);
        }
      } else if (ok) {
        for (int i = tid; i < live * 128; i += NT)
          if (key_of < width) out[(size_t)(i >> 7) * p.rank + key_of] = s_out[i];
      }
      bar_sync(1, NT);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kIssuer) {
    tc_fence_after();
    tmem_dealloc(tmem, cols);
  }
}

// joins the split key ranges of one row; grid (rows of the longest short sequence, B)
__global__ void __launch_bounds__(128) latent_combine_kernel(LatentRowsParams p, int R) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, rr = blockIdx.x, r0 = p.q_start[b], qlen = p.q_start[b + 1] - r0;
  if (qlen > p.max_tokens || rr >= qlen * p.heads) return;
  __shared__ float s_w[32];
  const size_t w = ((size_t)b * p.row_blocks + rr / R) * p.splits * R + rr % R;      // split s at w + s * R
  const int lane = threadIdx.x & 31;
  const bool mine = lane < p.splits;
  const float m = mine ? p.part_ml[(w + (size_t)lane * R) * 2] : kLrNone, l = mine ? p.part_ml[(w + (size_t)lane * R) * 2 + 1] : 0.f;
  const float top = warp_max(m), f = m == kLrNone ? 0.f : ex2(m - top);
  const float inv = 1.f / (warp_sum(f * l) + (p.sink ? ex2(p.sink[rr % p.heads] * kLog2e - top) : 0.f));
  if (threadIdx.x < 32) s_w[lane] = f * inv;
  __syncthreads();
  for (int c = threadIdx.x; c < p.rank; c += 128) {
    float o = 0.f;
    for (int s0 = 0; s0 < p.splits; s0 += 8) {
      float x[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) x[k] = s0 + k < p.splits && s_w[s0 + k] != 0.f ? p.part_o[(w + (size_t)(s0 + k) * R) * p.rank + c] : 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) o = fmaf(x[k], s_w[(s0 + k) & 31], o);
    }
    reinterpret_cast<__nv_bfloat16*>(p.out)[((size_t)r0 * p.heads + rr) * p.rank + c] = __float2bfloat16(o);
  }
}

static int rows_smem(int R, int D, int stages) { return 128 + 128 + kLrRowBytes * R + 2 * R * D + 512 * R + stages * 256 * D + 2048; }
static constexpr int kLrSmem = 227 * 1024, kLrSmemHalf = 113 * 1024;      // one CTA per SM, two

template <int R>
static int launch_rows(LatentRowsParams p, int B, int longest, cudaStream_t s) {
  const int fit = R <= 32 && rows_smem(R, p.D, 1) <= kLrSmemHalf ? kLrSmemHalf : kLrSmem;
  int st = 4;
  while (st > 1 && rows_smem(R, p.D, st) > fit) --st;
  const int sm = rows_smem(R, p.D, st);
  if (sm > kLrSmem || (2 + 2 * ((p.rank + 127) / 128)) * R > 512 || p.splits > 32) return (int)cudaErrorInvalidValue;
  p.stages = st;
  static PerDeviceOnce once;
  cudaError_t e = once.smem_limit(latent_rows_kernel<R>, kLrSmem);
  if (e != cudaSuccess) return (int)e;
  e = launch_pdl(latent_rows_kernel<R>, dim3(p.row_blocks * p.splits, B), dim3(lr_threads(R)), sm, s, p);
  if (e != cudaSuccess || p.splits == 1) return (int)e;
  return (int)launch_pdl(latent_combine_kernel, dim3(longest * p.heads, B), dim3(128), 0, s, p, R);
}

// ------------------------------------------------------------------------------------------ many new tokens: keys and values by head
// rows of the listed pages' latents -> [pages * 16, rank]; 8 columns per thread
__global__ void __launch_bounds__(256) latent_gather_kernel(const __nv_bfloat16* pool, long long page_stride, const int* pages, int n,
                                                            __nv_bfloat16* out, int rank, int D) {
  pdl_trigger();
  pdl_wait();
  const int per = (rank + 7) / 8;
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < (long long)n * 16 * per; i += (long long)gridDim.x * 256) {
    const int c = (int)(i % per) * 8, t = (int)(i / per & 15), pg = (int)(i / per >> 4);
    const uint4 u = *reinterpret_cast<const uint4*>(pool + (size_t)pages[pg] * page_stride + core_off(t, c, D));
    __nv_bfloat16* dst = out + ((size_t)pg * 16 + t) * rank + c;
    if (rank % 8 == 0) {
      *reinterpret_cast<uint4*>(dst) = u;
    } else {
      const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&u);
      for (int k = 0; k < 8 && c + k < rank; ++k) dst[k] = e[k];
    }
  }
}

struct ExpandParams {
  const __nv_bfloat16* kv;     // [n * 16, ld]: keys [heads][dim] | values [heads][vdim]
  const __nv_bfloat16* pool;   // latent pages, for the rotated key parts
  __nv_bfloat16* out;          // [n][heads][K 16 x dp | V 16 x vp]
  const int* pages;
  long long ld, page_stride;
  int n, heads, dim, rot, vdim, rank;
};

// one thread per (page, head, 8 columns of K | V, token), tokens first: a warp writes whole core matrices
__global__ void __launch_bounds__(256) expand_store_kernel(ExpandParams p, int vec) {
  pdl_trigger();
  pdl_wait();
  const int dp = up16(p.dim + p.rot), vp = up16(p.vdim), per = (dp + vp) / 8, rp = up16(p.rank), D = rp + up16(p.rot), be = 16 * (dp + vp);
  const long long total = (long long)p.n * p.heads * per * 16;
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < total; i += (long long)gridDim.x * 256) {
    const int t8 = (int)(i & 7), c = (int)(i / 8 % per), t = (int)(i / (8LL * per) & 1) * 8 + t8, h = (int)(i / (16LL * per) % p.heads),
              pg = (int)(i / (16LL * per * p.heads));
    const bool val = c * 8 >= dp;
    const int j = val ? c * 8 - dp : c * 8;
    const __nv_bfloat16* row = p.kv + ((size_t)pg * 16 + t) * p.ld;
    const __nv_bfloat16* lat = p.pool + (size_t)p.pages[pg] * p.page_stride;
    const __nv_bfloat16* src = val ? row + (size_t)p.heads * p.dim + (size_t)h * p.vdim + j : row + (size_t)h * p.dim + j;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (vec) {
      if (val ? j < p.vdim : j < p.dim) u = *reinterpret_cast<const uint4*>(src);
      else if (!val && j < p.dim + p.rot) u = *reinterpret_cast<const uint4*>(lat + core_off(t, rp + j - p.dim, D));
    } else {
      __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&u);
      for (int k = 0; k < 8; ++k) {
        const int jj = j + k;
        if (val ? jj < p.vdim : jj < p.dim) e[k] = src[k];
        else if (!val && jj < p.dim + p.rot) e[k] = lat[core_off(t, rp + jj - p.dim, D)];
      }
    }
    *reinterpret_cast<uint4*>(p.out + ((size_t)pg * p.heads + h) * be + (val ? 16 * dp : 0) + core_off(t, j, val ? vp : dp)) = u;
  }
}

static bool aligned16(const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; }
static unsigned blocks_of(long long units) { return (unsigned)(units < 65536 ? (units > 0 ? units : 1) : 65536); }

}  // namespace blz

// Normed latents of the T rows of proj (element offsets q_off, kv_off): the queries' to q_lat [T, q_rank], the keys' with their rotated
// part to the page slots (-1: skip; pool null: queries only).  f32: everything is fp32, else bf16.
BLZ_API int blz_latent_prep(const void* proj, long long ld, long long q_off, long long kv_off, void* q_lat, void* pool, long long page_stride,
                            const float* q_norm, const float* c_norm, const float* freq, const int* positions, const int* slot_mapping, int T,
                            int q_rank, int rank, int rot, int rot_dims, float eps, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || q_rank < 1 || rank < 1 || rot < 1 || rot_dims < 0 || rot_dims > rot || rot_dims % 2 || (rot_dims && !freq))
    return (int)cudaErrorInvalidValue;
  const LatentPrepParams p = {proj, q_lat, pool, q_norm, c_norm, freq, positions, slot_mapping, ld, q_off, kv_off, page_stride, q_rank, rank,
                              rot, rot_dims, eps};
  const dim3 grid(T, pool ? 2 : 1);
  if (f32) return (int)launch_pdl(latent_prep_kernel<float, 1>, grid, dim3(128), 0, s, p);
  auto ok = [](const void* q) { return !q || (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (ok(proj) && ok(q_lat) && ok(pool) && ok(q_norm) && ok(c_norm) && (ld | q_off | kv_off | (long long)q_rank | (long long)rank | page_stride) % 8 == 0)
    return (int)launch_pdl(latent_prep_kernel<__nv_bfloat16, 8>, grid, dim3(128), 0, s, p);
  return (int)launch_pdl(latent_prep_kernel<__nv_bfloat16, 1>, grid, dim3(128), 0, s, p);
}

// Rotation in place of the queries q [T, heads, dim + rot] of sequences with more than max_tokens new tokens.
BLZ_API int blz_latent_rot(void* q, const float* freq, const int* positions, const int* seq_of_row, const int* q_start, int T, int heads, int dim,
                           int rot, int rot_dims, int max_tokens, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || heads < 1 || dim < 1 || rot < 1 || rot_dims < 2 || rot_dims > rot || rot_dims % 2 || rot_dims > 4096 || !freq)
    return (int)cudaErrorInvalidValue;
  const LatentRotParams p = {q, nullptr, freq, positions, {seq_of_row, q_start, max_tokens}, heads, dim, rot, rot_dims, 0};
  const size_t sm = rot_dims * sizeof(float);
  if (f32) return (int)launch_pdl(latent_rot_kernel<float>, dim3(T), dim3(128), sm, s, p);
  return (int)launch_pdl(latent_rot_kernel<__nv_bfloat16>, dim3(T), dim3(128), sm, s, p);
}

static int run_head_gemm(blz::HeadGemmParams p, int heads, int f32, cudaStream_t s) {
  using namespace blz;
  if (p.M <= 0 || p.N < 1 || p.K < 1 || heads < 1 || heads > 65535 || (p.M + 63) / 64 > 65535) return (int)cudaErrorInvalidValue;
  const dim3 grid((p.N + 63) / 64 + (p.rot.q_eff ? 1 : 0), (p.M + 63) / 64, heads);
  if (f32) return (int)launch_pdl(head_gemm_f32_kernel, grid, dim3(256), 0, s, p);
  const int vec = aligned16(p.a) && aligned16(p.b) && (reinterpret_cast<uintptr_t>(p.c) & 3) == 0 && (p.lda | p.sa | (long long)p.K) % 8 == 0 &&
                  (p.ldc | p.sc | (long long)p.N) % 2 == 0;
  const int tiles = (p.K + 63) / 64, sm = (tiles < kHgStages ? tiles : kHgStages) * 128 * kHgPitch * 2;
  static PerDeviceOnce once;
  const cudaError_t e = once.smem_limit(head_gemm_kernel, kHgStages * 128 * kHgPitch * 2);
  if (e != cudaSuccess) return (int)e;
  return (int)launch_pdl(head_gemm_kernel, grid, dim3(128), sm, s, p, vec);
}

// C[m, h, :N] = A[m, h, :K] B[h]^T, B [heads][N][K], for the rows of sequences with at most max_tokens new tokens; strides in elements.
BLZ_API int blz_head_gemm(const void* a, long long lda, long long sa, const void* b, void* c, long long ldc, long long sc, int M, int N, int K,
                          int heads, const int* seq_of_row, const int* q_start, int max_tokens, int f32, cudaStream_t s) {
  const blz::HeadGemmParams p = {a, b, c, lda, sa, ldc, sc, M, N, K, {seq_of_row, q_start, max_tokens}, {}};
  return run_head_gemm(p, heads, f32, s);
}

// Queries q [T, heads, dim + rot] of the same rows mapped to the latents: q_eff [T, heads, D] = [map_h q_nope (rank) | rotated part], both
// padded to 16 columns with zeros; map [heads][rank][dim].
BLZ_API int blz_latent_map(void* q, const void* map, void* q_eff, const float* freq, const int* positions, int T, int heads, int dim, int rot,
                           int rot_dims, int rank, const int* seq_of_row, const int* q_start, int max_tokens, int f32, cudaStream_t s) {
  using namespace blz;
  if (rot < 1 || rot_dims < 0 || rot_dims > rot || rot_dims % 2 || (rot_dims && !freq) || !q_eff) return (int)cudaErrorInvalidValue;
  const long long D = up16(rank) + up16(rot);
  const RowFilter rows = {seq_of_row, q_start, max_tokens};
  const HeadGemmParams p = {q, map, q_eff, (long long)heads * (dim + rot), dim + rot, heads * D, D, T, rank, dim, rows,
                            {q, q_eff, freq, positions, rows, heads, dim, rot, rot_dims, rank}};
  return run_head_gemm(p, heads, f32, s);
}

// Query rows per CTA of blz_latent_rows for sequences of up to `rows` (new tokens x heads) rows; 0: not these sizes.  *per_sm (may be
// null): how many CTAs share an SM.
BLZ_API int blz_latent_rows_block(int rank, int rot, int rows, int* per_sm) {
  using namespace blz;
  const int D = up16(rank) + up16(rot), nvb = (rank + 127) / 128;
  int R = rows > 32 ? 64 : rows > 16 ? 32 : 16;
  while (R >= 16 && ((2 + 2 * nvb) * R > 512 || rows_smem(R, D, R > 16 ? 2 : 1) > kLrSmem)) R /= 2;
  if (R < 16) R = 0;
  if (per_sm) *per_sm = R && R <= 32 && rows_smem(R, D, 1) <= kLrSmemHalf ? 2 : 1;
  return R;
}

// Attention of q [T, heads, D] over latent pages, bf16, sequences with at most max_tokens new tokens (the longest has `longest`): out
// [T, heads, rank], the weighted sums of the latents.  R from blz_latent_rows_block, row_blocks * R >= longest * heads; splits > 1:
// part_o [B * row_blocks * splits * R][rank], part_ml [..][2] fp32.
BLZ_API int blz_latent_rows(const void* q, void* out, const void* pool, long long page_stride, const int* block_table, int bt_stride,
                            const int* slots, const int* q_start, const int* ctx_len, const float* sink, int B, int heads, int rank, int rot,
                            int window, float scale, int max_tokens, int longest, int R, int row_blocks, int splits, float* part_o,
                            float* part_ml, cudaStream_t s) {
  using namespace blz;
  if (B < 1 || B > 65535 || heads < 1 || rank < 1 || rot < 1 || window < 0 || longest < 1 || longest > max_tokens || splits < 1 ||
      (long long)row_blocks * R < (long long)longest * heads || (splits > 1 && (!part_o || !part_ml)) || page_stride % 8 || !aligned16(pool) ||
      !aligned16(q))
    return (int)cudaErrorInvalidValue;
  LatentRowsParams p = {q, out, pool, sink, block_table, slots, q_start, ctx_len, part_o, part_ml, page_stride, bt_stride, heads, rank,
                        up16(rank) + up16(rot), window, max_tokens, row_blocks, splits, 1, scale, status_word()};
  switch (R) {
    case 16: return launch_rows<16>(p, B, longest, s);
    case 32: return launch_rows<32>(p, B, longest, s);
    case 64: return launch_rows<64>(p, B, longest, s);
  }
  return (int)cudaErrorInvalidValue;
}

// Latents of the n listed pages as rows [n * 16, rank], bf16.
BLZ_API int blz_latent_gather(const void* pool, long long page_stride, const int* pages, int n, void* out, int rank, int rot, cudaStream_t s) {
  using namespace blz;
  if (n < 1 || rank < 1 || rot < 1 || page_stride % 8 || !aligned16(pool) || !aligned16(out)) return (int)cudaErrorInvalidValue;
  return (int)launch_pdl(latent_gather_kernel, dim3(blocks_of(((long long)n * 16 * ((rank + 7) / 8) + 255) / 256)), dim3(256), 0, s,
                         (const __nv_bfloat16*)pool, page_stride, pages, n, (__nv_bfloat16*)out, rank, up16(rank) + up16(rot));
}

// Keys [dim | rotated part] and values by head of the n listed pages, from kv [n * 16, ld] (keys [heads][dim] | values [heads][vdim]), as
// page blocks out [n][heads][16 * (up16(dim + rot) + up16(vdim))], bf16.
BLZ_API int blz_expand_store(const void* kv, long long ld, const void* pool, long long page_stride, const int* pages, void* out, int n, int heads,
                             int dim, int rot, int vdim, int rank, cudaStream_t s) {
  using namespace blz;
  if (n < 1 || heads < 1 || dim < 1 || rot < 1 || vdim < 1 || rank < 1 || !aligned16(out)) return (int)cudaErrorInvalidValue;
  const ExpandParams p = {(const __nv_bfloat16*)kv, (const __nv_bfloat16*)pool, (__nv_bfloat16*)out, pages, ld, page_stride, n, heads, dim, rot,
                          vdim, rank};
  const int vec = aligned16(kv) && aligned16(pool) && (ld | dim | rot | vdim) % 8 == 0 && page_stride % 8 == 0;
  const long long total = (long long)n * heads * ((up16(dim + rot) + up16(vdim)) / 8) * 16;
  return (int)launch_pdl(expand_store_kernel, dim3(blocks_of((total + 255) / 256)), dim3(256), 0, s, p, vec);
}
