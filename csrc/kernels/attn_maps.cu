// Softmax attention of one or two maps per head (attn_maps.cuh) over paged bf16 / fp32 keys and values: the page write, a plain
// kernel for any size and for fp32, the same with sigmoid weights, and the short-row kernel (decode, verify rows, short prompt portions).  Long prompt portions
// are attn_maps_tc.cu's.
//
// Short rows: a CTA takes 16 query rows (new tokens x group) of one key/value head and a range of pages; its four warps take
// pages in turn, each with a ring of page blocks of its own that one lane keeps filled with bulk copies, and each with the
// online softmax of its maps in registers, so that two maps share every value byte.  The products are warp-level MMAs on the
// page blocks as they lie in memory (one 8 x 16-byte core matrix is one ldmatrix row set): with 16 rows per key the kernel is
// bound by the bytes of the window, not by the tensor pipe.  Scores, weights and sums are fp32; a weight enters the value
// product as the sum of two bf16 numbers, so it is not rounded to 8 bits on the way.  The warps' partial results meet in
// shared memory, those of split key ranges in a workspace.
#include "blaze/attn_maps.cuh"
#include "blaze/attn.cuh"
#include "blaze/host.h"

namespace blz {

// ------------------------------------------------------------------------------------------ page write
// one thread per (row, key/value head, 8 columns of K map 1 | K map 2 | V)
template <typename T>
__global__ void __launch_bounds__(256) maps_store_kernel(MapsParams p, int vec) {
  pdl_trigger();
  pdl_wait();
  const int dp = p.dp(), vp = p.vp(), per = (p.maps * dp + vp) / 8;
  const long long n = (long long)p.T * p.kv_heads * per;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const int c = (int)(i % per);
    const int g = (int)(i / per % p.kv_heads), t = (int)(i / ((long long)per * p.kv_heads));
    const int slot = p.slot_mapping[t];
    if (slot < 0) continue;
    const int part = min(c * 8 / dp, p.maps);                  // a map's keys, or (maps) the values
    const bool val = part == p.maps;
    const int j = c * 8 - part * dp, D = val ? vp : dp, live = (val ? p.vdim : p.dim) - j;               // columns from j on
    const T* src = reinterpret_cast<const T*>(p.kv) + (size_t)t * p.ld +
                   (val ? (size_t)p.kv_heads * p.maps * p.dim + (size_t)g * p.vdim : (size_t)(g * p.maps + part) * p.dim) + j;
    T* dst = reinterpret_cast<T*>(p.pool) + (size_t)(slot >> 4) * p.page_stride + (size_t)g * p.head_stride + part * 16 * dp +
             core_off(slot & 15, j, D);
    if (vec && live >= 8) {
#pragma unroll
      for (int k = 0; k < (int)sizeof(T) / 2; ++k) reinterpret_cast<uint4*>(dst)[k] = reinterpret_cast<const uint4*>(src)[k];
    } else {
#pragma unroll
      for (int k = 0; k < 8; ++k) ad_st(dst + k, k < live ? ad_ld(src + k) : 0.f);
    }
  }
}

// ------------------------------------------------------------------------------------------ any size, either type
// One CTA (128 threads) per (row, head): 128 keys at a time, a key per thread for the scores, value columns over the threads.
template <typename T, int MAPS, bool SIG = false>
__global__ void __launch_bounds__(128) maps_plain_kernel(MapsParams p) {
  constexpr int VC = 8;                                // value columns per thread: vdim <= 128 * VC
  extern __shared__ float sh[];
  float* s_q = sh;                                     // [MAPS][dim]
  float* s_p = s_q + MAPS * p.dim;                     // [MAPS][128]
  __shared__ float red[MAPS][4];
  __shared__ int s_page[8];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = p.seq_of_row[t];
  if (b < 0) return;
  const int g = h / p.group(), dp = p.dp(), vp = p.shared_kv ? dp : p.vp(), v_at = p.shared_kv ? 0 : MAPS * 16 * dp;
  const int pos = p.ctx_len[b] - (p.q_start[b + 1] - t);
  const int lo = first_key(pos, p.window);
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)t * p.ld + (size_t)h * MAPS * p.dim;
  for (int i = tid; i < MAPS * p.dim; i += 128) s_q[i] = ad_ld(q + i);
  const int* bt = p.block_table + (size_t)p.slots[b] * p.bt_stride;
  const T* pool = reinterpret_cast<const T*>(p.pool) + (size_t)g * p.head_stride;
  float acc[MAPS][VC] = {}, m[MAPS], l[MAPS];
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) { m[mp] = -INFINITY; l[mp] = 0.f; }
  for (int k0 = lo & ~15; k0 <= pos; k0 += 128) {
    __syncthreads();
    if (tid < 8) s_page[tid] = k0 + tid * 16 <= pos ? bt[(k0 >> 4) + tid] : 0;
    __syncthreads();
    const int key = k0 + tid;
    float s[MAPS];
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) s[mp] = -INFINITY;
    if (key >= lo && key <= pos) {
      const T* blk = pool + (size_t)s_page[tid >> 4] * p.page_stride;
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp) {
        const T* kr = blk + mp * 16 * dp;
        float d = 0.f;
        for (int j = 0; j < p.dim; ++j) d = fmaf(s_q[mp * p.dim + j], ad_ld(kr + core_off(key & 15, j, dp)), d);
        s[mp] = d * p.scale;
        if constexpr (SIG) s[mp] += p.bias[(size_t)h * p.bias_len() + kBiasPad + min(pos - key, p.reach - 1)];
      }
    }
    if constexpr (SIG) {
      s_p[tid] = s[0] == -INFINITY ? 0.f : 1.f / (1.f + expf(-s[0]));
    } else {
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp) {
        const float v = warp_max(s[mp]);
        if (lane == 0) red[mp][warp] = v;
      }
      __syncthreads();
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp) {
        const float mt = fmaxf(fmaxf(red[mp][0], red[mp][1]), fmaxf(red[mp][2], red[mp][3]));
        const float mn = fmaxf(m[mp], mt);
        const float f = m[mp] == -INFINITY ? 0.f : expf(m[mp] - mn);
        const float w = s[mp] == -INFINITY ? 0.f : expf(s[mp] - mn);
        s_p[mp * 128 + tid] = w;
        l[mp] = l[mp] * f + w;                           // this thread's share of the sum
        m[mp] = mn;
#pragma unroll
        for (int c = 0; c < VC; ++c) acc[mp][c] *= f;
      }
    }
    __syncthreads();
    const int k_end = min(128, pos - k0 + 1);
    for (int kk = max(lo - k0, 0); kk < k_end; ++kk) {
      const T* vr = pool + (size_t)s_page[kk >> 4] * p.page_stride + v_at;
#pragma unroll
      for (int c = 0; c < VC; ++c) {
        const int e = tid + c * 128;
        if (e < p.vdim) {
          const float v = ad_ld(vr + core_off(kk & 15, e, vp));
#pragma unroll
          for (int mp = 0; mp < MAPS; ++mp) acc[mp][c] = fmaf(s_p[mp * 128 + kk], v, acc[mp][c]);
        }
      }
    }
  }
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)h * p.vdim;
  if constexpr (SIG) {
#pragma unroll
    for (int c = 0; c < VC; ++c)
      if (tid + c * 128 < p.vdim) ad_st(out + tid + c * 128, acc[0][c] * gate_factor<T>(p, t, h, tid + c * 128));
    return;
  }
  __syncthreads();
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
    const float v = warp_sum(l[mp]);
    if (lane == 0) red[mp][warp] = v;
  }
  __syncthreads();
  const float l0 = red[0][0] + red[0][1] + red[0][2] + red[0][3];
  if constexpr (MAPS == 1) {
    const float sink = p.sink ? p.sink[h] : -INFINITY, mx = fmaxf(m[0], sink), f = expf(m[0] - mx);
    const float inv = f / (l0 * f + (p.sink ? expf(sink - mx) : 0.f));
#pragma unroll
    for (int c = 0; c < VC; ++c)
      if (tid + c * 128 < p.vdim) ad_st(out + tid + c * 128, acc[0][c] * inv * gate_factor<T>(p, t, h, tid + c * 128));
  } else {
    const float l1 = red[1][0] + red[1][1] + red[1][2] + red[1][3];
    float o[VC], ss = 0.f;
#pragma unroll
    for (int c = 0; c < VC; ++c) {
      o[c] = acc[0][c] / l0 - p.lam * (acc[1][c] / l1);
      if (tid + c * 128 < p.vdim) ss = fmaf(o[c], o[c], ss);
    }
    __syncthreads();
    ss = warp_sum(ss);
    if (lane == 0) red[0][warp] = ss;
    __syncthreads();
    const float f = p.post / sqrtf((red[0][0] + red[0][1] + red[0][2] + red[0][3]) / (float)p.vdim + p.eps);
#pragma unroll
    for (int c = 0; c < VC; ++c)
      if (tid + c * 128 < p.vdim) ad_st(out + tid + c * 128, o[c] * f);
  }
}

// ------------------------------------------------------------------------------------------ short rows
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two weights as bf16 pairs (value and remainder): their sum is the weight to about 2^-17
__device__ __forceinline__ void split_bf16x2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16x2(a - __low2float(h), b - __high2float(h));
}

static constexpr int kShortWarps = 4;
static constexpr float kLazy = 8.f;      // log2 of how far a row's weights may outgrow its running maximum before a rescale

// what a CTA's finished rows become: the head's output (one key range) or an entry of the workspace.
// 8 threads per row; o holds this thread's columns, relative to the maxima m (log2), with sums l.
template <int MAPS, int VP, bool SIG>
__device__ __forceinline__ void finish_rows(const MapsParams& p, float (&o)[MAPS][VP / 8], const float (&m)[MAPS], const float (&l)[MAPS],
                                            int row_t, int head, int sub) {
  float f;
  if constexpr (MAPS == 1) {
    if (row_t < 0) return;
    f = SIG ? 1.f : 1.f / (l[0] + (p.sink ? ex2(p.sink[head] * kLog2e - m[0]) : 0.f));
  } else {
    const float i0 = 1.f / l[0], i1 = p.lam / l[1];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VP / 8; ++k) {
      o[0][k] = o[0][k] * i0 - o[1][k] * i1;
      if (sub + 8 * k < p.vdim) ss = fmaf(o[0][k], o[0][k], ss);
    }
#pragma unroll
    for (int s = 1; s < 8; s <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    f = p.post / sqrtf(ss / (float)p.vdim + p.eps);
    if (row_t < 0) return;
  }
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)row_t * p.ld_out + (size_t)head * p.vdim;
#pragma unroll
  for (int k = 0; k < VP / 8; ++k) {
    const int e = sub + 8 * k;
    if (e < p.vdim) out[e] = __float2bfloat16(o[0][k] * f * (MAPS == 1 ? gate_factor<__nv_bfloat16>(p, row_t, head, e) : 1.f));
  }
}

template <int MAPS, int VP, bool SIG>
__global__ void __launch_bounds__(kShortWarps * 32) maps_short_kernel(MapsParams p) {
  extern __shared__ __align__(128) uint8_t smem_raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.z, g = blockIdx.y, rb = blockIdx.x / p.splits, split = blockIdx.x % p.splits;
  pdl_trigger();
  pdl_wait();
  const int r0 = p.q_start[b], qlen = p.q_start[b + 1] - r0, group = p.group();
  const int rows = qlen * group;
  if (rows > p.max_rows || rb * 16 >= rows) return;
  const int dp = p.dp(), vp = p.vp(), be = p.block_elems(), ST = p.stages;
  uint8_t* base = smem_raw;
  uint64_t* bars = reinterpret_cast<uint64_t*>(base);                              // [warps][ST] (at most 8 stages)
  volatile int* abort_flag = reinterpret_cast<volatile int*>(base + kShortWarps * 8 * 8);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(base + 512);                // [MAPS][16 x dp]
  __nv_bfloat16* ring = sQ + MAPS * 16 * dp;
  const int ctx = p.ctx_len[b], pos0 = ctx - qlen;
  const int tok_lo = rb * 16 / group, tok_hi = (min(rb * 16 + 16, rows) - 1) / group;
  const int pg_lo = first_key(pos0 + tok_lo, p.window) >> 4, pg_hi = (pos0 + tok_hi) >> 4;
  const int pages = pg_hi - pg_lo + 1, per = (pages + p.splits - 1) / p.splits;
  const int s_lo = pg_lo + split * per, s_n = max(min(per, pg_hi + 1 - s_lo), 0);   // this CTA's pages
  const int n = s_n > warp ? (s_n - warp + kShortWarps - 1) / kShortWarps : 0;      // this warp's: s_lo + warp + i * 4
  if (tid < kShortWarps * ST) mbar_init(&bars[tid], 1);
  if (tid == 0) { *abort_flag = 0; mbar_fence_init(); }
  // query rows, zero beyond the live ones, in the core-matrix order ldmatrix wants
  for (int i = tid; i < MAPS * 16 * (dp / 8); i += kShortWarps * 32) {
    const int c = i % (dp / 8), r = i / (dp / 8) % 16, mp = i / (dp / 8) / 16;
    const int rr = rb * 16 + r;
    __nv_bfloat16* dst = sQ + mp * 16 * dp + core_off(r, c * 8, dp);
    const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)(r0 + rr / group) * p.ld +
                               (size_t)((g * group + rr % group) * MAPS + mp) * p.dim + c * 8;
#pragma unroll
    for (int k = 0; k < 8; ++k) dst[k] = (rr < rows && c * 8 + k < p.dim) ? src[k] : __float2bfloat16(0.f);
  }
  __syncthreads();
  const int* bt = p.block_table + (size_t)p.slots[b] * p.bt_stride;
  const __nv_bfloat16* pool = reinterpret_cast<const __nv_bfloat16*>(p.pool) + (size_t)g * p.head_stride;
  __nv_bfloat16* my_ring = ring + (size_t)warp * ST * be;
  uint64_t* my_bar = bars + warp * ST;
  int pg_cache = 0;                            // lane i holds the table entry of this warp's page (issue index & ~31) + i
  int issued = 0;
  auto issue = [&]() {                         // the next page block of this warp into its ring slot (all lanes call)
    if ((issued & 31) == 0) {
      const int k = issued + lane;
      pg_cache = k < n ? bt[s_lo + warp + k * kShortWarps] : 0;
    }
    const int page = __shfl_sync(0xffffffffu, pg_cache, issued & 31);
    if (lane == 0) {
      const int st = issued % ST;
      mbar_expect_tx(&my_bar[st], be * 2);
      bulk_load(my_ring + (size_t)st * be, pool + (size_t)page * p.page_stride, be * 2, &my_bar[st]);
    }
    ++issued;
  };
  while (issued < n && issued < ST) issue();

  float o[MAPS][VP / 8][4];
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp)
#pragma unroll
    for (int i = 0; i < VP / 8; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) o[mp][i][k] = 0.f;
  float m[MAPS][2], l[MAPS][2];                      // [map][row half]
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) { m[mp][0] = m[mp][1] = -INFINITY; l[mp][0] = l[mp][1] = 0.f; }
  const float sc = p.scale * 1.4426950408889634f;
  const int row_a = rb * 16 + (lane >> 2);
  const int pos_a = row_a < rows ? pos0 + row_a / group : -1, pos_b = row_a + 8 < rows ? pos0 + (row_a + 8) / group : -1;
  const int lo_a = first_key(pos_a, p.window), lo_b = first_key(pos_b, p.window);
  // sigmoid: this thread's two rows of the bias table, and their last entries
  const float *ba = nullptr, *bb = nullptr;
  float far_a = 0.f, far_b = 0.f;
  int far_key = -1;                             // pages that end at or before it are beyond the listed distances for every row
  if constexpr (SIG) {
    ba = p.bias + (size_t)(g * group + row_a % group) * p.bias_len() + kBiasPad;
    bb = p.bias + (size_t)(g * group + (row_a + 8) % group) * p.bias_len() + kBiasPad;
    far_a = ba[p.reach - 1];
    far_b = bb[p.reach - 1];
    far_key = pos0 + tok_lo - (p.reach - 1);
  }
  const int mat = lane >> 3, mrow = lane & 7;
  const uint32_t q_addr = smem_u32(sQ) + ((mat & 1) * 8 * dp + (mat >> 1) * 64 + mrow * 8) * 2;
  bool ok = true;
  for (int i = 0; i < n; ++i) {
    const int st = i % ST;
    ok = __all_sync(0xffffffffu, mbar_wait(&my_bar[st], (uint32_t)((i / ST) & 1), abort_flag, p.status));
    if (!ok) break;
    const uint32_t blk = smem_u32(my_ring + (size_t)st * be);
    const int k0 = (s_lo + warp + i * kShortWarps) * 16;
    float s[MAPS][2][4];                          // [map][8 keys][...]
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int k = 0; k < 4; ++k) s[mp][h][k] = 0.f;
      const uint32_t ka = blk + (mp * 16 * dp + (mat >> 1) * 8 * dp + (mat & 1) * 64 + mrow * 8) * 2;
      for (int ks = 0; ks < dp / 16; ++ks) {
        uint32_t a[4], kb[4];
        ldm4(a, q_addr + (mp * 16 * dp + ks * 128) * 2);
        ldm4(kb, ka + ks * 256);
        mma16816(s[mp][0], a, kb[0], kb[1]);
        mma16816(s[mp][1], a, kb[2], kb[3]);
      }
    }
    const int key = k0 + 2 * (lane & 3);
    uint32_t hi[MAPS][4], lo[MAPS][4];
    if constexpr (SIG) {
      const bool far = k0 + 15 <= far_key && p.window == 0;
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          float t = k < 2 ? far_a : far_b;
          if (!far) {
            const int pos = k < 2 ? pos_a : pos_b, kk = key + h * 8 + (k & 1);
            const bool vis = kk <= pos && kk >= (k < 2 ? lo_a : lo_b);
            t = vis ? (k < 2 ? ba : bb)[min(pos - kk, p.reach - 1)] : INFINITY;
          }
          s[0][h][k] = sigmoid_ex2(fmaf(s[0][h][k], -sc, t));
        }
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int r = 0; r < 2; ++r) split_bf16x2(s[0][h][2 * r], s[0][h][2 * r + 1], hi[0][h * 2 + r], lo[0][h * 2 + r]);
    } else {
      float mx[MAPS][2];
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp) {
        mx[mp][0] = mx[mp][1] = -INFINITY;
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int kk = key + h * 8 + (k & 1);
            const bool vis = k < 2 ? (kk <= pos_a && kk >= lo_a) : (kk <= pos_b && kk >= lo_b);
            s[mp][h][k] = vis ? s[mp][h][k] * sc : -INFINITY;
            mx[mp][k >> 1] = fmaxf(mx[mp][k >> 1], s[mp][h][k]);
          }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          mx[mp][r] = fmaxf(mx[mp][r], __shfl_xor_sync(0xffffffffu, mx[mp][r], 1));
          mx[mp][r] = fmaxf(mx[mp][r], __shfl_xor_sync(0xffffffffu, mx[mp][r], 2));
        }
      }
      // the running maximum moves only when a row has outgrown it by 2^kLazy (or has none yet): weights stay far from overflow
      bool grow = false;
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp)
#pragma unroll
        for (int r = 0; r < 2; ++r) grow |= mx[mp][r] > m[mp][r] + kLazy || (m[mp][r] == -INFINITY && mx[mp][r] != -INFINITY);
      if (__any_sync(0xffffffffu, grow)) {
#pragma unroll
        for (int mp = 0; mp < MAPS; ++mp) {
          float f[2];
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const float mn = fmaxf(m[mp][r], mx[mp][r]);
            f[r] = m[mp][r] == -INFINITY ? 0.f : ex2(m[mp][r] - mn);
            m[mp][r] = mn;
            l[mp][r] *= f[r];
          }
#pragma unroll
          for (int c = 0; c < VP / 8; ++c) { o[mp][c][0] *= f[0]; o[mp][c][1] *= f[0]; o[mp][c][2] *= f[1]; o[mp][c][3] *= f[1]; }
        }
      }
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp) {
        float w[2][4];
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            w[h][k] = s[mp][h][k] == -INFINITY ? 0.f : ex2(s[mp][h][k] - m[mp][k >> 1]);
            l[mp][k >> 1] += w[h][k];
          }
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int r = 0; r < 2; ++r) split_bf16x2(w[h][2 * r], w[h][2 * r + 1], hi[mp][h * 2 + r], lo[mp][h * 2 + r]);
      }
    }
    const uint32_t va = blk + (MAPS * 16 * dp + (mat & 1) * 8 * vp + (mat >> 1) * 64 + mrow * 8) * 2;
#pragma unroll
    for (int c = 0; c < VP / 16; ++c) {
      if (c * 16 < vp) {
        uint32_t vb[4];
        ldm4t(vb, va + c * 256);
#pragma unroll
        for (int mp = 0; mp < MAPS; ++mp) {
          mma16816(o[mp][2 * c], hi[mp], vb[0], vb[1]);
          mma16816(o[mp][2 * c + 1], hi[mp], vb[2], vb[3]);
          mma16816(o[mp][2 * c], lo[mp], vb[0], vb[1]);
          mma16816(o[mp][2 * c + 1], lo[mp], vb[2], vb[3]);
        }
      }
    }
    __syncwarp();                              // every lane is done with the slot before it is filled again
    if (issued < n) issue();
  }
  if (!ok) {
    // let the copies in flight land before the block's shared memory can be given away
    for (int k = 0; k < ST; ++k) {
      const long long t0 = clock64();
      while (k < issued && !mbar_try_sleep(&my_bar[k], (uint32_t)(((issued - 1 - k) / ST) & 1), 20000u) && clock64() - t0 < kSpinLimit) {}
    }
  }
  // the warps' partial rows -> shared memory (over the rings, which every warp has drained)
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      l[mp][r] += __shfl_xor_sync(0xffffffffu, l[mp][r], 1);
      l[mp][r] += __shfl_xor_sync(0xffffffffu, l[mp][r], 2);
    }
  __syncthreads();
  constexpr int OP = VP + 4;                   // row pitch
  float* s_o = reinterpret_cast<float*>(ring); // [warps][MAPS][16][OP]
  float* s_ml = s_o + kShortWarps * MAPS * 16 * OP;
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
    float* dst = s_o + (size_t)((warp * MAPS + mp) * 16 + (lane >> 2)) * OP + 2 * (lane & 3);
    const bool live_a = row_a < rows, live_b = row_a + 8 < rows;
#pragma unroll
    for (int c = 0; c < VP / 8; ++c) {
      if (c * 8 < vp) {
        if (live_a) *reinterpret_cast<float2*>(dst + c * 8) = make_float2(o[mp][c][0], o[mp][c][1]);
        if (live_b) *reinterpret_cast<float2*>(dst + 8 * OP + c * 8) = make_float2(o[mp][c][2], o[mp][c][3]);
      }
    }
    if ((lane & 3) == 0) {
      float* ml = s_ml + ((warp * MAPS + mp) * 16 + (lane >> 2)) * 2;
      ml[0] = m[mp][0]; ml[1] = l[mp][0];
      ml[16] = m[mp][1]; ml[17] = l[mp][1];
    }
  }
  __syncthreads();
  const int r = tid >> 3, sub = tid & 7, rr = rb * 16 + r;
  float f[MAPS][kShortWarps], mm[MAPS], ll[MAPS];
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
    mm[mp] = -INFINITY; ll[mp] = 0.f;
#pragma unroll
    for (int w = 0; w < kShortWarps; ++w) mm[mp] = fmaxf(mm[mp], s_ml[((w * MAPS + mp) * 16 + r) * 2]);
#pragma unroll
    for (int w = 0; w < kShortWarps; ++w) {
      if constexpr (SIG) { f[mp][w] = rb * 16 + r < rows ? 1.f : 0.f; continue; }
      const float mw = s_ml[((w * MAPS + mp) * 16 + r) * 2];
      f[mp][w] = mw == -INFINITY ? 0.f : ex2(mw - mm[mp]);
      ll[mp] = fmaf(f[mp][w], s_ml[((w * MAPS + mp) * 16 + r) * 2 + 1], ll[mp]);
    }
  }
  float res[MAPS][VP / 8];
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp)
#pragma unroll
    for (int k = 0; k < VP / 8; ++k) {
      res[mp][k] = 0.f;
      if (rr < rows && sub + 8 * k < p.vdim) {
#pragma unroll
        for (int w = 0; w < kShortWarps; ++w)
          if (f[mp][w] != 0.f) res[mp][k] = fmaf(f[mp][w], s_o[(size_t)((w * MAPS + mp) * 16 + r) * OP + sub + 8 * k], res[mp][k]);
      }
    }
  if (p.splits == 1) {
    finish_rows<MAPS, VP, SIG>(p, res, mm, ll, rr < rows ? r0 + rr / group : -1, g * group + rr % group, sub);
  } else if (rr < rows) {
    const size_t w = (((size_t)b * p.kv_heads + g) * p.row_blocks + rb) * p.splits + split;
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
#pragma unroll
      for (int k = 0; k < VP / 8; ++k)
        if (sub + 8 * k < p.vdim) p.part_o[((w * MAPS + mp) * 16 + r) * VP + sub + 8 * k] = res[mp][k];
      if (sub == 0) { p.part_ml[((w * MAPS + mp) * 16 + r) * 2] = mm[mp]; p.part_ml[((w * MAPS + mp) * 16 + r) * 2 + 1] = ll[mp]; }
    }
  }
}

// joins the split key ranges of one (sequence, key/value head, 16 rows)
template <int MAPS, int VP, bool SIG>
__global__ void __launch_bounds__(128) maps_combine_kernel(MapsParams p) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, g = blockIdx.y, rb = blockIdx.x;
  const int r0 = p.q_start[b], rows = (p.q_start[b + 1] - r0) * p.group();
  if (rows > p.max_rows || rb * 16 >= rows) return;
  const int r = threadIdx.x >> 3, sub = threadIdx.x & 7, rr = rb * 16 + r;
  const size_t w0 = (((size_t)b * p.kv_heads + g) * p.row_blocks + rb) * p.splits;
  float o[MAPS][VP / 8], mx[MAPS], l[MAPS];
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
#pragma unroll
    for (int k = 0; k < VP / 8; ++k) o[mp][k] = 0.f;
    mx[mp] = 0.f;
    l[mp] = 1.f;
    if (rr >= rows) continue;
    float mm = -INFINITY;
    l[mp] = 0.f;
    for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.part_ml[(((w0 + s) * MAPS + mp) * 16 + r) * 2]);
    for (int s = 0; s < p.splits; ++s) {
      const float* ml = p.part_ml + (((w0 + s) * MAPS + mp) * 16 + r) * 2;
      if (!SIG && ml[0] == -INFINITY) continue;
      const float f = SIG ? 1.f : ex2(ml[0] - mm);
      l[mp] = fmaf(f, ml[1], l[mp]);
      const float* po = p.part_o + (((w0 + s) * MAPS + mp) * 16 + r) * VP + sub;
#pragma unroll
      for (int k = 0; k < VP / 8; ++k)
        if (sub + 8 * k < p.vdim) o[mp][k] = fmaf(f, po[8 * k], o[mp][k]);
    }
    mx[mp] = mm;
  }
  finish_rows<MAPS, VP, SIG>(p, o, mx, l, rr < rows ? r0 + rr / p.group() : -1, g * p.group() + rr % p.group(), sub);
}

static constexpr int kShortSmemTarget = 110 * 1024;      // two CTAs per SM

template <int MAPS, int VP, bool SIG = false>
static cudaError_t launch_short(MapsParams p, cudaStream_t s) {
  const int be = p.block_elems() * 2, fixed = 512 + MAPS * 16 * p.dp() * 2;
  const int merge = (kShortWarps * MAPS * 16 * (VP + 4) + kShortWarps * MAPS * 16 * 2) * 4;
  int st = (kShortSmemTarget - fixed) / (kShortWarps * be);
  st = st > 8 ? 8 : (st < 2 ? 2 : st);
  int ring = kShortWarps * st * be;
  if (ring < merge) ring = merge;
  if (fixed + ring > 227 * 1024) return cudaErrorInvalidValue;
  p.stages = st;
  auto kern = maps_short_kernel<MAPS, VP, SIG>;
  static PerDeviceOnce once;
  cudaError_t e = once.smem_limit(kern, 227 * 1024);
  if (e != cudaSuccess) return e;
  e = launch_pdl(kern, dim3(p.row_blocks * p.splits, p.kv_heads, p.B), dim3(kShortWarps * 32), fixed + ring, s, p);
  if (e != cudaSuccess || p.splits == 1) return e;
  return launch_pdl(maps_combine_kernel<MAPS, VP, SIG>, dim3(p.row_blocks, p.kv_heads, p.B), dim3(128), 0, s, p);
}

static cudaError_t check_maps(const MapsParams& p, int esz) {
  if (p.T <= 0 || p.B <= 0 || p.heads < 1 || p.kv_heads < 1 || p.heads % p.kv_heads || p.dim < 1 || p.vdim < 1 || p.window < 0)
    return cudaErrorInvalidValue;
  if ((p.page_stride * esz) % 16 || (p.head_stride * esz) % 16 || (reinterpret_cast<uintptr_t>(p.pool) & 15)) return cudaErrorInvalidValue;
  return cudaSuccess;
}

static int run_plain(const MapsParams& p, int f32, cudaStream_t s) {
  if (check_maps(p, f32 ? 4 : 2) != cudaSuccess || p.vdim > 1024 || p.dim > 4096 || p.heads > 65535 || !p.seq_of_row) return (int)cudaErrorInvalidValue;
  const size_t sm = p.maps * (p.dim + 128) * sizeof(float);
  const dim3 grid(p.T, p.heads);
  if (p.bias) {
    if (p.maps != 1 || p.reach < 1) return (int)cudaErrorInvalidValue;
    if (f32) return (int)launch_pdl(maps_plain_kernel<float, 1, true>, grid, dim3(128), sm, s, p);
    return (int)launch_pdl(maps_plain_kernel<__nv_bfloat16, 1, true>, grid, dim3(128), sm, s, p);
  }
  if (p.maps == 1) {
    if (f32) return (int)launch_pdl(maps_plain_kernel<float, 1>, grid, dim3(128), sm, s, p);
    return (int)launch_pdl(maps_plain_kernel<__nv_bfloat16, 1>, grid, dim3(128), sm, s, p);
  }
  if (f32) return (int)launch_pdl(maps_plain_kernel<float, 2>, grid, dim3(128), sm, s, p);
  return (int)launch_pdl(maps_plain_kernel<__nv_bfloat16, 2>, grid, dim3(128), sm, s, p);
}

static int run_short(const MapsParams& p, cudaStream_t s) {
  if (check_maps(p, 2) != cudaSuccess || p.dim > 128 || p.vdim > 128) return (int)cudaErrorInvalidValue;
  if (p.max_rows < 1 || p.row_blocks < 1 || p.splits < 1 || p.B > 65535 || p.kv_heads > 65535 || (p.splits > 1 && (!p.part_o || !p.part_ml)))
    return (int)cudaErrorInvalidValue;
  if (p.bias) {
    if (p.maps != 1 || p.reach < 1) return (int)cudaErrorInvalidValue;
    return (int)(p.vdim <= 32 ? launch_short<1, 32, true>(p, s) : p.vdim <= 64 ? launch_short<1, 64, true>(p, s) : launch_short<1, 128, true>(p, s));
  }
#define BLZ_SHORT(M) return (int)(p.vdim <= 32 ? launch_short<M, 32>(p, s) : p.vdim <= 64 ? launch_short<M, 64>(p, s) : launch_short<M, 128>(p, s))
  if (p.maps == 1) { BLZ_SHORT(1); }
  BLZ_SHORT(2);
#undef BLZ_SHORT
}

static MapsParams diff_params(const void* qkv, long long ld, void* out, void* pool, long long page_stride, long long head_stride,
                              const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                              int T, int B, int heads, int kv_heads, int dim, int vdim, int window, float scale, float lam,
                              float post, float eps) {
  MapsParams p = {};
  p.q = qkv; p.ld = ld; p.out = out; p.ld_out = (long long)heads * vdim; p.pool = pool; p.page_stride = page_stride; p.head_stride = head_stride;
  p.block_table = block_table; p.bt_stride = bt_stride; p.slots = slots; p.q_start = q_start; p.ctx_len = ctx_len;
  p.T = T; p.B = B; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.window = window; p.maps = 2;
  p.scale = scale; p.lam = lam; p.post = post; p.eps = eps;
  p.max_rows = 0x7fffffff; p.row_blocks = p.splits = p.stages = 1;
  p.status = status_word();
  return p;
}

}  // namespace blz

// Keys and values of the T rows of qkv (q [heads][2][dim] | k [kv_heads][2][dim] | v [kv_heads][vdim]) into their page slots
// (-1: skip the row).
BLZ_API int blz_diff_store(const void* qkv, long long ld, void* pool, long long page_stride, long long head_stride,
                           const int* slot_mapping, int T, int heads, int kv_heads, int dim, int vdim, int f32, cudaStream_t s) {
  using namespace blz;
  MapsParams p = diff_params(qkv, ld, nullptr, pool, page_stride, head_stride, nullptr, 0, nullptr, nullptr, nullptr, T, 1, heads, kv_heads,
                             dim, vdim, 0, 1.f, 0.f, 1.f, 0.f);
  const int esz = f32 ? 4 : 2;
  if (check_maps(p, esz) != cudaSuccess) return (int)cudaErrorInvalidValue;
  p.slot_mapping = slot_mapping;
  p.kv = reinterpret_cast<const char*>(qkv) + (size_t)heads * 2 * dim * esz;
  const int vec = (reinterpret_cast<uintptr_t>(qkv) & 15) == 0 && ld * esz % 16 == 0 && dim * esz % 16 == 0 && vdim * esz % 16 == 0;
  const long long n = (long long)T * kv_heads * (2 * p.dp() + p.vp()) / 8;
  const dim3 grid((unsigned)((n + 255) / 256 < 65536 ? (n + 255) / 256 : 65536));
  if (f32) return (int)launch_pdl(maps_store_kernel<float>, grid, dim3(256), 0, s, p, vec);
  return (int)launch_pdl(maps_store_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, p, vec);
}

// Differential attention of any size (vdim <= 1024), fp32 or bf16, every row of the step.
BLZ_API int blz_diff_plain(const void* qkv, long long ld, void* out, void* pool, long long page_stride, long long head_stride,
                           const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                           const int* seq_of_row, int T, int B, int heads, int kv_heads, int dim, int vdim, int window, float scale,
                           float lam, float post, float eps, int f32, cudaStream_t s) {
  blz::MapsParams p = blz::diff_params(qkv, ld, out, pool, page_stride, head_stride, block_table, bt_stride, slots, q_start, ctx_len, T, B,
                                       heads, kv_heads, dim, vdim, window, scale, lam, post, eps);
  p.seq_of_row = seq_of_row;
  return blz::run_plain(p, f32, s);
}

// bf16; the sequences with at most max_rows = new tokens * group rows (row_blocks covers them: 16 rows each).  dim, vdim <= 128.
// splits > 1: part_o [B * kv_heads * row_blocks * splits][2][16][VP] and part_ml [...][2][16][2] fp32, VP = 32 / 64 / 128.
BLZ_API int blz_diff_short(const void* qkv, long long ld, void* out, void* pool, long long page_stride, long long head_stride,
                           const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len, int T, int B,
                           int heads, int kv_heads, int dim, int vdim, int window, float scale, float lam, float post, float eps,
                           int max_rows, int row_blocks, int splits, float* part_o, float* part_ml, cudaStream_t s) {
  blz::MapsParams p = blz::diff_params(qkv, ld, out, pool, page_stride, head_stride, block_table, bt_stride, slots, q_start, ctx_len, T, B,
                                       heads, kv_heads, dim, vdim, window, scale, lam, post, eps);
  p.max_rows = max_rows; p.row_blocks = row_blocks; p.splits = splits; p.part_o = part_o; p.part_ml = part_ml;
  return blz::run_short(p, s);
}

// ------------------------------------------------------------------------------------------ one map: rotation, page write
namespace blz {

struct PrepParams {
  const void* qkv;             // [T, ld]: q [heads][dim] from q_off on, k [kv_heads][dim] from k_off, v [kv_heads][vdim] from v_off
  void* q_out;                 // [T, heads * dim]
  void* pool;
  const int* positions;        // [T]
  const int* slot_mapping;     // [T], -1 = padding
  const float* freq;           // [2][rot_dims / 2]: frequencies, and what their rounding to 32 bits left over
  long long ld, q_off, k_off, v_off, page_stride, head_stride;
  int T, heads, kv_heads, dim, vdim, rot_dims, interleaved, unit_rms;
  int pairs;                   // bf16: neighbouring dimensions can be read and written as 32-bit words
  float eps;
};

static constexpr int kPrepHeads = 4;       // heads of one row that a warp turns by the same angles

// One warp per (row, up to 4 heads): rotary positions on the first rot_dims dimensions (pairs (2i, 2i + 1), or (i, i + rot_dims / 2)),
// then each q and k head divided by its root mean square (unit_rms); q to its buffer, k and v to their page.
template <typename T>
__global__ void __launch_bounds__(128) attn_prep_pages_kernel(PrepParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, units = p.heads + 2 * p.kv_heads, blocks = (units + kPrepHeads - 1) / kPrepHeads;
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int t = (int)(w / blocks), u0 = (int)(w % blocks) * kPrepHeads;
  if (t >= p.T) return;
  const int slot = p.slot_mapping[t], half = p.rot_dims / 2, dp = (p.dim + 15) / 16 * 16, vp = (p.vdim + 15) / 16 * 16;
  const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld;
  const float pos = (float)p.positions[t];
  float f[kPrepHeads];                     // 1 / rms
  const int u1 = min(u0 + kPrepHeads, units);
#pragma unroll
  for (int k = 0; k < kPrepHeads; ++k) {
    f[k] = 1.f;
    const int u = u0 + k;
    if (u < u1 && u < p.heads + p.kv_heads && p.unit_rms) {
      const T* src = row + (u < p.heads ? p.q_off + (size_t)u * p.dim : p.k_off + (size_t)(u - p.heads) * p.dim);
      float ss = 0.f;
      if (sizeof(T) == 2 && p.pairs) {
        for (int j = lane; j < p.dim / 2; j += 32) {
          const uint32_t w = *reinterpret_cast<const uint32_t*>(src + 2 * j);
          const float x = __uint_as_float(w << 16), y = __uint_as_float(w & 0xffff0000u);
          ss = fmaf(x, x, fmaf(y, y, ss));
        }
      } else {
        for (int j = lane; j < p.dim; j += 32) { const float v = ad_ld(src + j); ss = fmaf(v, v, ss); }
      }
      f[k] = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);         // a rotation leaves the sum of squares as it is
    }
  }
  T* page = slot < 0 ? nullptr : reinterpret_cast<T*>(p.pool) + (size_t)(slot >> 4) * p.page_stride;
  if (u0 < p.heads + p.kv_heads) {
    for (int i = lane; i < dp / 2; i += 32) {
      const bool turned = i < half;
      const int a = turned && !p.interleaved ? i : 2 * i, b = turned && !p.interleaved ? i + half : 2 * i + 1;
      float c = 1.f, s = 0.f;
      if (turned) {
        const float hi = p.freq[i], ang = pos * hi, rest = fmaf(pos, hi, -ang) + pos * p.freq[half + i];
        float s0, c0;
        sincosf(ang, &s0, &c0);
        c = fmaf(-rest, s0, c0);
        s = fmaf(rest, c0, s0);
      }
#pragma unroll
      for (int k = 0; k < kPrepHeads; ++k) {
        const int u = u0 + k;
        if (u >= u1 || u >= p.heads + p.kv_heads) continue;
        const bool is_q = u < p.heads;
        const T* src = row + (is_q ? p.q_off + (size_t)u * p.dim : p.k_off + (size_t)(u - p.heads) * p.dim);
        if (sizeof(T) == 2 && p.pairs && b == a + 1) {             // a pair is one 32-bit word everywhere
          const uint32_t w = a < p.dim ? *reinterpret_cast<const uint32_t*>(src + a) : 0u;
          const float x = __uint_as_float(w << 16), y = __uint_as_float(w & 0xffff0000u);
          const uint32_t r = pack_bf16x2((x * c - y * s) * f[k], (y * c + x * s) * f[k]);
          if (!is_q) {
            if (page) *reinterpret_cast<uint32_t*>(page + (size_t)(u - p.heads) * p.head_stride + core_off(slot & 15, a, dp)) = r;
          } else if (a < p.dim) {
            *reinterpret_cast<uint32_t*>(reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.heads + u) * p.dim + a) = r;
          }
          continue;
        }
        const float x = a < p.dim ? ad_ld(src + a) : 0.f, y = b < p.dim ? ad_ld(src + b) : 0.f;
        const float xr = (x * c - y * s) * f[k], yr = (y * c + x * s) * f[k];
        if (is_q) {
          T* dst = reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.heads + u) * p.dim;
          if (a < p.dim) ad_st(dst + a, xr);
          if (b < p.dim) ad_st(dst + b, yr);
        } else if (page) {
          T* dst = page + (size_t)(u - p.heads) * p.head_stride;
          ad_st(dst + core_off(slot & 15, a, dp), xr);
          ad_st(dst + core_off(slot & 15, b, dp), yr);
        }
      }
    }
  }
  if (page) {
#pragma unroll
    for (int k = 0; k < kPrepHeads; ++k) {
      const int g = u0 + k - p.heads - p.kv_heads;
      if (u0 + k >= u1 || g < 0) continue;
      const T* src = row + p.v_off + (size_t)g * p.vdim;
      T* dst = page + (size_t)g * p.head_stride + 16 * dp;
      if (sizeof(T) == 2 && p.pairs) {
        for (int j = 2 * lane; j < vp; j += 64)
          *reinterpret_cast<uint32_t*>(dst + core_off(slot & 15, j, vp)) = j < p.vdim ? *reinterpret_cast<const uint32_t*>(src + j) : 0u;
      } else {
        for (int j = lane; j < vp; j += 32) ad_st(dst + core_off(slot & 15, j, vp), j < p.vdim ? ad_ld(src + j) : 0.f);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------ convolution, value norm, page write
struct ConvPrepParams {
  PrepParams a;                // sizes, offsets, query buffer, pages
  const float* w;              // [taps][C], C = q | k | v columns
  void* state;                 // [rows][taps - 1][C]: the last projected rows of each sequence
  const int *slots, *q_start, *ctx_len, *no_store;
  int taps, unit_v, state_only;
  float temp_coef, temp_every;
};
static constexpr int kConvPrepTok = 8;     // tokens per warp, at least the taps before the current one

template <typename T, int VEC> struct alignas(sizeof(T) * VEC) PrepVec { T e[VEC]; };

// A warp per (8 tokens of a sequence, head): a causal convolution over time of each projected channel, then queries (times their position's
// temperature) to their buffer, keys and values (divided by their root mean square: unit_v) to their page.  The rows before the sequence's
// new ones come from its state, which only the first 8 tokens' warp of a channel reads, and then writes.  TAPS: the real ones rounded up.
// ONCE: one turn of the warp takes a whole head (dim and vdim up to 32 * VEC), whose rows then stay in registers.
template <typename T, int TAPS, int VEC, bool ONCE>
__global__ void __launch_bounds__(128) conv_prep_pages_kernel(ConvPrepParams q) {
  pdl_trigger();
  pdl_wait();
  constexpr int IN = TAPS - 1 + kConvPrepTok;          // rows that the block's tokens need
  using Vec = PrepVec<T, VEC>;
  const PrepParams& p = q.a;
  const int lane = threadIdx.x & 31, u = blockIdx.y * 4 + (threadIdx.x >> 5), b = blockIdx.z, t0 = blockIdx.x * kConvPrepTok;
  const int r0 = q.q_start[b], n = q.q_start[b + 1] - r0;
  if (u >= p.heads + 2 * p.kv_heads || t0 >= n) return;
  const bool fresh = q.ctx_len[b] == n;
  const bool is_q = u < p.heads, is_v = u >= p.heads + p.kv_heads;
  const int D = is_v ? p.vdim : p.dim, g = is_v ? u - p.heads - p.kv_heads : u - p.heads, taps = q.taps, m = min(kConvPrepTok, n - t0);
  const int C = p.heads * p.dim + p.kv_heads * (p.dim + p.vdim);
  const int ch = is_q ? u * p.dim : is_v ? p.heads * p.dim + p.kv_heads * p.dim + g * p.vdim : p.heads * p.dim + g * p.dim;     // first channel
  const T* src = reinterpret_cast<const T*>(p.qkv) + (size_t)(r0 + t0) * p.ld + (is_q ? p.q_off + (size_t)u * p.dim
                                                                               : is_v ? p.v_off + (size_t)g * p.vdim : p.k_off + (size_t)g * p.dim);
  T* st = reinterpret_cast<T*>(q.state) + (size_t)q.slots[b] * (taps - 1) * C + ch;
  const int dp = (p.dim + 15) / 16 * 16, vp = (p.vdim + 15) / 16 * 16;
  // lane k has token k's slot, and its query's factor
  int my_slot = -1;
  float my_f = 1.f;
  if (lane < m && !q.state_only) {
    if (!is_q) my_slot = p.slot_mapping[r0 + t0 + lane];
    else if (q.temp_coef != 0.f)
      my_f = fmaf(q.temp_coef, logf(floorf(__fdiv_rn((float)(p.positions[r0 + t0 + lane] + 1), q.temp_every)) + 1.f), 1.f);
  }
  // projected columns c.. of the block's row i - (TAPS - 1): a new token's, one before the run's first (from the state), or none
  auto input = [&](int i, int c) {
    Vec v;
    const int k = i - (TAPS - 1);
    if (t0 + k >= 0) {
      v = *reinterpret_cast<const Vec*>(src + (long long)k * p.ld + c);
    } else if (!fresh && k > -taps) {
      v = *reinterpret_cast<const Vec*>(st + (size_t)(taps - 1 + k) * C + c);
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) ad_st(v.e + j, 0.f);
    }
    return v;
  };
  auto weights = [&](int c, float (&w)[TAPS][VEC]) {
#pragma unroll
    for (int i = 0; i < TAPS; ++i) {
      const int r = i - (TAPS - taps);
#pragma unroll
      for (int j = 0; j < VEC; ++j) w[i][j] = 0.f;
      if (r < 0) continue;
      const PrepVec<float, VEC> f = *reinterpret_cast<const PrepVec<float, VEC>*>(q.w + (size_t)r * C + ch + c);
#pragma unroll
      for (int j = 0; j < VEC; ++j) w[i][j] = f.e[j];
    }
  };
  auto put = [&](int k, int c, const float (&y)[VEC], float f, int slot) {
    T* dst;
    if (is_q) {
      dst = reinterpret_cast<T*>(p.q_out) + ((size_t)(r0 + t0 + k) * p.heads + u) * p.dim + c;
    } else {
      if (slot < 0) return;
      dst = reinterpret_cast<T*>(p.pool) + (size_t)(slot >> 4) * p.page_stride + (size_t)g * p.head_stride +
            (is_v ? 16 * dp + core_off(slot & 15, c, vp) : core_off(slot & 15, c, dp));
    }
    Vec o;
#pragma unroll
    for (int j = 0; j < VEC; ++j) ad_st(o.e + j, y[j] * f);
    *reinterpret_cast<Vec*>(dst) = o;
  };
  const bool advance = t0 == 0 && taps > 1 && !(q.no_store != nullptr && q.no_store[b]);
  if constexpr (ONCE) {
    const int c = lane * VEC;
    const bool live = c < D;
    Vec in[IN];                                        // as they are: all reads go out before the first is used
    float w[TAPS][VEC], x[IN][VEC];
    const int cc = live ? c : 0;
    if (t0 >= TAPS - 1 && m == kConvPrepTok) {         // every row is a new token's
      const T* at = src - (TAPS - 1) * p.ld + cc;
#pragma unroll
      for (int i = 0; i < IN; ++i, at += p.ld) in[i] = *reinterpret_cast<const Vec*>(at);
    } else {
#pragma unroll
      for (int i = 0; i < IN; ++i) in[i] = input(min(i, TAPS - 2 + m), cc);
    }
    if (!q.state_only) weights(cc, w);
#pragma unroll
    for (int i = 0; i < IN; ++i)
#pragma unroll
      for (int j = 0; j < VEC; ++j) x[i][j] = ad_ld(in[i].e + j);
    // where this lane's columns of the tokens go: a row of the query buffer, or a place in the page that a token's slot adds to
    T* base = is_q ? reinterpret_cast<T*>(p.q_out) + ((size_t)(r0 + t0) * p.heads + u) * p.dim + cc
                   : reinterpret_cast<T*>(p.pool) + (size_t)g * p.head_stride + (is_v ? 16 * dp : 0) + (cc >> 3) * 64 + (cc & 7);
    const long long row = is_q ? (long long)p.heads * p.dim : 0;
    // lane k: offset of token k's slot (-1: none)
    const int pad8 = 8 * (is_v ? vp : dp);
    const long long my_at = is_q ? (long long)lane * row : my_slot < 0 ? -1 : (my_slot >> 4) * p.page_stride + (my_slot >> 3 & 1) * pad8 + (my_slot & 7) * 8;
#pragma unroll
    for (int k = 0; k < kConvPrepTok; ++k) {
      if (k >= m || q.state_only) break;
      float y[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        y[j] = w[0][j] * x[k][j];
#pragma unroll
        for (int i = 1; i < TAPS; ++i) y[j] = fmaf(w[i][j], x[k + i][j], y[j]);
      }
      float f = __shfl_sync(0xffffffffu, my_f, k);
      if (is_v && q.unit_v) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss = fmaf(y[j], y[j], ss);
        f = 1.f / sqrtf(warp_sum(live ? ss : 0.f) / (float)D + p.eps);
      }
      const long long at = __shfl_sync(0xffffffffu, my_at, k);
      if (live && at >= 0) {
        Vec o;
        if constexpr (VEC == 4 && sizeof(T) == 2) {
          reinterpret_cast<uint2&>(o) = make_uint2(pack_bf16x2(y[0] * f, y[1 % VEC] * f), pack_bf16x2(y[2 % VEC] * f, y[3 % VEC] * f));
        } else {
#pragma unroll
          for (int j = 0; j < VEC; ++j) ad_st(o.e + j, y[j] * f);
        }
        *reinterpret_cast<Vec*>(base + at) = o;
      }
    }
    if (!advance || !live) return;
    // the state after the run, entry i the row taps - 1 - i before the next token; entries of a short run move up
    if (n <= kConvPrepTok) {
#pragma unroll
      for (int k = 0; k < IN; ++k) {
        const int i = k - (TAPS - 1) - n + taps - 1;
        if (i >= 0 && i < taps - 1) *reinterpret_cast<Vec*>(st + (size_t)i * C + c) = in[k];
      }
    } else {
      for (int i = 0; i < taps - 1; ++i)
        *reinterpret_cast<Vec*>(st + (size_t)i * C + c) = *reinterpret_cast<const Vec*>(src + (size_t)(n - (taps - 1) + i) * p.ld + c);
    }
  } else {
    auto conv = [&](int k, int c, float (&y)[VEC]) {
      float w[TAPS][VEC];
      weights(c, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) y[j] = 0.f;
#pragma unroll
      for (int i = 0; i < TAPS; ++i) {
        const Vec v = input(k + i, c);
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] = fmaf(w[i][j], ad_ld(v.e + j), y[j]);
      }
    };
    for (int k = 0; k < m && !q.state_only; ++k) {
      float f = __shfl_sync(0xffffffffu, my_f, k), y[VEC];
      const int slot = __shfl_sync(0xffffffffu, my_slot, k);
      if (is_v && q.unit_v) {
        float ss = 0.f;
        for (int c = lane * VEC; c < D; c += 32 * VEC) {
          conv(k, c, y);
#pragma unroll
          for (int j = 0; j < VEC; ++j) ss = fmaf(y[j], y[j], ss);
        }
        f = 1.f / sqrtf(warp_sum(ss) / (float)D + p.eps);
      }
      for (int c = lane * VEC; c < D; c += 32 * VEC) {
        conv(k, c, y);
        put(k, c, y, f, slot);
      }
    }
    if (!advance) return;
    for (int c = lane * VEC; c < D; c += 32 * VEC)
      for (int i = 0; i < taps - 1; ++i)               // ascending: an entry is read before it is written over
        *reinterpret_cast<Vec*>(st + (size_t)i * C + c) = input(TAPS - 1 + n - (taps - 1) + i, c);
  }
}

template <typename T, int TAPS>
static int launch_conv_prep(const ConvPrepParams& q, bool vec, int B, int max_q, cudaStream_t s) {
  const PrepParams& p = q.a;
  const dim3 grid((max_q + kConvPrepTok - 1) / kConvPrepTok, (p.heads + 2 * p.kv_heads + 3) / 4, B);
  const int D = p.dim > p.vdim ? p.dim : p.vdim;
  if (vec && D <= 128) return (int)launch_pdl(conv_prep_pages_kernel<T, TAPS, 4, true>, grid, dim3(128), 0, s, q);
  if (vec) return (int)launch_pdl(conv_prep_pages_kernel<T, TAPS, 4, false>, grid, dim3(128), 0, s, q);
  return (int)launch_pdl(conv_prep_pages_kernel<T, TAPS, 1, false>, grid, dim3(128), 0, s, q);
}

static MapsParams soft_params(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, long long head_stride,
                              const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                              const float* sink, const void* gate, long long ld_gate, int T, int B, int heads, int kv_heads, int dim,
                              int vdim, int window, float scale, float post) {
  MapsParams p = diff_params(q, ld, out, pool, page_stride, head_stride, block_table, bt_stride, slots, q_start, ctx_len, T, B, heads,
                             kv_heads, dim, vdim, window, scale, 0.f, post, 0.f);
  p.maps = 1; p.ld_out = ld_out; p.sink = sink; p.gate = gate; p.ld_gate = ld_gate;
  return p;
}

}  // namespace blz

// q, k and v of the T rows (element offsets into a row of qkv): rotary positions on the first rot_dims dimensions of q and k,
// their root mean square divided out (unit_rms), q to q_out [T, heads * dim], k and v to their page slots (-1: skip).
BLZ_API int blz_attn_prep_pages(const void* qkv, long long ld, long long q_off, long long k_off, long long v_off, void* q_out, void* pool,
                                long long page_stride, long long head_stride, const int* positions, const int* slot_mapping,
                                const float* freq, int T, int heads, int kv_heads, int dim, int vdim, int rot_dims, int interleaved,
                                int unit_rms, float eps, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || heads < 1 || kv_heads < 1 || dim < 1 || vdim < 1 || rot_dims < 0 || rot_dims > dim || rot_dims % 2 || (rot_dims && !freq))
    return (int)cudaErrorInvalidValue;
  PrepParams p;
  p.qkv = qkv; p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.q_out = q_out; p.pool = pool;
  p.page_stride = page_stride; p.head_stride = head_stride; p.positions = positions; p.slot_mapping = slot_mapping; p.freq = freq;
  p.T = T; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.rot_dims = rot_dims; p.interleaved = interleaved;
  p.unit_rms = unit_rms; p.eps = eps;
  p.pairs = !f32 && (reinterpret_cast<uintptr_t>(qkv) & 3) == 0 && ld % 2 == 0 && (q_off | k_off | v_off) % 2 == 0 && dim % 2 == 0 && vdim % 2 == 0;
  const long long warps = (long long)T * ((heads + 2 * kv_heads + kPrepHeads - 1) / kPrepHeads);
  const dim3 grid((unsigned)((warps + 3) / 4));
  if (f32) return (int)launch_pdl(attn_prep_pages_kernel<float>, grid, dim3(128), 0, s, p);
  return (int)launch_pdl(attn_prep_pages_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, p);
}

// q, k and v of the T rows (element offsets into a row of qkv) through a causal convolution over time (w [taps][C] fp32, taps <= 8, C the
// columns q | k | v; state [rows][taps - 1][C], activation type, which advances unless no_store): q times 1 + temp_coef ln(floor((position
// + 1) / temp_every) + 1) to q_out, k and v (divided by their root mean square: unit_v) to their page slots (-1: skip).  max_q: the longest
// run of the batch.  state_only: the state advances and nothing else is written.
BLZ_API int blz_conv_prep_pages(const void* qkv, long long ld, long long q_off, long long k_off, long long v_off, void* q_out, void* pool,
                                long long page_stride, long long head_stride, const int* positions, const int* slot_mapping, const float* w,
                                void* state, const int* slots, const int* q_start, const int* ctx_len, const int* no_store, int B, int max_q,
                                int T, int heads, int kv_heads, int dim, int vdim, int taps, int unit_v, float temp_coef, float temp_every,
                                float eps, int state_only, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || B < 1 || B > 65535 || max_q < 1 || heads < 1 || kv_heads < 1 || heads + 2 * kv_heads > 4 * 65535 || dim < 1 || vdim < 1 ||
      taps < 1 || taps > kConvPrepTok || !w || (taps > 1 && !state) || temp_every <= 0.f)
    return (int)cudaErrorInvalidValue;
  ConvPrepParams q = {};
  PrepParams& p = q.a;
  p.qkv = qkv; p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.q_out = q_out; p.pool = pool;
  p.page_stride = page_stride; p.head_stride = head_stride; p.positions = positions; p.slot_mapping = slot_mapping;
  p.T = T; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.eps = eps;
  q.w = w; q.state = state; q.slots = slots; q.q_start = q_start; q.ctx_len = ctx_len; q.no_store = no_store;
  q.taps = taps; q.unit_v = unit_v; q.state_only = state_only; q.temp_coef = temp_coef; q.temp_every = temp_every;
  const int unit = f32 ? 16 : 8;                       // bytes of four columns
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && (ld | q_off | k_off | v_off) % 4 == 0 && reinterpret_cast<uintptr_t>(qkv) % unit == 0 &&
                   reinterpret_cast<uintptr_t>(state) % unit == 0;
  if (f32) return taps <= 4 ? launch_conv_prep<float, 4>(q, vec, B, max_q, s) : launch_conv_prep<float, 8>(q, vec, B, max_q, s);
  return taps <= 4 ? launch_conv_prep<__nv_bfloat16, 4>(q, vec, B, max_q, s) : launch_conv_prep<__nv_bfloat16, 8>(q, vec, B, max_q, s);
}

// One softmax map per head with an optional sink ([heads] fp32) and an optional output gate ([T, ld_gate], columns like out's);
// out [T, ld_out] = attention * sigmoid(gate) * post.  Any size (vdim <= 1024), fp32 or bf16, every row of the step.
BLZ_API int blz_soft_plain(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, long long head_stride,
                           const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                           const float* sink, const void* gate, long long ld_gate, const int* seq_of_row, int T, int B, int heads,
                           int kv_heads, int dim, int vdim, int window, float scale, float post, int f32, cudaStream_t s) {
  blz::MapsParams p = blz::soft_params(q, ld, out, ld_out, pool, page_stride, head_stride, block_table, bt_stride, slots, q_start, ctx_len,
                                       sink, gate, ld_gate, T, B, heads, kv_heads, dim, vdim, window, scale, post);
  p.seq_of_row = seq_of_row;
  return blz::run_plain(p, f32, s);
}

// Every head against the one vector a token has in its page (dim columns, a multiple of 16, of which the first vdim are the value), with an
// optional sink; otherwise as above.
BLZ_API int blz_shared_plain(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, const int* block_table,
                             int bt_stride, const int* slots, const int* q_start, const int* ctx_len, const float* sink, const int* seq_of_row,
                             int T, int B, int heads, int dim, int vdim, int window, float scale, int f32, cudaStream_t s) {
  if (dim % 16 || vdim > dim) return (int)cudaErrorInvalidValue;
  blz::MapsParams p = blz::soft_params(q, ld, out, ld_out, pool, page_stride, 0, block_table, bt_stride, slots, q_start, ctx_len, sink, nullptr, 0,
                                       T, B, heads, 1, dim, vdim, window, scale, 1.f);
  p.seq_of_row = seq_of_row;
  p.shared_kv = 1;
  return blz::run_plain(p, f32, s);
}

// One softmax map (blz_soft_plain) for the short sequences of a bf16 step; see blz_diff_short (one map: part_o [...][1][16][VP]).
BLZ_API int blz_soft_short(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, long long head_stride,
                           const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                           const float* sink, const void* gate, long long ld_gate, int T, int B, int heads, int kv_heads, int dim, int vdim,
                           int window, float scale, float post, int max_rows, int row_blocks, int splits, float* part_o, float* part_ml,
                           cudaStream_t s) {
  blz::MapsParams p = blz::soft_params(q, ld, out, ld_out, pool, page_stride, head_stride, block_table, bt_stride, slots, q_start, ctx_len,
                                       sink, gate, ld_gate, T, B, heads, kv_heads, dim, vdim, window, scale, post);
  p.max_rows = max_rows; p.row_blocks = row_blocks; p.splits = splits; p.part_o = part_o; p.part_ml = part_ml;
  return blz::run_short(p, s);
}

// Sigmoid attention (attn_maps.cuh): bias [heads][reach + 256] fp32, every row of the step; otherwise as blz_soft_plain.
BLZ_API int blz_sigmoid_plain(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, long long head_stride,
                              const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                              const float* bias, int reach, const int* seq_of_row, int T, int B, int heads, int kv_heads, int dim, int vdim,
                              int window, float scale, float post, int f32, cudaStream_t s) {
  blz::MapsParams p = blz::soft_params(q, ld, out, ld_out, pool, page_stride, head_stride, block_table, bt_stride, slots, q_start, ctx_len,
                                       nullptr, nullptr, 0, T, B, heads, kv_heads, dim, vdim, window, scale, post);
  if (!bias) return (int)cudaErrorInvalidValue;
  p.seq_of_row = seq_of_row; p.bias = bias; p.reach = reach;
  return blz::run_plain(p, f32, s);
}

// The same for the short sequences of a bf16 step (see blz_soft_short); bias times -log2(e).
BLZ_API int blz_sigmoid_short(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, long long head_stride,
                              const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                              const float* bias, int reach, int T, int B, int heads, int kv_heads, int dim, int vdim, int window, float scale,
                              float post, int max_rows, int row_blocks, int splits, float* part_o, float* part_ml, cudaStream_t s) {
  blz::MapsParams p = blz::soft_params(q, ld, out, ld_out, pool, page_stride, head_stride, block_table, bt_stride, slots, q_start, ctx_len,
                                       nullptr, nullptr, 0, T, B, heads, kv_heads, dim, vdim, window, scale, post);
  if (!bias) return (int)cudaErrorInvalidValue;
  p.max_rows = max_rows; p.row_blocks = row_blocks; p.splits = splits; p.part_o = part_o; p.part_ml = part_ml; p.bias = bias; p.reach = reach;
  return blz::run_short(p, s);
}
