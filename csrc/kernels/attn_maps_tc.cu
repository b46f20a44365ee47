// Softmax attention of one or two maps per head (attn_maps.cuh) for long prompt portions, on tcgen05.
//
// Two maps: a CTA takes up to 128 query rows (tokens x group) of one key/value head.  The two maps of a head are the two halves of a
// ping-pong: warpgroup 0 runs the softmax of map 1, warpgroup 1 that of map 2, while the tensor core works on the other map.
// One map: a CTA takes two blocks of up to 128 query rows; the blocks are the two halves, and share keys and values.
// Sigmoid (one map): a weight needs no maximum and no sum, so O is never rescaled; the biases of a row's listed distances are read from a
// table in shared memory, and beyond them a tile has one number per row.  The table also masks what a row may not see.
//   S_m = Q_m K_m^T   A = Q_m [128 x dim], B = K_m [128 keys x dim], both K-major in shared memory
//   O_m += P_m V      A = P_m in tensor memory, B = V [keys x vdim], the pages' token-major blocks read as an MN-major operand
// Tensor memory (512 columns): S_1 | S_2 | O_1 | O_2, 128 each.  A map's weights overwrite its scores as two bf16 halves, value
// and remainder (64 columns each), and both enter the value product, so a weight is not rounded to 8 bits.  O accumulates in
// tensor memory over the key tiles; a row's running maximum moves only when its scores outgrow it by 2^8, and then the row's
// thread rescales O there (QK of a tile is issued behind PV of the tile before, so O is quiet while scores are looked at).
// At the end, with two maps each thread joins one half of a row's columns: a1 - lam a2, the head's RMS norm, the output; with one
// each thread divides its row by the sum of its weights (and the sink), gates it and writes it.
//
// Roles (three warpgroups): warps 0-3 / 4-7 softmax of half 1 / 2 (one row per thread), warp 8 loads pages with bulk copies,
// warp 9 issues the MMAs.  setmaxnreg moves registers from the last warpgroup to the softmax ones (216 / 216 / 72 of 3 x 168).
#include "blaze/attn.cuh"
#include "blaze/attn_maps.cuh"
#include "blaze/host.h"

namespace blz {

static constexpr int kTcThreads = 384;
template <int N> __device__ __forceinline__ void maps_reg_inc() { asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(N)); }
template <int N> __device__ __forceinline__ void maps_reg_dec() { asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(N)); }
static constexpr float kTcLazy = 8.f;

// D += A (tensor memory) x B (shared memory)
__device__ __forceinline__ void mma_f16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}\n"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
struct MapsTc {
  int ks, vs;                  // K and V ring depths
  int tab_ld;                  // sigmoid: floats per head of the bias table in shared memory (0: it stays in global memory)
};

template <int MAPS, bool SIG>
__global__ void __launch_bounds__(kTcThreads, 1) maps_tc_kernel(MapsParams p, MapsTc c, int vec_q, int vec_o) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~uintptr_t(127));
  const int dp = p.dp(), vp = p.vp(), group = p.group(), tph = 128 / group, tpb = MAPS == 1 ? 2 * tph : tph;   // tokens per half, per CTA
  const int q_bytes = 128 * dp * 2, k_bytes = 128 * dp * 2, v_bytes = 128 * vp * 2;     // one half's queries, one map's keys; one tile of values
  uint8_t* sQ = smem;                                  // [2]
  uint8_t* sK = sQ + 2 * q_bytes;                      // [ks][MAPS]
  uint8_t* sV = sK + c.ks * MAPS * k_bytes;               // [vs]
  float* s_l = reinterpret_cast<float*>(sV + c.vs * v_bytes);   // [2][128] sums of the weights
  float* s_ss = s_l + 256;                             // [2][128] sums of squares of a row's halves
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_ss + 256);
  uint64_t *k_full = bars, *k_empty = bars + 2, *v_full = bars + 4, *v_empty = bars + 6, *s_full = bars + 8, *p_full = bars + 10,
           *o_full = bars + 12, *q_full = bars + 14;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_item = reinterpret_cast<int*>(tmem_slot + 2);          // sequence, first token of the row block
  float* s_tab = reinterpret_cast<float*>(s_item + 2);          // [group][tab_ld]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_trigger();
  pdl_wait();
  if (warp == 8) {
    // which sequence and row block this CTA has: the long sequences' blocks in order
    int item = gridDim.x - 1 - blockIdx.x, b = -1, q0 = 0;         // the last blocks of a sequence see the most keys: they start first
    for (int base = 0; base < p.B; base += 32) {
      const int i = base + lane;
      const int qlen = i < p.B ? p.q_start[i + 1] - p.q_start[i] : 0;
      const int n = qlen * group > p.max_rows ? (qlen + tpb - 1) / tpb : 0;
      int incl = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += v;
      }
      const unsigned hit = __ballot_sync(0xffffffffu, item >= incl - n && item < incl);
      if (hit) {
        const int src = __ffs(hit) - 1;
        b = base + src;
        q0 = (item - __shfl_sync(0xffffffffu, incl - n, src)) * tpb;
        break;
      }
      item -= __shfl_sync(0xffffffffu, incl, 31);
    }
    if (lane == 0) { s_item[0] = b; s_item[1] = q0; }
  }
  if (threadIdx.x == 0) {
    for (int i = 0; i < 8; ++i) mbar_init(&bars[i], 1);            // k / v full and empty
    for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 4); mbar_init(&o_full[i], 1); }
    mbar_init(q_full, 8);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if constexpr (SIG) {
    if (c.tab_ld)
      for (int i = threadIdx.x; i < group * p.bias_len(); i += kTcThreads)
        s_tab[i / p.bias_len() * c.tab_ld + i % p.bias_len()] = p.bias[(size_t)blockIdx.y * group * p.bias_len() + i];
  }
  __syncwarp();
  if (warp == 9) tmem_alloc(tmem_slot, 512);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const int b = s_item[0], q0 = s_item[1];
  const int g = blockIdx.y, bb = max(b, 0);
  const int r0 = p.q_start[bb], qlen = p.q_start[bb + 1] - r0, pos0 = p.ctx_len[bb] - qlen;
  const int ntok = b < 0 ? 0 : min(qlen - q0, tpb);
  const int pg_lo = first_key(pos0 + q0, p.window) >> 4, pg_hi = (pos0 + q0 + ntok - 1) >> 4;
  const int n = b < 0 ? 0 : (pg_hi - pg_lo + 8) / 8;               // tiles of 8 pages
  if (warp >= 8) {
    maps_reg_dec<72>();
    if (warp == 8) {
      // -------------------------------------------------------------- page loader
      const int* bt = p.block_table + (size_t)p.slots[b] * p.bt_stride;
      const __nv_bfloat16* pool = reinterpret_cast<const __nv_bfloat16*>(p.pool) + (size_t)g * p.head_stride;
      const int part = lane >> 3, pg = lane & 7;
      int i = 0;
      for (; i < n; ++i) {
        const int ks = i % c.ks, vs = i % c.vs;
        const int pidx = pg_lo + i * 8 + pg;
        int page = 0;                                    // page 0: finite numbers, masked
        if (lane < 8 * (MAPS + 1) && pidx <= pg_hi) page = p.page_base ? p.page_base[b] + pidx : bt[pidx];
        const __nv_bfloat16* src = pool + (size_t)page * p.page_stride;
        if (!__all_sync(0xffffffffu, mbar_wait(&k_empty[ks], (uint32_t)(((i / c.ks) & 1) ^ 1), abort_flag, p.status))) break;
        if (lane == 0) mbar_expect_tx(&k_full[ks], MAPS * k_bytes);
        __syncwarp();
        if (part < MAPS) bulk_load(sK + (ks * MAPS + part) * k_bytes + pg * 32 * dp, src + part * 16 * dp, 32 * dp, &k_full[ks]);
        if (!__all_sync(0xffffffffu, mbar_wait(&v_empty[vs], (uint32_t)(((i / c.vs) & 1) ^ 1), abort_flag, p.status))) {
          // this tile's keys are on their way: they land before the block may end
          const long long t0 = clock64();
          while (!mbar_try_sleep(&k_full[ks], (uint32_t)((i / c.ks) & 1), 20000u) && clock64() - t0 < kSpinLimit) {}
          break;
        }
        if (lane == 0) mbar_expect_tx(&v_full[vs], v_bytes);
        __syncwarp();
        if (part == MAPS) bulk_load(sV + vs * v_bytes + pg * 32 * vp, src + MAPS * 16 * dp, 32 * vp, &v_full[vs]);
        __syncwarp();
      }
      if (i < n) {
        // given up: what was sent for the earlier tiles lands too
        for (int k = max(i - 2, 0); k < i; ++k) {
          const long long t0 = clock64();
          while ((!mbar_try_sleep(&k_full[k % c.ks], (uint32_t)((k / c.ks) & 1), 20000u) ||
                  !mbar_try_sleep(&v_full[k % c.vs], (uint32_t)((k / c.vs) & 1), 20000u)) && clock64() - t0 < kSpinLimit) {}
        }
      }
    } else if (warp == 9 && n > 0) {
      // -------------------------------------------------------------- MMA issuer
      if (lane == 0) {
        const uint32_t id_s = make_idesc(1, 1, 128, 128), id_o = make_idesc(1, 1, 128, (uint32_t)vp, 0, 1);
        auto qk = [&](int m, int i) {
          const uint32_t qa = smem_u32(sQ + m * q_bytes), ka = smem_u32(sK + ((i % c.ks) * MAPS + (MAPS == 2 ? m : 0)) * k_bytes);
          for (int s = 0; s < dp / 16; ++s)
            mma_f16(tmem + m * 128, make_smem_desc(qa + s * 256, 128, dp * 16, kSwzNone),
                    make_smem_desc(ka + s * 256, 128, dp * 16, kSwzNone), id_s, s > 0);
          mma_commit(&s_full[m]);
          if (m == 1) mma_commit(&k_empty[i % c.ks]);
        };
        bool ok = mbar_wait(q_full, 0, abort_flag, p.status) && mbar_wait(&k_full[0], 0, abort_flag, p.status);
        if (ok) {
          tc_fence_after();
          qk(0, 0);
          qk(1, 0);
        }
        for (int i = 0; i < n && ok; ++i) {
          ok = mbar_wait(&v_full[i % c.vs], (uint32_t)((i / c.vs) & 1), abort_flag, p.status);
          for (int m = 0; m < 2 && ok; ++m) {
            if (!mbar_wait(&p_full[m], (uint32_t)(i & 1), abort_flag, p.status)) { ok = false; break; }
            tc_fence_after();
            const uint32_t va = smem_u32(sV + (i % c.vs) * v_bytes);
            for (int half = 0; half < 2; ++half)
              for (int s = 0; s < 8; ++s)            // a page of 16 keys per MMA
                mma_f16_ts(tmem + 256 + m * 128, tmem + m * 128 + half * 64 + s * 8,
                           make_smem_desc(va + s * 32 * vp, vp * 16, 128, kSwzNone), id_o, i > 0 || half > 0 || s > 0);
            if (m == 1) mma_commit(&v_empty[i % c.vs]);
            if (i + 1 < n) {
              if (m == 0 && !mbar_wait(&k_full[(i + 1) % c.ks], (uint32_t)(((i + 1) / c.ks) & 1), abort_flag, p.status)) { ok = false; break; }
              tc_fence_after();
              qk(m, i + 1);
            } else {
              mma_commit(&o_full[m]);
            }
          }
        }
      }
    }
  } else {
    maps_reg_inc<216>();
    if (n > 0) {
      // -------------------------------------------------------------- softmax of one half (one row per thread)
      const int m = warp >> 2, r = threadIdx.x & 127;
      const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
      const int t0 = q0 + (MAPS == 1 ? m * tph : 0);               // this half's first token
      const bool live = r < tph * group && t0 + r / group < q0 + ntok;
      const int tq = t0 + r / group, head = g * group + r % group;
      const int pos = live ? pos0 + tq : -1, lo = first_key(pos, p.window);
      {
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(sQ + m * q_bytes);
        auto row_of = [&](int x) -> const __nv_bfloat16* {
          const int t = t0 + x / group, h = g * group + x % group;
          if (x >= tph * group || t >= q0 + ntok) return nullptr;
          return reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)(r0 + t) * p.ld + (size_t)(MAPS == 2 ? h * 2 + m : h) * p.dim;
        };
        if (vec_q) {
          copy_rows(dst, 128, dp, p.dim, r, 128, p.q, row_of);
          copies_wait();
        } else {
          const __nv_bfloat16* src = row_of(r);
          for (int j = 0; j < dp; j += 8) {
            uint4 u = make_uint4(0, 0, 0, 0);
            __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&u);
#pragma unroll
            for (int k = 0; k < 8; ++k)
              if (live && j + k < p.dim) e[k] = src[j + k];
            *reinterpret_cast<uint4*>(dst + core_off(r, j, dp)) = u;
          }
        }
        fence_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(q_full);
      }
      const float sc = p.scale * kLog2e;
      const uint32_t s_addr = tmem + m * 128 + lanes, o_addr = tmem + 256 + m * 128 + lanes;
      float mx = -INFINITY, l = 0.f;
      bool ok = true;
      const float* tab = nullptr;                      // this row's biases by distance
      float far = 0.f;
      if constexpr (SIG) {
        tab = (c.tab_ld ? s_tab + (r % group) * c.tab_ld : p.bias + (size_t)head * p.bias_len()) + kBiasPad;
        far = tab[p.reach - 1];
      }
      for (int i = 0; i < n; ++i) {
        ok = __all_sync(0xffffffffu, mbar_wait(&s_full[m], (uint32_t)(i & 1), abort_flag, p.status));
        if (!ok) break;
        tc_fence_after();
        uint32_t v[4][32];
#pragma unroll
        for (int k = 0; k < 4; ++k) tmem_ld32(s_addr + k * 32, v[k]);
        tmem_ld_wait();
        const int k0 = (pg_lo + i * 8) * 16, a = lo - k0, z = pos - k0;       // columns a..z are visible
        if constexpr (SIG) {
          const float nsc = -sc;
          if (__all_sync(0xffffffffu, z - 127 >= p.reach - 1)) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
              for (int j = 0; j < 32; ++j) v[k][j] = __float_as_uint(fmaf(__uint_as_float(v[k][j]), nsc, far));
          } else {
            const float* at = tab + max(min(z, p.reach + 126), -1);
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
              for (int j = 0; j < 32; ++j) v[k][j] = __float_as_uint(fmaf(__uint_as_float(v[k][j]), nsc, at[-(k * 32 + j)]));
          }
          if (__any_sync(0xffffffffu, a > 0)) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (k * 32 + j < a) v[k][j] = 0x7f800000u;                     // weight 0
          }
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            uint32_t hi[16], rm[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) {
              const float w0 = sigmoid_ex2(__uint_as_float(v[k][2 * j])), w1 = sigmoid_ex2(__uint_as_float(v[k][2 * j + 1]));
              const __nv_bfloat162 h = __floats2bfloat162_rn(w0, w1);
              hi[j] = *reinterpret_cast<const uint32_t*>(&h);
              rm[j] = pack_bf16x2(w0 - __uint_as_float(hi[j] << 16), w1 - __uint_as_float(hi[j] & 0xffff0000u));
            }
            tmem_st16(s_addr + k * 16, hi);
            tmem_st16(s_addr + 64 + k * 16, rm);
          }
        } else {
          if (!__all_sync(0xffffffffu, a <= 0 && z >= 127)) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (k * 32 + j < a || k * 32 + j > z) v[k][j] = 0xff800000u;     // -inf
          }
          float t = -INFINITY;
#pragma unroll
          for (int k = 0; k < 4; ++k)
#pragma unroll
            for (int j = 0; j < 32; j += 2) t = fmaxf(t, fmaxf(__uint_as_float(v[k][j]), __uint_as_float(v[k][j + 1])));
          t *= sc;
          const bool grow = t > mx + kTcLazy || (mx == -INFINITY && t != -INFINITY);
          if (__any_sync(0xffffffffu, grow)) {
            const float mn = grow ? t : mx;
            const float f = grow ? (mx == -INFINITY ? 0.f : ex2(mx - mn)) : 1.f;
            mx = mn;
            l *= f;
            if (i > 0) {
              for (int k = 0; k < vp; k += 16) {
                uint32_t w[16];
                tmem_ld16(o_addr + k, w);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 16; ++j) w[j] = __float_as_uint(__uint_as_float(w[j]) * f);
                tmem_st16(o_addr + k, w);
              }
            }
          }
          const float off = mx == -INFINITY ? 0.f : -mx;        // a row that has seen no key yet: every weight is 2^-inf
          float l0 = 0.f, l1 = 0.f;
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            uint32_t hi[16], rm[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) {
              const float w0 = ex2(fmaf(__uint_as_float(v[k][2 * j]), sc, off)), w1 = ex2(fmaf(__uint_as_float(v[k][2 * j + 1]), sc, off));
              l0 += w0;
              l1 += w1;
              const __nv_bfloat162 h = __floats2bfloat162_rn(w0, w1);
              hi[j] = *reinterpret_cast<const uint32_t*>(&h);
              rm[j] = pack_bf16x2(w0 - __uint_as_float(hi[j] << 16), w1 - __uint_as_float(hi[j] & 0xffff0000u));
            }
            tmem_st16(s_addr + k * 16, hi);
            tmem_st16(s_addr + 64 + k * 16, rm);
          }
          l += l0 + l1;
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[m]);
      }
      if constexpr (MAPS == 1) {
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&o_full[m], 0, abort_flag, p.status));
        tc_fence_after();
        const float f = SIG ? 1.f : 1.f / (l + (p.sink ? ex2(p.sink[head] * kLog2e - mx) : 0.f));
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(r0 + tq) * p.ld_out + (size_t)head * p.vdim;
        const __nv_bfloat16* gate =
            p.gate ? reinterpret_cast<const __nv_bfloat16*>(p.gate) + (size_t)(r0 + tq) * p.ld_gate + (size_t)head * p.vdim : nullptr;
        for (int k = 0; k < vp && ok; k += 16) {
          uint32_t x[16];
          tmem_ld16(o_addr + k, x);
          tmem_ld_wait();
          if (live) {
#pragma unroll
            for (int h = 0; h < 16; h += 8) {
              const int col = k + h;
              float y[8];
#pragma unroll
              for (int j = 0; j < 8; ++j) y[j] = __uint_as_float(x[h + j]) * f * p.post;
              if (vec_o && col + 8 <= p.vdim) {
                if (gate) {
                  const uint4 u = *reinterpret_cast<const uint4*>(gate + col);
                  const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&u);
#pragma unroll
                  for (int j = 0; j < 8; ++j) y[j] = __fdividef(y[j], 1.f + __expf(-bf2f(e[j])));
                }
                *reinterpret_cast<uint4*>(out + col) = make_uint4(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]),
                                                                  pack_bf16x2(y[4], y[5]), pack_bf16x2(y[6], y[7]));
              } else {
#pragma unroll
                for (int j = 0; j < 8; ++j)
                  if (col + j < p.vdim) out[col + j] = __float2bfloat16(gate ? y[j] / (1.f + __expf(-bf2f(gate[col + j]))) : y[j]);
              }
            }
          }
        }
      } else {
        s_l[m * 128 + r] = l;
        // both maps are done: this thread joins columns [m * half, ...) of its row
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&o_full[0], 0, abort_flag, p.status) && mbar_wait(&o_full[1], 0, abort_flag, p.status));
        bar_sync(1, 256);
        tc_fence_after();
        const float i1 = 1.f / s_l[r], i2 = p.lam / s_l[128 + r];
        const int h16 = (vp / 16 + 1) / 2 * 16, c0 = m * h16, c1 = m ? vp : h16;     // 16-column groups of this half: at most 4
        float o[64];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          if (c0 + k * 16 < c1 && ok) {
            uint32_t x[16], y[16];
            tmem_ld16(tmem + 256 + lanes + c0 + k * 16, x);
            tmem_ld16(tmem + 384 + lanes + c0 + k * 16, y);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) {
              const float d = __uint_as_float(x[j]) * i1 - __uint_as_float(y[j]) * i2;   // padded columns are zero in both
              o[k * 16 + j] = d;
              ss = fmaf(d, d, ss);
            }
          }
        }
        s_ss[m * 128 + r] = ss;
        bar_sync(1, 256);
        if (ok && live) {
          const float f = p.post / sqrtf((s_ss[r] + s_ss[128 + r]) / (float)p.vdim + p.eps);
          __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(r0 + tq) * p.ld_out + (size_t)head * p.vdim;
#pragma unroll
          for (int k = 0; k < 64; k += 8) {
            const int col = c0 + k;
            if (col >= c1) break;
            if (vec_o && col + 8 <= p.vdim) {
              *reinterpret_cast<uint4*>(out + col) = make_uint4(pack_bf16x2(o[k] * f, o[k + 1] * f), pack_bf16x2(o[k + 2] * f, o[k + 3] * f),
                                                                pack_bf16x2(o[k + 4] * f, o[k + 5] * f), pack_bf16x2(o[k + 6] * f, o[k + 7] * f));
            } else {
#pragma unroll
              for (int j = 0; j < 8; ++j)
                if (col + j < p.vdim) out[col + j] = __float2bfloat16(o[k + j] * f);
            }
          }
        }
  }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int MAPS, bool SIG = false>
static int run_tc(const MapsParams& p, int items, cudaStream_t s) {
  if (p.T <= 0 || p.B <= 0 || p.heads < 1 || p.kv_heads < 1 || p.kv_heads > 65535 || p.heads % p.kv_heads || p.group() > 128 || p.dim < 1 ||
      p.dim > 256 || p.vdim < 1 || p.vdim > 128 || p.window < 0 || items < 1)
    return (int)cudaErrorInvalidValue;
  if ((p.page_stride * 2) % 16 || (p.head_stride * 2) % 16 || (reinterpret_cast<uintptr_t>(p.pool) & 15)) return (int)cudaErrorInvalidValue;
  const int q_bytes = 256 * p.dp() * 2, k_bytes = MAPS * 128 * p.dp() * 2, v_bytes = 128 * p.vp() * 2, fixed = 128 + 2048 + 256;
  if (SIG && (!p.bias || p.reach < 1)) return (int)cudaErrorInvalidValue;
  MapsTc c = {2, 2, 0};
  int tab = 0;
  auto total = [&]() { return fixed + q_bytes + c.ks * k_bytes + c.vs * v_bytes + tab; };
  if (SIG && p.bias_len() <= 16384) {
    // neighbouring tokens of a head read neighbouring entries; the heads of a warp's rows are set apart by as many banks as it has tokens
    const int ld = (p.bias_len() + 31) / 32 * 32 + (p.group() < 32 ? 32 / p.group() : 1);
    tab = p.group() * ld * 4;
    if (total() <= 227 * 1024) c.tab_ld = ld;
    else tab = 0;
  }
  if (total() > 227 * 1024) c.ks = 1;
  if (total() > 227 * 1024) c.vs = 1;
  if (total() > 227 * 1024) return (int)cudaErrorInvalidValue;
  const int vec_q = (reinterpret_cast<uintptr_t>(p.q) & 15) == 0 && p.ld % 8 == 0 && p.dim % 8 == 0;
  const int vec_o = (reinterpret_cast<uintptr_t>(p.out) & 15) == 0 && p.ld_out % 8 == 0 && p.vdim % 8 == 0 &&
                    (!p.gate || ((reinterpret_cast<uintptr_t>(p.gate) & 15) == 0 && p.ld_gate % 8 == 0));
  static PerDeviceOnce once;
  cudaError_t e = once.smem_limit(maps_tc_kernel<MAPS, SIG>, 227 * 1024);
  if (e != cudaSuccess) return (int)e;
  return (int)launch_pdl(maps_tc_kernel<MAPS, SIG>, dim3(items, p.kv_heads), dim3(kTcThreads), total(), s, p, c, vec_q, vec_o);
}

}  // namespace blz

// Differential attention, bf16; the sequences with more than max_rows = new tokens * group rows, `items` row blocks of 128 / group
// tokens in all.  dim, vdim <= 128, group <= 128.
BLZ_API int blz_diff_tc(const void* qkv, long long ld, void* out, void* pool, long long page_stride, long long head_stride,
                        const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len, int T, int B,
                        int heads, int kv_heads, int dim, int vdim, int window, float scale, float lam, float post, float eps,
                        int max_rows, int items, cudaStream_t s) {
  using namespace blz;
  MapsParams p = {};
  p.q = qkv; p.ld = ld; p.out = out; p.ld_out = (long long)heads * vdim; p.pool = pool; p.page_stride = page_stride; p.head_stride = head_stride;
  p.block_table = block_table; p.bt_stride = bt_stride; p.slots = slots; p.q_start = q_start; p.ctx_len = ctx_len;
  p.T = T; p.B = B; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.window = window; p.maps = 2;
  p.scale = scale; p.lam = lam; p.post = post; p.eps = eps; p.max_rows = max_rows;
  p.status = status_word();
  return run_tc<2>(p, items, s);
}

// One softmax map per head with optional sink and gate (see blz_soft_plain), bf16; the sequences with more than max_rows rows,
// `items` row blocks of 2 * (128 / group) tokens in all.  vdim <= 128, group <= 128, dim as far as shared memory goes (192 at least).
// page_base ([B] or null): the pages of sequence b lie one after the other from page_base[b] (of position 0, which need not exist) on.
BLZ_API int blz_soft_tc(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, long long head_stride,
                        const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len, const float* sink,
                        const void* gate, long long ld_gate, int T, int B, int heads, int kv_heads, int dim, int vdim, int window,
                        float scale, float post, int max_rows, int items, const int* page_base, cudaStream_t s) {
  using namespace blz;
  MapsParams p = {};
  p.page_base = page_base;
  p.q = q; p.ld = ld; p.out = out; p.ld_out = ld_out; p.pool = pool; p.page_stride = page_stride; p.head_stride = head_stride;
  p.block_table = block_table; p.bt_stride = bt_stride; p.slots = slots; p.q_start = q_start; p.ctx_len = ctx_len;
  p.sink = sink; p.gate = gate; p.ld_gate = ld_gate;
  p.T = T; p.B = B; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.window = window; p.maps = 1;
  p.scale = scale; p.post = post; p.max_rows = max_rows;
  p.status = status_word();
  return run_tc<1>(p, items, s);
}

// Sigmoid attention (attn_maps.cuh) of the long sequences of a bf16 step; bias [heads][reach + 256] fp32 times -log2(e); otherwise as
// blz_soft_tc.
BLZ_API int blz_sigmoid_tc(const void* q, long long ld, void* out, long long ld_out, void* pool, long long page_stride, long long head_stride,
                           const int* block_table, int bt_stride, const int* slots, const int* q_start, const int* ctx_len,
                           const float* bias, int reach, int T, int B, int heads, int kv_heads, int dim, int vdim, int window, float scale,
                           float post, int max_rows, int items, cudaStream_t s) {
  using namespace blz;
  MapsParams p = {};
  p.q = q; p.ld = ld; p.out = out; p.ld_out = ld_out; p.pool = pool; p.page_stride = page_stride; p.head_stride = head_stride;
  p.block_table = block_table; p.bt_stride = bt_stride; p.slots = slots; p.q_start = q_start; p.ctx_len = ctx_len;
  p.T = T; p.B = B; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.window = window; p.maps = 1;
  p.scale = scale; p.post = post; p.max_rows = max_rows; p.bias = bias; p.reach = reach;
  p.status = status_word();
  return run_tc<1, true>(p, items, s);
}
