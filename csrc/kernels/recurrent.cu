// Recurrent mixers with an fp32 state per sequence and head, token by token, for decode rows and prompt runs alike:
//   delta rule with a decay per key channel:  S <- g * S (rows);  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//       g = exp(-A softplus(a + dt_bias)), beta = sigmoid(b), q and k made unit vectors, q times dim^-1/2; or one decay per head
//   state-space duality:  S <- exp(-A dt) S + dt B x^T;  y = S^T C + D x,  dt = softplus(dt_raw + dt_bias)
//   minGRU, element by element:  S <- (1 - z) S + z c;  o = S silu(g),  z = sigmoid(z_raw), c = u + 1/2 (u >= 0) or sigmoid(u)
//   gated linear (HGRN2): S <- f * S + (1 - f) v^T (f acts on rows);  o = S^T silu(q),  f = lo + (1 - lo) sigmoid(f_raw + bias)
//       (rows beyond dk have f = 0 and q = 0)
// and the norm over groups of columns with a gate before or after it that follows either of them.
// State: [rows, heads, keys (or state size), vdim] fp32; rows are sequence slots; a sequence without earlier tokens starts at zero.
//
// A warp holds 4 * VPT columns of a head's state in registers: 8 lanes share a column's rows (R each), so that a token costs R * VPT
// multiply-adds per lane and product, and one reduction over 8 lanes.  The delta rule takes both of its products from the decayed
// state at once (o = S^T q + (k . q) u), which leaves a single reduction on the path from token to token.  What a token needs
// besides the state (unit vectors, decays, steps: all fp32) does not depend on the state:
//   single tokens (decode) take it straight from memory; runs of a few (verify rows) prepare it in shared memory, 8 tokens at a time;
//   long runs have it prepared for all tokens at once by a kernel of its own, as one record per token and head (or group) in a
//   workspace, and the kernel that holds the state streams the records of 8 tokens at a time through a ring of bulk copies.
#include "blaze/host.h"
#include "blaze/sm100.cuh"

namespace blz {

static constexpr int kRecTok = 8;            // tokens per group
static constexpr int kRecWarps = 4;          // warps that hold state

struct RecParams {
  const void* conv;            // [T, ld_conv] convolved inputs: delta q | k | v, state space x | B | C; gated linear: v
  const void* a;               // delta: decay inputs [T, ld_a], heads * dk columns (one decay per head: heads columns); state space: dt_raw [T, ld_a], heads columns;
                               // gated linear: f_raw, heads * dk columns
  const void* b;               // delta: beta inputs [T, ld_b], heads columns; gated linear: q before its activation, heads * dk columns
  const float* A;              // [heads], positive; gated linear: lower bounds [heads * dk]
  const float* dt_bias;        // delta and gated linear [heads * dk], state space and delta with one decay per head [heads]
  const float* D;              // [heads] or null
  float* state;
  float* out;                  // [T, heads * dv] or null (the state only)
  const int *slots, *q_start, *ctx_len, *no_store;
  long long ld_conv, ld_a, ld_b;
  int heads, groups, dk, dv;   // groups: key heads (delta), B / C groups (state space), heads (gated linear)
  const int* seq_of_row;       // [T], -1 = padding
  float* records;              // workspace of the long runs
  int T, long_rows;            // sequences with at least long_rows new tokens are long runs
  int* status;
};

__device__ __forceinline__ float rc_ld(const float* p) { return *p; }
__device__ __forceinline__ float rc_ld(const __nv_bfloat16* p) { return bf2f(*p); }
template <typename T>
__device__ __forceinline__ float rc_exp(float x) {
  if constexpr (sizeof(T) == 4) return expf(x);
  return __expf(x);
}
template <typename T>
__device__ __forceinline__ float rc_softplus(float x) { return x > 20.f ? x : log1pf(rc_exp<T>(x)); }
template <typename T>
__device__ __forceinline__ float rc_sigmoid(float x) { return 1.f / (1.f + rc_exp<T>(-x)); }

// the recurrences; GATED shares the kernels of SSM, which have no reduction between tokens, HDELTA (one decay per head) those of DELTA
enum RecKind { DELTA, SSM, GATED, HDELTA };
// the decay of a head (HDELTA)
template <typename T>
__device__ __forceinline__ float head_decay(const RecParams& p, size_t row, int h) {
  return rc_exp<T>(-p.A[h] * rc_softplus<T>(rc_ld(reinterpret_cast<const T*>(p.a) + row * p.ld_a + h) + p.dt_bias[h]));
}
template <typename T>
__device__ __forceinline__ float rc_silu(float x) { return x * rc_sigmoid<T>(x); }
template <typename T>
__device__ __forceinline__ float forget_gate(float z, float lo) { return fmaf(1.f - lo, rc_sigmoid<T>(z), lo); }

// lane (row group kl < KL, column group cg) of a warp: rows kl * 4 + 4 KL * (i / 4) + i % 4, i < R; columns col .. col + VPT
template <int KL, int R, int VPT>
__device__ __forceinline__ void load_state(float (&S)[R][VPT], const float* st, int kl, int col, int dk, int dv, bool zero, bool vec) {
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = kl * 4 + 4 * KL * (i / 4) + (i & 3);
#pragma unroll
    for (int c = 0; c < VPT; ++c) S[i][c] = 0.f;
    if (zero || r >= dk) continue;
    const float* p = st + (size_t)r * dv + col;
    if (VPT == 4 && vec && col < dv) {
      const float4 f = *reinterpret_cast<const float4*>(p);
      S[i][0] = f.x; S[i][1 % VPT] = f.y; S[i][2 % VPT] = f.z; S[i][3 % VPT] = f.w;
    } else {
#pragma unroll
      for (int c = 0; c < VPT; ++c)
        if (col + c < dv) S[i][c] = p[c];
    }
  }
}
template <int KL, int R, int VPT>
__device__ __forceinline__ void store_state(const float (&S)[R][VPT], float* st, int kl, int col, int dk, int dv, bool vec) {
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = kl * 4 + 4 * KL * (i / 4) + (i & 3);
    if (r >= dk) continue;
    float* p = st + (size_t)r * dv + col;
    if (VPT == 4 && vec && col < dv) {
      *reinterpret_cast<float4*>(p) = make_float4(S[i][0], S[i][1 % VPT], S[i][2 % VPT], S[i][3 % VPT]);
    } else {
#pragma unroll
      for (int c = 0; c < VPT; ++c)
        if (col + c < dv) p[c] = S[i][c];
    }
  }
}

// sums of y[token][column] over the KL (8 or 16) lanes of a column, the 8 tokens spread over them: lane kl ends with token kl % 8 in y[0]
template <int KL, int VPT>
__device__ __forceinline__ void spread_tokens(float (&y)[kRecTok][VPT], int kl) {
  const bool u4 = kl & 4, u2 = kl & 2, u1 = kl & 1;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    float z4[4], z2[2];
#pragma unroll
    for (int j = 0; j < 4; ++j) z4[j] = (u4 ? y[j + 4][v] : y[j][v]) + __shfl_xor_sync(0xffffffffu, u4 ? y[j][v] : y[j + 4][v], 4);
#pragma unroll
    for (int j = 0; j < 2; ++j) z2[j] = (u2 ? z4[j + 2] : z4[j]) + __shfl_xor_sync(0xffffffffu, u2 ? z4[j] : z4[j + 2], 2);
    y[0][v] = (u1 ? z2[1] : z2[0]) + __shfl_xor_sync(0xffffffffu, u1 ? z2[0] : z2[1], 1);
    if constexpr (KL == 16) y[0][v] += __shfl_xor_sync(0xffffffffu, y[0][v], 8);
  }
}
template <int VPT>
__device__ __forceinline__ void store_cols(float* o, const float (&y)[VPT], int col, int dv, bool vec) {
  if (VPT == 4 && vec) {
    if (col < dv) *reinterpret_cast<float4*>(o) = make_float4(y[0], y[1 % VPT], y[2 % VPT], y[3 % VPT]);
  } else {
#pragma unroll
    for (int v = 0; v < VPT; ++v)
      if (col + v < dv) o[v] = y[v];
  }
}

// grid (B * slices, heads), 128 threads
template <typename T, int R, int VPT, bool HD>
__global__ void __launch_bounds__(kRecWarps * 32, R * VPT <= 64 ? 4 : 2) delta_rule_kernel(RecParams p, int slices) {
  constexpr int DKP = R * 8, COLS = kRecWarps * 4 * VPT, V0 = (HD ? 2 : 3) * DKP, TOK = V0 + COLS + 4, NV = DKP / 32;
  extern __shared__ float sm[];              // [2][kRecTok][q | k | (g) | v | beta | k . q | (g)]; a token is a multiple of 16 bytes
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane & 7;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n <= 1 || n >= p.long_rows) return;          // single tokens and long runs have kernels of their own
  const int dk = p.dk, dv = p.dv, hk = h / (p.heads / p.groups);
  const int col = slice * COLS + warp * 4 * VPT + (lane >> 3) * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * dk * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT];
  load_state<8, R, VPT>(S, st, kl, col, dk, dv, ctx == n, vec);
  const float A = p.A[h], qs = rsqrtf((float)dk);

  auto stage = [&](int t0, float* buf) {
    for (int j = warp; j < kRecTok && t0 + j < n; j += kRecWarps) {
      const size_t row = (size_t)(r0 + t0 + j);
      float* s = buf + j * TOK;
      const T* cv = reinterpret_cast<const T*>(p.conv) + row * p.ld_conv;
      const T* av = reinterpret_cast<const T*>(p.a) + row * p.ld_a + (size_t)(HD ? 0 : h) * dk;
      float q[NV], k[NV], qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = lane + i * 32;
        q[i] = d < dk ? rc_ld(cv + (size_t)hk * dk + d) : 0.f;
        k[i] = d < dk ? rc_ld(cv + (size_t)(p.groups + hk) * dk + d) : 0.f;
        qq = fmaf(q[i], q[i], qq);
        kk = fmaf(k[i], k[i], kk);
        kq = fmaf(k[i], q[i], kq);
      }
      const float qn = qs / sqrtf(warp_sum(qq) + 1e-6f), kn = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
      kq = warp_sum(kq) * qn * kn;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = lane + i * 32;
        s[d] = q[i] * qn;
        s[DKP + d] = k[i] * kn;
        if constexpr (!HD) s[2 * DKP + d] = d < dk ? rc_exp<T>(-A * rc_softplus<T>(rc_ld(av + d) + p.dt_bias[(size_t)h * dk + d])) : 1.f;
      }
      for (int c = lane; c < COLS; c += 32) {
        const int e = slice * COLS + c;
        s[V0 + c] = e < dv ? rc_ld(cv + (size_t)2 * p.groups * dk + (size_t)h * dv + e) : 0.f;
      }
      if (lane == 0) {
        s[V0 + COLS] = rc_sigmoid<T>(rc_ld(reinterpret_cast<const T*>(p.b) + row * p.ld_b + h));
        s[V0 + COLS + 1] = kq;
        if constexpr (HD) s[V0 + COLS + 2] = head_decay<T>(p, row, h);
      }
    }
  };

  const int lc = warp * 4 * VPT + (lane >> 3) * VPT;       // this lane's columns inside the block
  stage(0, sm);
  __syncthreads();
  for (int t0 = 0, c = 0; t0 < n; t0 += kRecTok, ++c) {
    {
      const float* buf = sm + (c & 1) * kRecTok * TOK;
      const int m = min(kRecTok, n - t0);
      for (int j = 0; j < m; ++j) {
        const float* s = buf + j * TOK;
        const float gh = HD ? s[V0 + COLS + 2] : 0.f;
        float part[VPT], po[VPT], kr[R <= 16 ? R : 1];
#pragma unroll
        for (int v = 0; v < VPT; ++v) part[v] = po[v] = 0.f;
#pragma unroll
        for (int i4 = 0; i4 < R / 4; ++i4) {
          const float4 q4 = *reinterpret_cast<const float4*>(s + kl * 4 + 32 * i4);
          const float4 k4 = *reinterpret_cast<const float4*>(s + DKP + kl * 4 + 32 * i4);
          const float4 g4 = HD ? make_float4(gh, gh, gh, gh) : *reinterpret_cast<const float4*>(s + 2 * DKP + kl * 4 + 32 * i4);
          const float qa[4] = {q4.x, q4.y, q4.z, q4.w}, ka[4] = {k4.x, k4.y, k4.z, k4.w}, ga[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if constexpr (R <= 16) kr[i4 * 4 + i] = ka[i];
#pragma unroll
            for (int v = 0; v < VPT; ++v) {
              float& x = S[i4 * 4 + i][v];
              x *= ga[i];
              part[v] = fmaf(x, ka[i], part[v]);
              po[v] = fmaf(x, qa[i], po[v]);
            }
          }
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1)
#pragma unroll
          for (int v = 0; v < VPT; ++v) part[v] += __shfl_xor_sync(0xffffffffu, part[v], o);
        const float beta = s[V0 + COLS], kq = s[V0 + COLS + 1];
        float u[VPT];
#pragma unroll
        for (int v = 0; v < VPT; ++v) u[v] = beta * (s[V0 + lc + v] - part[v]);
#pragma unroll
        for (int i4 = 0; i4 < R / 4; ++i4) {
          float ka[4];
          if constexpr (R <= 16) {
#pragma unroll
            for (int i = 0; i < 4; ++i) ka[i] = kr[i4 * 4 + i];
          } else {
            const float4 k4 = *reinterpret_cast<const float4*>(s + DKP + kl * 4 + 32 * i4);
            ka[0] = k4.x; ka[1] = k4.y; ka[2] = k4.z; ka[3] = k4.w;
          }
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int v = 0; v < VPT; ++v) S[i4 * 4 + i][v] = fmaf(ka[i], u[v], S[i4 * 4 + i][v]);
        }
        if (p.out) {
          // sums over the 8 lanes, the columns spread over them
          int v0 = 0;
          float o1 = po[0], u1 = u[0];
          if constexpr (VPT == 4) {
            const bool up = kl & 4, up2 = kl & 2;
            const float x0 = (up ? po[2] : po[0]) + __shfl_xor_sync(0xffffffffu, up ? po[0] : po[2], 4);
            const float x1 = (up ? po[3] : po[1]) + __shfl_xor_sync(0xffffffffu, up ? po[1] : po[3], 4);
            o1 = (up2 ? x1 : x0) + __shfl_xor_sync(0xffffffffu, up2 ? x0 : x1, 2);
            v0 = (up ? 2 : 0) + (up2 ? 1 : 0);
            u1 = up ? (up2 ? u[3] : u[2]) : (up2 ? u[1] : u[0]);
          } else if constexpr (VPT == 2) {
            const bool up = kl & 4;
            o1 = (up ? po[1] : po[0]) + __shfl_xor_sync(0xffffffffu, up ? po[0] : po[1], 4);
            o1 += __shfl_xor_sync(0xffffffffu, o1, 2);
            v0 = up ? 1 : 0;
            u1 = up ? u[1] : u[0];
          } else {
            o1 += __shfl_xor_sync(0xffffffffu, o1, 4);
            o1 += __shfl_xor_sync(0xffffffffu, o1, 2);
          }
          o1 += __shfl_xor_sync(0xffffffffu, o1, 1);
          constexpr int SAME = VPT == 4 ? 1 : (VPT == 2 ? 3 : 7);      // lanes that hold the same column
          if ((kl & SAME) == 0 && col + v0 < dv) p.out[((size_t)(r0 + t0 + j) * p.heads + h) * dv + col + v0] = fmaf(kq, u1, o1);
        }
      }
    }
    if (t0 + kRecTok < n) stage(t0 + kRecTok, sm + ((c + 1) & 1) * kRecTok * TOK);
    __syncthreads();
  }
  if (!(p.no_store != nullptr && p.no_store[b])) store_state<8, R, VPT>(S, st, kl, col, dk, dv, vec);
}

template <typename T, int R, int VPT, bool G>
__global__ void __launch_bounds__(kRecWarps * 32, R * VPT <= 64 ? 4 : 2) state_space_kernel(RecParams p, int slices) {
  constexpr int NP = R * 8, COLS = kRecWarps * 4 * VPT, TOK = 2 * NP + COLS + 4;
  extern __shared__ float sm[];              // [2][kRecTok][B | C | x | dt | decay]; G: [f | q | v | ..]
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane & 7;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n <= 1 || n >= p.long_rows) return;          // single tokens and long runs have kernels of their own
  const int N = p.dk, dv = p.dv, g = h / (p.heads / p.groups);
  const int col = slice * COLS + warp * 4 * VPT + (lane >> 3) * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * N * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT];
  load_state<8, R, VPT>(S, st, kl, col, N, dv, ctx == n, vec);
  const float A = G ? 0.f : p.A[h], bias = G ? 0.f : p.dt_bias[h], D = !G && p.D ? p.D[h] : 0.f;

  auto stage = [&](int t0, float* buf) {
    for (int j = warp; j < kRecTok; j += kRecWarps) {
      float* s = buf + j * TOK;
      if constexpr (G) {
        if (t0 + j >= n) continue;
        const size_t row = (size_t)(r0 + t0 + j), hd = (size_t)h * N;
        const T* fr = reinterpret_cast<const T*>(p.a) + row * p.ld_a + hd;
        const T* qr = reinterpret_cast<const T*>(p.b) + row * p.ld_b + hd;
#pragma unroll
        for (int i = 0; i < NP / 32; ++i) {
          const int d = lane + i * 32;
          s[d] = d < N ? forget_gate<T>(rc_ld(fr + d) + p.dt_bias[hd + d], p.A[hd + d]) : 0.f;
          s[NP + d] = d < N ? rc_silu<T>(rc_ld(qr + d)) : 0.f;
        }
        for (int c = lane; c < COLS; c += 32) {
          const int e = slice * COLS + c;
          s[2 * NP + c] = e < dv ? rc_ld(reinterpret_cast<const T*>(p.conv) + row * p.ld_conv + (size_t)h * dv + e) : 0.f;
        }
        continue;
      }
      if (t0 + j >= n) {                     // beyond the run: a step that changes nothing
        for (int d = lane; d < TOK; d += 32) s[d] = d == 2 * NP + COLS + 1 ? 1.f : 0.f;
        continue;
      }
      const size_t row = (size_t)(r0 + t0 + j);
      const T* cv = reinterpret_cast<const T*>(p.conv) + row * p.ld_conv;
      const T* bc = cv + (size_t)p.heads * dv + (size_t)g * N;
#pragma unroll
      for (int i = 0; i < NP / 32; ++i) {
        const int d = lane + i * 32;
        s[d] = d < N ? rc_ld(bc + d) : 0.f;
        s[NP + d] = d < N ? rc_ld(bc + (size_t)p.groups * N + d) : 0.f;
      }
      for (int c = lane; c < COLS; c += 32) {
        const int e = slice * COLS + c;
        s[2 * NP + c] = e < dv ? rc_ld(cv + (size_t)h * dv + e) : 0.f;
      }
      if (lane == 0) {
        const float dt = rc_softplus<T>(rc_ld(reinterpret_cast<const T*>(p.a) + row * p.ld_a + h) + bias);
        s[2 * NP + COLS] = dt;
        s[2 * NP + COLS + 1] = rc_exp<T>(-A * dt);
      }
    }
  };

  const int lc = warp * 4 * VPT + (lane >> 3) * VPT;
  stage(0, sm);
  __syncthreads();
  for (int t0 = 0, c = 0; t0 < n; t0 += kRecTok, ++c) {
    {
      const float* buf = sm + (c & 1) * kRecTok * TOK;
      float y[kRecTok][VPT];
#pragma unroll
      for (int j = 0; j < kRecTok; ++j) {
        const float* s = buf + j * TOK;
        const float dt = G ? 1.f : s[2 * NP + COLS], dec = G ? 0.f : s[2 * NP + COLS + 1];
        float x[VPT];
#pragma unroll
        for (int v = 0; v < VPT; ++v) { x[v] = dt * s[2 * NP + lc + v]; y[j][v] = 0.f; }
        if (t0 + j < n) {
#pragma unroll
          for (int i4 = 0; i4 < R / 4; ++i4) {
            const float4 b4 = *reinterpret_cast<const float4*>(s + kl * 4 + 32 * i4);
            const float4 c4 = *reinterpret_cast<const float4*>(s + NP + kl * 4 + 32 * i4);
            const float ba[4] = {b4.x, b4.y, b4.z, b4.w}, ca[4] = {c4.x, c4.y, c4.z, c4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
              for (int v = 0; v < VPT; ++v) {
                float& z = S[i4 * 4 + i][v];
                z = G ? fmaf(z, ba[i], (1.f - ba[i]) * x[v]) : fmaf(z, dec, ba[i] * x[v]);
                y[j][v] = fmaf(z, ca[i], y[j][v]);
              }
          }
        }
      }
      if (p.out) {
        spread_tokens<8, VPT>(y, kl);
        if (t0 + kl < n) {
          const float* s = buf + kl * TOK + 2 * NP + lc;
#pragma unroll
          for (int v = 0; v < VPT && !G; ++v) y[0][v] = fmaf(D, s[v], y[0][v]);
          store_cols<VPT>(p.out + ((size_t)(r0 + t0 + kl) * p.heads + h) * dv + col, y[0], col, dv, vec);
        }
      }
    }
    if (t0 + kRecTok < n) stage(t0 + kRecTok, sm + ((c + 1) & 1) * kRecTok * TOK);
    __syncthreads();
  }
  if (!(p.no_store != nullptr && p.no_store[b])) store_state<8, R, VPT>(S, st, kl, col, N, dv, vec);
}

// ------------------------------------------------------------------------------------------ single tokens
// A decode row's state is read, changed and written back once; every lane takes what it needs of the token straight from memory, so
// that all of a warp's reads are under way together and no warp waits for another.
// KL lanes per column; elements of a vector as in load_state
template <typename T, int KL, int R>
__device__ __forceinline__ void load_vec_rows(float (&x)[R], const T* src, int kl, int n, bool vec) {
#pragma unroll
  for (int i4 = 0; i4 < R / 4; ++i4) {
    const int r = kl * 4 + 4 * KL * i4;
    if (vec && sizeof(T) == 2) {
      uint2 u = make_uint2(0u, 0u);
      if (r < n) u = *reinterpret_cast<const uint2*>(src + r);
      x[i4 * 4] = __uint_as_float(u.x << 16); x[i4 * 4 + 1] = __uint_as_float(u.x & 0xffff0000u);
      x[i4 * 4 + 2] = __uint_as_float(u.y << 16); x[i4 * 4 + 3] = __uint_as_float(u.y & 0xffff0000u);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i4 * 4 + i] = r + i < n ? rc_ld(src + r + i) : 0.f;
    }
  }
}
template <int KL>
__device__ __forceinline__ float lanes_sum(float x) {
#pragma unroll
  for (int o = KL / 2; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
  return x;
}

template <typename T, int KL, int R, int VPT, bool HD>
__global__ void __launch_bounds__(kRecWarps * 32, 3) delta_step_kernel(RecParams p, int slices, int vec_t) {
  constexpr int CG = 32 / KL;
  __shared__ __align__(16) float s_g[KL * R];
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n != 1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % KL;
  const int dk = p.dk, dv = p.dv, hk = h / (p.heads / p.groups);
  const int col = slice * kRecWarps * CG * VPT + warp * CG * VPT + lane / KL * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * dk * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT], q[R], k[R];
  alignas(16) float g[R];
  load_state<KL, R, VPT>(S, st, kl, col, dk, dv, ctx == 1, vec);
  const T* cv = reinterpret_cast<const T*>(p.conv) + (size_t)r0 * p.ld_conv;
  load_vec_rows<T, KL, R>(q, cv + (size_t)hk * dk, kl, dk, vec_t);
  load_vec_rows<T, KL, R>(k, cv + (size_t)(p.groups + hk) * dk, kl, dk, vec_t);
  float v[VPT];
#pragma unroll
  for (int c = 0; c < VPT; ++c) v[c] = col + c < dv ? rc_ld(cv + (size_t)2 * p.groups * dk + (size_t)h * dv + col + c) : 0.f;
  const float beta = rc_sigmoid<T>(rc_ld(reinterpret_cast<const T*>(p.b) + (size_t)r0 * p.ld_b + h)), A = p.A[h];
  // the decays, one per thread
  const T* av = reinterpret_cast<const T*>(p.a) + (size_t)r0 * p.ld_a + (size_t)(HD ? 0 : h) * dk;
  const float gh = HD ? head_decay<T>(p, r0, h) : 0.f;
  for (int d = threadIdx.x; !HD && d < KL * R; d += kRecWarps * 32)
    s_g[d] = d < dk ? rc_exp<T>(-A * rc_softplus<T>(rc_ld(av + d) + p.dt_bias[(size_t)h * dk + d])) : 1.f;
  float qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    qq = fmaf(q[i], q[i], qq);
    kk = fmaf(k[i], k[i], kk);
    kq = fmaf(k[i], q[i], kq);
  }
  const float qn = rsqrtf((float)dk) / sqrtf(lanes_sum<KL>(qq) + 1e-6f), kn = 1.f / sqrtf(lanes_sum<KL>(kk) + 1e-6f);
  kq = lanes_sum<KL>(kq) * qn * kn;
  if constexpr (!HD) __syncthreads();
#pragma unroll
  for (int i4 = 0; i4 < R / 4 && !HD; ++i4) *reinterpret_cast<float4*>(&g[i4 * 4]) = *reinterpret_cast<const float4*>(s_g + kl * 4 + 4 * KL * i4);
  float part[VPT], po[VPT];
#pragma unroll
  for (int c = 0; c < VPT; ++c) part[c] = po[c] = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i)
#pragma unroll
    for (int c = 0; c < VPT; ++c) {
      S[i][c] *= HD ? gh : g[i];
      part[c] = fmaf(S[i][c], k[i], part[c]);
      po[c] = fmaf(S[i][c], q[i], po[c]);
    }
#pragma unroll
  for (int c = 0; c < VPT; ++c) {
    const float u = beta * (v[c] - lanes_sum<KL>(part[c]) * kn);
    po[c] = fmaf(kq, u, lanes_sum<KL>(po[c]) * qn);
    part[c] = u * kn;
  }
#pragma unroll
  for (int i = 0; i < R; ++i)
#pragma unroll
    for (int c = 0; c < VPT; ++c) S[i][c] = fmaf(k[i], part[c], S[i][c]);
  if (p.out && kl == 0) store_cols<VPT>(p.out + ((size_t)r0 * p.heads + h) * dv + col, po, col, dv, vec);
  if (!(p.no_store != nullptr && p.no_store[b])) store_state<KL, R, VPT>(S, st, kl, col, dk, dv, vec);
}

template <typename T, int KL, int R, int VPT>
__global__ void __launch_bounds__(kRecWarps * 32, 4) state_space_step_kernel(RecParams p, int slices, int vec_t) {
  constexpr int CG = 32 / KL;
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n != 1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % KL;
  const int N = p.dk, dv = p.dv, grp = h / (p.heads / p.groups);
  const int col = slice * kRecWarps * CG * VPT + warp * CG * VPT + lane / KL * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * N * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT], B[R], C[R];
  load_state<KL, R, VPT>(S, st, kl, col, N, dv, ctx == 1, vec);
  const T* cv = reinterpret_cast<const T*>(p.conv) + (size_t)r0 * p.ld_conv;
  const T* bc = cv + (size_t)p.heads * dv + (size_t)grp * N;
  load_vec_rows<T, KL, R>(B, bc, kl, N, vec_t);
  load_vec_rows<T, KL, R>(C, bc + (size_t)p.groups * N, kl, N, vec_t);
  float x[VPT], y[VPT];
#pragma unroll
  for (int c = 0; c < VPT; ++c) x[c] = col + c < dv ? rc_ld(cv + (size_t)h * dv + col + c) : 0.f;
  const float dt = rc_softplus<T>(rc_ld(reinterpret_cast<const T*>(p.a) + (size_t)r0 * p.ld_a + h) + p.dt_bias[h]);
  const float dec = rc_exp<T>(-p.A[h] * dt), D = p.D ? p.D[h] : 0.f;
#pragma unroll
  for (int c = 0; c < VPT; ++c) y[c] = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i)
#pragma unroll
    for (int c = 0; c < VPT; ++c) {
      S[i][c] = fmaf(S[i][c], dec, B[i] * (dt * x[c]));
      y[c] = fmaf(S[i][c], C[i], y[c]);
    }
  if (!(p.no_store != nullptr && p.no_store[b])) store_state<KL, R, VPT>(S, st, kl, col, N, dv, vec);
  if (p.out) {
#pragma unroll
    for (int c = 0; c < VPT; ++c) y[c] = fmaf(D, x[c], lanes_sum<KL>(y[c]));
    if (kl == 0) store_cols<VPT>(p.out + ((size_t)r0 * p.heads + h) * dv + col, y, col, dv, vec);
  }
}

// The gates and queries of a row, one per thread, meet in shared memory.
template <typename T, int KL, int R, int VPT>
__global__ void __launch_bounds__(kRecWarps * 32, 4) gated_step_kernel(RecParams p, int slices, int) {
  constexpr int CG = 32 / KL, NP = KL * R;
  __shared__ __align__(16) float s_f[NP], s_q[NP];
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n != 1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % KL, N = p.dk, dv = p.dv;
  const int col = slice * kRecWarps * CG * VPT + warp * CG * VPT + lane / KL * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * N * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT], v[VPT], y[VPT];
  load_state<KL, R, VPT>(S, st, kl, col, N, dv, ctx == 1, vec);
  const size_t hd = (size_t)h * N;
  const T* fr = reinterpret_cast<const T*>(p.a) + (size_t)r0 * p.ld_a + hd;
  const T* qr = reinterpret_cast<const T*>(p.b) + (size_t)r0 * p.ld_b + hd;
  const T* vr = reinterpret_cast<const T*>(p.conv) + (size_t)r0 * p.ld_conv + (size_t)h * dv + col;
#pragma unroll
  for (int c = 0; c < VPT; ++c) { v[c] = col + c < dv ? rc_ld(vr + c) : 0.f; y[c] = 0.f; }
  for (int d = threadIdx.x; d < NP; d += kRecWarps * 32) {
    s_f[d] = d < N ? forget_gate<T>(rc_ld(fr + d) + p.dt_bias[hd + d], p.A[hd + d]) : 0.f;
    s_q[d] = d < N ? rc_silu<T>(rc_ld(qr + d)) : 0.f;
  }
  __syncthreads();
#pragma unroll
  for (int i4 = 0; i4 < R / 4; ++i4) {
    const float4 f4 = *reinterpret_cast<const float4*>(s_f + kl * 4 + 4 * KL * i4);
    const float4 q4 = *reinterpret_cast<const float4*>(s_q + kl * 4 + 4 * KL * i4);
    const float fa[4] = {f4.x, f4.y, f4.z, f4.w}, qa[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int c = 0; c < VPT; ++c) {
        float& z = S[i4 * 4 + i][c];
        z = fmaf(z, fa[i], (1.f - fa[i]) * v[c]);
        y[c] = fmaf(z, qa[i], y[c]);
      }
  }
  if (!(p.no_store != nullptr && p.no_store[b])) store_state<KL, R, VPT>(S, st, kl, col, N, dv, vec);
  if (p.out) {
#pragma unroll
    for (int c = 0; c < VPT; ++c) y[c] = lanes_sum<KL>(y[c]);
    if (kl == 0) store_cols<VPT>(p.out + ((size_t)r0 * p.heads + h) * dv + col, y, col, dv, vec);
  }
}

// ------------------------------------------------------------------------------------------ long runs
// Records: delta [heads][T][q | k | g | beta, k . q, 0, 0] (one decay per head: see delta_block_records_kernel), state space [groups][T][B | C] and [heads][T][dt, decay, 0, 0], gated
// linear [heads][T][f | q]; vectors padded to 32, 64, 128, 256 or 512 floats.
__device__ __forceinline__ bool in_long_run(const RecParams& p, int t) {
  const int b = p.seq_of_row[t];
  return b >= 0 && p.q_start[b + 1] - p.q_start[b] >= p.long_rows;
}

// a warp per (row, head)
template <typename T, int DKP>
__global__ void __launch_bounds__(128) delta_records_kernel(RecParams p) {
  constexpr int REC = 3 * DKP + 4, NV = DKP / 32;
  const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int t = (int)(w / p.heads), h = (int)(w % p.heads), lane = threadIdx.x & 31;
  if (t >= p.T || !in_long_run(p, t)) return;
  const int dk = p.dk, hk = h / (p.heads / p.groups);
  const T* cv = reinterpret_cast<const T*>(p.conv) + (size_t)t * p.ld_conv;
  const T* av = reinterpret_cast<const T*>(p.a) + (size_t)t * p.ld_a + (size_t)h * dk;
  float q[NV], k[NV], a[NV], qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = lane + i * 32;
    q[i] = d < dk ? rc_ld(cv + (size_t)hk * dk + d) : 0.f;
    k[i] = d < dk ? rc_ld(cv + (size_t)(p.groups + hk) * dk + d) : 0.f;
    a[i] = d < dk ? rc_ld(av + d) + p.dt_bias[(size_t)h * dk + d] : 0.f;
  }
  const float beta = rc_sigmoid<T>(rc_ld(reinterpret_cast<const T*>(p.b) + (size_t)t * p.ld_b + h)), A = p.A[h];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    qq = fmaf(q[i], q[i], qq);
    kk = fmaf(k[i], k[i], kk);
    kq = fmaf(k[i], q[i], kq);
  }
  const float qn = rsqrtf((float)dk) / sqrtf(warp_sum(qq) + 1e-6f), kn = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
  kq = warp_sum(kq) * qn * kn;
  float* s = p.records + ((size_t)h * p.T + t) * REC;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = lane + i * 32;
    s[d] = q[i] * qn;
    s[DKP + d] = k[i] * kn;
    s[2 * DKP + d] = d < dk ? rc_exp<T>(-A * rc_softplus<T>(a[i])) : 1.f;
  }
  if (lane == 0) *reinterpret_cast<float4*>(s + 3 * DKP) = make_float4(beta, kq, 0.f, 0.f);
}

// One decay per head: four tokens at a time.  With S the state before them, G_i the decay over tokens 0..i and D_ij that over j+1..i,
//   u_i = beta_i (v_i - G_i S^T k_i) - sum_{j<i} a_ij u_j,  a_ij = beta_i D_ij k_i . k_j
//   o_i = G_i S^T q_i + sum_{j<=i} c_ij u_j,                c_ij = D_ij q_i . k_j
//   S <- G_3 S + sum_j D_3j k_j u_j
// so that the products with the state do not wait for one another.  A warp per (4 tokens, head) writes what does not depend on the
// state: per token q | k | a_i0..3 | c_i0..3 | beta_i, beta_i G_i, G_i, D_3i | G_3, 0, 0, 0 (a sequence's last tokens: of those there are).
static constexpr int kBlockTok = 4, kBlockCoef = 16;
struct Whole { static constexpr bool value = true; };
struct Part { static constexpr bool value = false; };
template <typename T, int DKP>
__global__ void __launch_bounds__(128) delta_block_records_kernel(RecParams p) {
  constexpr int REC = 2 * DKP + kBlockCoef, NV = DKP / 32;
  const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int h = (int)(w % p.heads), lane = threadIdx.x & 31;
  // the block that starts in these rows: of a sequence that goes on through all of them exactly one does, and a warp whose rows see
  // one sequence end and another begin takes both of theirs in turn
  for (int t = (int)(w / p.heads) * kBlockTok, end = min(t + kBlockTok, p.T); t < end; ++t) {
    if (!in_long_run(p, t)) continue;
    const int seq = p.seq_of_row[t], rest = p.q_start[seq + 1] - t, m = min(kBlockTok, rest);
    if ((t - p.q_start[seq]) % kBlockTok) continue;
    const int dk = p.dk, hk = h / (p.heads / p.groups);
    float q[kBlockTok][NV], k[kBlockTok][NV], beta[kBlockTok], g[kBlockTok];
#pragma unroll
    for (int j = 0; j < kBlockTok; ++j) {
      const T* cv = reinterpret_cast<const T*>(p.conv) + (size_t)(t + min(j, m - 1)) * p.ld_conv;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = lane + i * 32;
        q[j][i] = d < dk && j < m ? rc_ld(cv + (size_t)hk * dk + d) : 0.f;
        k[j][i] = d < dk && j < m ? rc_ld(cv + (size_t)(p.groups + hk) * dk + d) : 0.f;
      }
    }
#pragma unroll
    for (int j = 0; j < kBlockTok; ++j) {
      const size_t row = t + min(j, m - 1);
      beta[j] = rc_sigmoid<T>(rc_ld(reinterpret_cast<const T*>(p.b) + row * p.ld_b + h));
      g[j] = head_decay<T>(p, row, h);
    }
    const float qs = rsqrtf((float)dk);
#pragma unroll
    for (int j = 0; j < kBlockTok; ++j) {
      float qq = 0.f, kk = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) { qq = fmaf(q[j][i], q[j][i], qq); kk = fmaf(k[j][i], k[j][i], kk); }
      const float qn = qs / sqrtf(warp_sum(qq) + 1e-6f), kn = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
#pragma unroll
      for (int i = 0; i < NV; ++i) { q[j][i] *= qn; k[j][i] *= kn; }
    }
    float G = 1.f, D[kBlockTok];                             // D[j]: decay over tokens j + 1 .. i
#pragma unroll
    for (int i = 0; i < kBlockTok; ++i) {
      if (i >= m) break;
      float* s = p.records + ((size_t)h * p.T + t + i) * REC;
      G *= g[i];
      float a[kBlockTok], c[kBlockTok];
#pragma unroll
      for (int j = 0; j < kBlockTok; ++j) {
        a[j] = c[j] = 0.f;
        if (j > i) continue;
        D[j] = j == i ? 1.f : D[j] * g[i];
        float kk = 0.f, qk = 0.f;
#pragma unroll
        for (int e = 0; e < NV; ++e) { kk = fmaf(k[i][e], k[j][e], kk); qk = fmaf(q[i][e], k[j][e], qk); }
        c[j] = D[j] * warp_sum(qk);
        if (j < i) a[j] = beta[i] * D[j] * warp_sum(kk);
      }
#pragma unroll
      for (int e = 0; e < NV; ++e) {
        s[lane + e * 32] = q[i][e];
        s[DKP + lane + e * 32] = k[i][e];
      }
      if (lane == 0) {
        float4* f = reinterpret_cast<float4*>(s + 2 * DKP);
        f[0] = make_float4(a[0], a[1], a[2], a[3]);
        f[1] = make_float4(c[0], c[1], c[2], c[3]);
        float last = 1.f, all = G;                           // decays to the end of the block
#pragma unroll
        for (int e = 1; e < kBlockTok; ++e)
          if (e > i && e < m) { last *= g[e]; all *= g[e]; }
        f[2] = make_float4(beta[i], beta[i] * G, G, last);
        f[3] = make_float4(all, 0.f, 0.f, 0.f);
      }
    }
  }
}

// a block per row
template <typename T, int DKP>
__global__ void __launch_bounds__(128) state_space_records_kernel(RecParams p) {
  constexpr int NP = DKP;
  const int t = blockIdx.x, N = p.dk;
  if (!in_long_run(p, t)) return;
  const T* bc = reinterpret_cast<const T*>(p.conv) + (size_t)t * p.ld_conv + (size_t)p.heads * p.dv;
  for (int i = threadIdx.x; i < p.groups * 2 * NP; i += 128) {
    const int g = i / (2 * NP), which = i / NP & 1, d = i % NP;
    p.records[((size_t)g * p.T + t) * 2 * NP + which * NP + d] = d < N ? rc_ld(bc + (size_t)(which * p.groups + g) * N + d) : 0.f;
  }
  float4* steps = reinterpret_cast<float4*>(p.records + (size_t)p.groups * p.T * 2 * NP);
  for (int h = threadIdx.x; h < p.heads; h += 128) {
    const float dt = rc_softplus<T>(rc_ld(reinterpret_cast<const T*>(p.a) + (size_t)t * p.ld_a + h) + p.dt_bias[h]);
    steps[(size_t)h * p.T + t] = make_float4(dt, rc_exp<T>(-p.A[h] * dt), 0.f, 0.f);
  }
}

// a warp per (row, head)
template <typename T, int DKP>
__global__ void __launch_bounds__(128) gated_records_kernel(RecParams p) {
  const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int t = (int)(w / p.heads), h = (int)(w % p.heads), lane = threadIdx.x & 31, N = p.dk;
  if (t >= p.T || !in_long_run(p, t)) return;
  const size_t hd = (size_t)h * N;
  const T* fr = reinterpret_cast<const T*>(p.a) + (size_t)t * p.ld_a + hd;
  const T* qr = reinterpret_cast<const T*>(p.b) + (size_t)t * p.ld_b + hd;
  float* s = p.records + ((size_t)h * p.T + t) * 2 * DKP;
#pragma unroll
  for (int i = 0; i < DKP / 32; ++i) {
    const int d = lane + i * 32;
    s[d] = d < N ? forget_gate<T>(rc_ld(fr + d) + p.dt_bias[hd + d], p.A[hd + d]) : 0.f;
    s[DKP + d] = d < N ? rc_silu<T>(rc_ld(qr + d)) : 0.f;
  }
}

// Ring of record groups: warp kRecWarps sends the copies, warps 0 .. kRecWarps - 1 wait for them and give the stages back.
static constexpr int kRecStages = 4;
struct RecRing {
  uint64_t *full, *empty;
  volatile int* abort_flag;
  int* status;
  __device__ __forceinline__ void init(uint8_t* sm, int* st) {
    full = reinterpret_cast<uint64_t*>(sm);
    empty = full + kRecStages;
    abort_flag = reinterpret_cast<volatile int*>(empty + kRecStages);
    status = st;
    if (threadIdx.x == 0) {
      for (int i = 0; i < kRecStages; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], kRecWarps); }
      *abort_flag = 0;
      mbar_fence_init();
    }
    __syncthreads();
  }
  __device__ __forceinline__ bool wait_full(int c) {
    return __all_sync(0xffffffffu, mbar_wait(&full[c % kRecStages], (uint32_t)((c / kRecStages) & 1), abort_flag, status));
  }
  __device__ __forceinline__ void release(int c) {
    __syncwarp();
    if ((threadIdx.x & 31) == 0) mbar_arrive(&empty[c % kRecStages]);
  }
  // one thread; send(c) puts group c on its way (expect_tx included)
  template <typename F>
  __device__ __forceinline__ void produce(int groups, F&& send) {
    int c = 0;
    for (; c < groups; ++c) {
      if (c >= kRecStages && !mbar_wait(&empty[c % kRecStages], (uint32_t)((c / kRecStages - 1) & 1), abort_flag, status)) break;
      send(c);
    }
    if (c < groups)          // given up: what is on its way lands before the block may end
      for (int k = max(c - kRecStages, 0); k < c; ++k) {
        const long long t0 = clock64();
        while (!mbar_try_sleep(&full[k % kRecStages], (uint32_t)((k / kRecStages) & 1), 20000u) && clock64() - t0 < kSpinLimit) {}
      }
  }
};

// v (x) columns of a group of tokens on their way into a warp's shared memory, kColsAhead groups ahead of their use; lane kl < 8
// brings token kl's VPT columns.  vec: they can be copied as one word of sizeof(T) * VPT bytes.
static constexpr int kColsAhead = 3;
template <typename T, int VPT>
__device__ __forceinline__ void send_cols(T* dst, const T* src, bool live, int col, int dv, bool vec) {
  if (live) {
    if (vec) {
      if (col < dv)
        asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(dst)), "l"(src), "n"((int)sizeof(T) * VPT) : "memory");
    } else {
#pragma unroll
      for (int i = 0; i < VPT; ++i)
        if (col + i < dv) dst[i] = src[i];
    }
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
}
__device__ __forceinline__ void wait_cols() { asm volatile("cp.async.wait_group %0;" ::"n"(kColsAhead) : "memory"); }

static constexpr int kRecHead = 128;         // barriers in front of the ring

template <typename T, int KL, int R, int VPT>
__global__ void __launch_bounds__((kRecWarps + 1) * 32, R * VPT <= 64 ? 2 : 1) delta_stream_kernel(RecParams p, int slices, int vec_v) {
  constexpr int DKP = R * KL, CG = 32 / KL, COLS = kRecWarps * CG * VPT, REC = 3 * DKP + 4, STAGE = kRecTok * REC;
  constexpr int PART = VPT == 2 ? 2 : 1;            // independent chains per sum
  extern __shared__ __align__(128) uint8_t sm8[];
  __shared__ __align__(16) T s_v[kRecWarps][kColsAhead + 1][kRecTok][CG * VPT];
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n < p.long_rows) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % KL, cg = lane / KL;
  const int groups = (n + kRecTok - 1) / kRecTok;
  float* ring = reinterpret_cast<float*>(sm8 + kRecHead);
  RecRing rr;
  rr.init(sm8, p.status);
  if (warp == kRecWarps) {
    if (lane == 0) {
      const float* src = p.records + ((size_t)h * p.T + r0) * REC;
      rr.produce(groups, [&](int c) {
        const uint32_t bytes = (uint32_t)min(kRecTok, n - c * kRecTok) * REC * 4;
        mbar_expect_tx(&rr.full[c % kRecStages], bytes);
        bulk_load(ring + (c % kRecStages) * STAGE, src + (size_t)c * STAGE, bytes, &rr.full[c % kRecStages]);
      });
    }
    return;
  }
  const int dk = p.dk, dv = p.dv, col = slice * COLS + warp * CG * VPT + cg * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * dk * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT];
  load_state<KL, R, VPT>(S, st, kl, col, dk, dv, ctx == n, vec);
  const T* vsrc = reinterpret_cast<const T*>(p.conv) + (size_t)(r0 + (kl & 7)) * p.ld_conv + (size_t)2 * p.groups * dk + (size_t)h * dv + col;
  auto send_group = [&](int c) {
    send_cols<T, VPT>(&s_v[warp][c % (kColsAhead + 1)][kl & 7][cg * VPT], vsrc + (size_t)c * kRecTok * p.ld_conv,
                      kl < kRecTok && c * kRecTok + kl < n, col, dv, vec_v);
  };
#pragma unroll
  for (int c = 0; c < kColsAhead; ++c) send_group(c);
  bool ok = true;
  for (int c = 0; c < groups; ++c) {
    const int t0 = c * kRecTok, m = min(kRecTok, n - t0);
    __syncwarp();                            // the last group's columns have been read
    send_group(c + kColsAhead);
    wait_cols();
    const T(*cols)[CG * VPT] = s_v[warp][c % (kColsAhead + 1)];
    ok = rr.wait_full(c);
    if (!ok) break;
    __syncwarp();
    const float* buf = ring + (c % kRecStages) * STAGE;
    float y[VPT <= 2 ? kRecTok : 1][VPT];
    // what a token brings: the lane's rows of q, k and g, its v, beta and k . q
    struct Tok {
      float q[R], k[R], g[R], v[VPT];
      float2 bk;
    };
    auto fetch = [&](int j, Tok& o) {
      const float* s = buf + j * REC;
#pragma unroll
      for (int i4 = 0; i4 < R / 4; ++i4) {
        const float4 q4 = *reinterpret_cast<const float4*>(s + kl * 4 + 4 * KL * i4);
        const float4 k4 = *reinterpret_cast<const float4*>(s + DKP + kl * 4 + 4 * KL * i4);
        o.q[i4 * 4] = q4.x; o.q[i4 * 4 + 1] = q4.y; o.q[i4 * 4 + 2] = q4.z; o.q[i4 * 4 + 3] = q4.w;
        o.k[i4 * 4] = k4.x; o.k[i4 * 4 + 1] = k4.y; o.k[i4 * 4 + 2] = k4.z; o.k[i4 * 4 + 3] = k4.w;
        const float4 g4 = *reinterpret_cast<const float4*>(s + 2 * DKP + kl * 4 + 4 * KL * i4);
        o.g[i4 * 4] = g4.x; o.g[i4 * 4 + 1] = g4.y; o.g[i4 * 4 + 2] = g4.z; o.g[i4 * 4 + 3] = g4.w;
      }
      o.bk = *reinterpret_cast<const float2*>(s + 3 * DKP);
#pragma unroll
      for (int v = 0; v < VPT; ++v) o.v[v] = rc_ld(&cols[j][cg * VPT + v]);
    };
    auto token = [&](int j, const Tok& x, float (&po)[VPT]) {
      float part[VPT][PART], pq[VPT][PART];
#pragma unroll
      for (int v = 0; v < VPT; ++v)
#pragma unroll
        for (int i = 0; i < PART; ++i) part[v][i] = pq[v][i] = 0.f;
#pragma unroll
      for (int i = 0; i < R; ++i)
#pragma unroll
        for (int v = 0; v < VPT; ++v) {
          S[i][v] *= x.g[i];
          part[v][i % PART] = fmaf(S[i][v], x.k[i], part[v][i % PART]);
          pq[v][i % PART] = fmaf(S[i][v], x.q[i], pq[v][i % PART]);
        }
      float sum[VPT];
#pragma unroll
      for (int v = 0; v < VPT; ++v) {
        sum[v] = part[v][0];
        po[v] = pq[v][0];
#pragma unroll
        for (int i = 1; i < PART; ++i) { sum[v] += part[v][i]; po[v] += pq[v][i]; }
      }
#pragma unroll
      for (int o = KL / 2; o > 0; o >>= 1)
#pragma unroll
        for (int v = 0; v < VPT; ++v) sum[v] += __shfl_xor_sync(0xffffffffu, sum[v], o);
      float u[VPT];
#pragma unroll
      for (int v = 0; v < VPT; ++v) u[v] = x.bk.x * (x.v[v] - sum[v]);
#pragma unroll
      for (int i = 0; i < R; ++i)
#pragma unroll
        for (int v = 0; v < VPT; ++v) S[i][v] = fmaf(x.k[i], u[v], S[i][v]);
#pragma unroll
      for (int v = 0; v < VPT; ++v) po[v] = kl == 0 ? fmaf(x.bk.y, u[v], po[v]) : po[v];
      if constexpr (VPT == 4) {
        static_assert(VPT != 4 || KL == 8);
        // the four columns spread over the lanes
        const bool up = kl & 4, up2 = kl & 2;
        const float x0 = (up ? po[2 % VPT] : po[0]) + __shfl_xor_sync(0xffffffffu, up ? po[0] : po[2 % VPT], 4);
        const float x1 = (up ? po[3 % VPT] : po[1 % VPT]) + __shfl_xor_sync(0xffffffffu, up ? po[1 % VPT] : po[3 % VPT], 4);
        float o1 = (up2 ? x1 : x0) + __shfl_xor_sync(0xffffffffu, up2 ? x0 : x1, 2);
        o1 += __shfl_xor_sync(0xffffffffu, o1, 1);
        const int v0 = (up ? 2 : 0) + (up2 ? 1 : 0);
        if ((kl & 1) == 0 && col + v0 < dv) p.out[((size_t)(r0 + t0 + j) * p.heads + h) * dv + col + v0] = o1;
      }
    };
    constexpr bool FETCH_AHEAD = R * VPT <= 16;          // registers for the next token's operands
    if (m == kRecTok) {
      Tok tok[2];
      if (FETCH_AHEAD) fetch(0, tok[0]);
#pragma unroll
      for (int j = 0; j < kRecTok; ++j) {
        if (!FETCH_AHEAD) fetch(j, tok[j & 1]);
        else if (j + 1 < kRecTok) fetch(j + 1, tok[(j + 1) & 1]);
        token(j, tok[j & 1], y[VPT <= 2 ? j : 0]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < kRecTok; ++j) {
        if (j < m) {
          Tok tok;
          fetch(j, tok);
          token(j, tok, y[VPT <= 2 ? j : 0]);
        } else if constexpr (VPT <= 2) {
#pragma unroll
          for (int v = 0; v < VPT; ++v) y[VPT <= 2 ? j : 0][v] = 0.f;
        }
      }
    }
    rr.release(c);
    if constexpr (VPT <= 2) {
      spread_tokens<KL, VPT>(y, kl);
      if (kl < m) store_cols<VPT>(p.out + ((size_t)(r0 + t0 + kl) * p.heads + h) * dv + col, y[0], col, dv, vec);
    }
  }
  if (ok && !(p.no_store != nullptr && p.no_store[b])) store_state<KL, R, VPT>(S, st, kl, col, dk, dv, vec);
}

// sums of y[token][column] over the KL (8 or 16) lanes of a column, the 4 tokens spread over them: lane kl ends with token kl % 4 in y[0]
template <int KL, int VPT>
__device__ __forceinline__ void spread_block(float (&y)[kBlockTok][VPT], int kl) {
  const bool u2 = kl & 2, u1 = kl & 1;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    float z[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) z[j] = (u2 ? y[j + 2][v] : y[j][v]) + __shfl_xor_sync(0xffffffffu, u2 ? y[j][v] : y[j + 2][v], 2);
    y[0][v] = (u1 ? z[1] : z[0]) + __shfl_xor_sync(0xffffffffu, u1 ? z[0] : z[1], 1);
#pragma unroll
    for (int o = 4; o < KL; o <<= 1) y[0][v] += __shfl_xor_sync(0xffffffffu, y[0][v], o);
  }
}

// long runs with one decay per head, four tokens at a time (see delta_block_records_kernel)
template <typename T, int KL, int R, int VPT>
__global__ void __launch_bounds__((kRecWarps + 1) * 32, R * VPT <= 64 ? 2 : 1) delta_block_kernel(RecParams p, int slices, int vec_v) {
  constexpr int DKP = R * KL, CG = 32 / KL, COLS = kRecWarps * CG * VPT, REC = 2 * DKP + kBlockCoef, STAGE = kRecTok * REC;
  constexpr bool KEEP_K = R <= 8;                   // registers for the block's keys
  constexpr int VC = sizeof(T) * VPT < 4 ? 2 : VPT; // v columns that a lane brings: at least 4 bytes
  extern __shared__ __align__(128) uint8_t sm8[];
  __shared__ __align__(16) T s_v[kRecWarps][kColsAhead + 1][kRecTok][CG * VC];
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n < p.long_rows) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % KL, cg = lane / KL;
  const int groups = (n + kRecTok - 1) / kRecTok;
  float* ring = reinterpret_cast<float*>(sm8 + kRecHead);
  RecRing rr;
  rr.init(sm8, p.status);
  if (warp == kRecWarps) {
    if (lane == 0) {
      const float* src = p.records + ((size_t)h * p.T + r0) * REC;
      rr.produce(groups, [&](int c) {
        const uint32_t bytes = (uint32_t)min(kRecTok, n - c * kRecTok) * REC * 4;
        mbar_expect_tx(&rr.full[c % kRecStages], bytes);
        bulk_load(ring + (c % kRecStages) * STAGE, src + (size_t)c * STAGE, bytes, &rr.full[c % kRecStages]);
      });
    }
    return;
  }
  const int dk = p.dk, dv = p.dv, col = slice * COLS + warp * CG * VPT + cg * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * dk * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT];
  load_state<KL, R, VPT>(S, st, kl, col, dk, dv, ctx == n, vec);
  const int vcol = VC > VPT ? col & ~1 : col;
  const T* vsrc = reinterpret_cast<const T*>(p.conv) + (size_t)(r0 + (kl & 7)) * p.ld_conv + (size_t)2 * p.groups * dk + (size_t)h * dv + vcol;
  auto send_group = [&](int c) {
    send_cols<T, VC>(&s_v[warp][c % (kColsAhead + 1)][kl & 7][cg * VC], vsrc + (size_t)c * kRecTok * p.ld_conv,
                     kl < kRecTok && c * kRecTok + kl < n, vcol, dv, vec_v);
  };
#pragma unroll
  for (int c = 0; c < kColsAhead; ++c) send_group(c);
  const int mine = kl & (kBlockTok - 1), quad = lane & ~(kBlockTok - 1);
  bool ok = true;
  for (int c = 0; c < groups; ++c) {
    const int t0 = c * kRecTok;
    __syncwarp();                            // the last group's columns have been read
    send_group(c + kColsAhead);
    wait_cols();
    const T(*cols)[CG * VC] = s_v[warp][c % (kColsAhead + 1)];
    ok = rr.wait_full(c);
    if (!ok) break;
    __syncwarp();
    const float* buf = ring + (c % kRecStages) * STAGE;
    auto block = [&](int j0, int m, auto whole) {
      constexpr bool WHOLE = decltype(whole)::value;       // m == kBlockTok
      const float* rec = buf + j0 * REC;
      float pk[kBlockTok][VPT], pq[kBlockTok][VPT];
      [[maybe_unused]] float kr[KEEP_K ? kBlockTok : 1][R];
#pragma unroll
      for (int j = 0; j < kBlockTok; ++j) {
#pragma unroll
        for (int v = 0; v < VPT; ++v) pk[j][v] = pq[j][v] = 0.f;
        if (!WHOLE && j >= m) continue;
#pragma unroll
        for (int i4 = 0; i4 < R / 4; ++i4) {
          const float4 q4 = *reinterpret_cast<const float4*>(rec + j * REC + kl * 4 + 4 * KL * i4);
          const float4 k4 = *reinterpret_cast<const float4*>(rec + j * REC + DKP + kl * 4 + 4 * KL * i4);
          const float qa[4] = {q4.x, q4.y, q4.z, q4.w}, ka[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if constexpr (KEEP_K) kr[j][i4 * 4 + i] = ka[i];
#pragma unroll
            for (int v = 0; v < VPT; ++v) {
              pk[j][v] = fmaf(S[i4 * 4 + i][v], ka[i], pk[j][v]);
              pq[j][v] = fmaf(S[i4 * 4 + i][v], qa[i], pq[j][v]);
            }
          }
        }
      }
      spread_block<KL, VPT>(pk, kl);
      spread_block<KL, VPT>(pq, kl);
      // this lane's token of the block
      const int my = WHOLE ? mine : min(mine, m - 1);
      const float* cf = rec + my * REC + 2 * DKP;
      const float4 a4 = *reinterpret_cast<const float4*>(cf), c4 = *reinterpret_cast<const float4*>(cf + 4), s4 = *reinterpret_cast<const float4*>(cf + 8);
      const float a[4] = {a4.x, a4.y, a4.z, a4.w}, cc[4] = {c4.x, c4.y, c4.z, c4.w};
      float u[VPT], o[VPT], uu[kBlockTok][VPT];
#pragma unroll
      for (int v = 0; v < VPT; ++v) {
        u[v] = fmaf(s4.x, rc_ld(&cols[j0 + my][cg * VC + (VC > VPT ? col & 1 : v)]), -s4.y * pk[0][v]);
        o[v] = s4.z * pq[0][v];
      }
#pragma unroll
      for (int j = 0; j < kBlockTok; ++j) {
        if (!WHOLE && j >= m) break;
        const float to_end = rec[j * REC + 2 * DKP + 11];
#pragma unroll
        for (int v = 0; v < VPT; ++v) {
          const float x = __shfl_sync(0xffffffffu, u[v], quad | j);
          u[v] = fmaf(-a[j], x, u[v]);
          o[v] = fmaf(cc[j], x, o[v]);
          uu[j][v] = to_end * x;
        }
      }
      if (kl < m) store_cols<VPT>(p.out + ((size_t)(r0 + t0 + j0 + kl) * p.heads + h) * dv + col, o, col, dv, vec);
      const float all = rec[2 * DKP + 12];
#pragma unroll
      for (int i = 0; i < R; ++i)
#pragma unroll
        for (int v = 0; v < VPT; ++v) S[i][v] *= all;
#pragma unroll
      for (int j = 0; j < kBlockTok; ++j) {
        if (!WHOLE && j >= m) break;
#pragma unroll
        for (int i4 = 0; i4 < R / 4; ++i4) {
          float ka[4];
          if constexpr (KEEP_K) {
#pragma unroll
            for (int i = 0; i < 4; ++i) ka[i] = kr[j][i4 * 4 + i];
          } else {
            const float4 k4 = *reinterpret_cast<const float4*>(rec + j * REC + DKP + kl * 4 + 4 * KL * i4);
            ka[0] = k4.x; ka[1] = k4.y; ka[2] = k4.z; ka[3] = k4.w;
          }
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int v = 0; v < VPT; ++v) S[i4 * 4 + i][v] = fmaf(ka[i], uu[j][v], S[i4 * 4 + i][v]);
        }
      }
    };
    const int m = min(kRecTok, n - t0);
#pragma unroll
    for (int j0 = 0; j0 < kRecTok; j0 += kBlockTok) {
      if (m >= j0 + kBlockTok) block(j0, kBlockTok, Whole{});
      else if (m > j0) block(j0, m - j0, Part{});
    }
    rr.release(c);
  }
  if (ok && !(p.no_store != nullptr && p.no_store[b])) store_state<KL, R, VPT>(S, st, kl, col, dk, dv, vec);
}

template <typename T, int KL, int R, int VPT, bool G>
__global__ void __launch_bounds__((kRecWarps + 1) * 32, R * VPT <= 64 ? 2 : 1) state_space_stream_kernel(RecParams p, int slices, int vec_v) {
  constexpr int NP = R * KL, CG = 32 / KL, COLS = kRecWarps * CG * VPT, REC = 2 * NP, STEPS = G ? 0 : 4, STAGE = kRecTok * (REC + STEPS);
  extern __shared__ __align__(128) uint8_t sm8[];
  __shared__ __align__(16) T s_v[kRecWarps][kColsAhead + 1][kRecTok][CG * VPT];
  const int b = blockIdx.x / slices, slice = blockIdx.x % slices, h = blockIdx.y;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, slot = p.slots[b], ctx = p.ctx_len[b];
  if (n < p.long_rows) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % KL, cg = lane / KL;
  const int groups = (n + kRecTok - 1) / kRecTok;
  float* ring = reinterpret_cast<float*>(sm8 + kRecHead);
  RecRing rr;
  rr.init(sm8, p.status);
  if (warp == kRecWarps) {
    if (lane == 0) {
      const float* src = p.records + ((size_t)(h / (p.heads / p.groups)) * p.T + r0) * REC;
      const float* steps = p.records + (size_t)p.groups * p.T * REC + ((size_t)h * p.T + r0) * 4;
      rr.produce(groups, [&](int c) {
        const uint32_t m = (uint32_t)min(kRecTok, n - c * kRecTok);
        float* dst = ring + (c % kRecStages) * STAGE;
        mbar_expect_tx(&rr.full[c % kRecStages], m * (REC + STEPS) * 4);
        bulk_load(dst, src + (size_t)c * kRecTok * REC, m * REC * 4, &rr.full[c % kRecStages]);
        if constexpr (!G) bulk_load(dst + kRecTok * REC, steps + (size_t)c * kRecTok * 4, m * 16, &rr.full[c % kRecStages]);
      });
    }
    return;
  }
  const int N = p.dk, dv = p.dv, col = slice * COLS + warp * CG * VPT + cg * VPT;
  float* st = p.state + ((size_t)slot * p.heads + h) * N * dv;
  const bool vec = dv % 4 == 0;
  float S[R][VPT];
  load_state<KL, R, VPT>(S, st, kl, col, N, dv, ctx == n, vec);
  const float D = !G && p.D ? p.D[h] : 0.f;
  const T* vsrc = reinterpret_cast<const T*>(p.conv) + (size_t)(r0 + (kl & 7)) * p.ld_conv + (size_t)h * dv + col;
  auto send_group = [&](int c) {
    send_cols<T, VPT>(&s_v[warp][c % (kColsAhead + 1)][kl & 7][cg * VPT], vsrc + (size_t)c * kRecTok * p.ld_conv,
                      kl < kRecTok && c * kRecTok + kl < n, col, dv, vec_v);
  };
#pragma unroll
  for (int c = 0; c < kColsAhead; ++c) send_group(c);
  bool ok = true;
  for (int c = 0; c < groups; ++c) {
    const int t0 = c * kRecTok, m = min(kRecTok, n - t0);
    __syncwarp();                            // the last group's columns have been read
    send_group(c + kColsAhead);
    wait_cols();
    const T(*cols)[CG * VPT] = s_v[warp][c % (kColsAhead + 1)];
    ok = rr.wait_full(c);
    if (!ok) break;
    __syncwarp();
    const float* buf = ring + (c % kRecStages) * STAGE;
    float y[kRecTok][VPT];
    struct Tok {
      float b[R], c[R], x[VPT], dec;
    };
    auto fetch = [&](int j, Tok& o) {
      const float* s = buf + j * REC;
#pragma unroll
      for (int i4 = 0; i4 < R / 4; ++i4) {
        const float4 b4 = *reinterpret_cast<const float4*>(s + kl * 4 + 4 * KL * i4);
        const float4 c4 = *reinterpret_cast<const float4*>(s + NP + kl * 4 + 4 * KL * i4);
        o.b[i4 * 4] = b4.x; o.b[i4 * 4 + 1] = b4.y; o.b[i4 * 4 + 2] = b4.z; o.b[i4 * 4 + 3] = b4.w;
        o.c[i4 * 4] = c4.x; o.c[i4 * 4 + 1] = c4.y; o.c[i4 * 4 + 2] = c4.z; o.c[i4 * 4 + 3] = c4.w;
      }
      const float2 step = G ? make_float2(1.f, 0.f) : *reinterpret_cast<const float2*>(buf + kRecTok * REC + j * 4);      // dt, decay
      o.dec = step.y;
#pragma unroll
      for (int v = 0; v < VPT; ++v) o.x[v] = step.x * rc_ld(&cols[j][cg * VPT + v]);
    };
    auto token = [&](int j, const Tok& k) {
#pragma unroll
      for (int v = 0; v < VPT; ++v) y[j][v] = 0.f;
#pragma unroll
      for (int i = 0; i < R; ++i)
#pragma unroll
        for (int v = 0; v < VPT; ++v) {
          S[i][v] = G ? fmaf(S[i][v], k.b[i], (1.f - k.b[i]) * k.x[v]) : fmaf(S[i][v], k.dec, k.b[i] * k.x[v]);
          y[j][v] = fmaf(S[i][v], k.c[i], y[j][v]);
        }
    };
    if (m == kRecTok) {
      Tok tok[2];                            // the next token's operands are fetched before this one's are used
      fetch(0, tok[0]);
#pragma unroll
      for (int j = 0; j < kRecTok; ++j) {
        if (j + 1 < kRecTok) fetch(j + 1, tok[(j + 1) & 1]);
        token(j, tok[j & 1]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < kRecTok; ++j) {
        if (j < m) {
          Tok tok;
          fetch(j, tok);
          token(j, tok);
        } else {
#pragma unroll
          for (int v = 0; v < VPT; ++v) y[j][v] = 0.f;
        }
      }
    }
    rr.release(c);
    spread_tokens<KL, VPT>(y, kl);
#pragma unroll
    for (int v = 0; v < VPT && !G; ++v) y[0][v] = fmaf(D, rc_ld(&cols[kl & 7][cg * VPT + v]), y[0][v]);
    if (kl < m) store_cols<VPT>(p.out + ((size_t)(r0 + t0 + kl) * p.heads + h) * dv + col, y[0], col, dv, vec);
  }
  if (ok && !(p.no_store != nullptr && p.no_store[b])) store_state<KL, R, VPT>(S, st, kl, col, N, dv, vec);
}

// ------------------------------------------------------------------------------------------ norm over groups with a gate
struct GroupNormParams {
  const float* o;              // [T, groups * n]
  const void* z;               // gate inputs [T, ldz] or null
  const float* w;              // [w_period]: the weight of a column is w[column % w_period]
  void* out;                   // [T, ld_out]
  long long ldz, ld_out;
  int T, groups, n, w_period;
  int sigmoid;                 // gate: sigmoid(z), else silu(z)
  int gate_first;              // the gate multiplies before the norm, else after it
  int vec;                     // rows and pointers allow 4 columns at a time
  float eps, post;             // everything times post at the end
};

template <typename T>
__device__ __forceinline__ float gate_of(float z, int sigmoid) {
  const float s = rc_sigmoid<T>(z);
  return sigmoid ? s : z * s;
}
template <typename T, int VEC>
__device__ __forceinline__ void gn_load(const GroupNormParams& p, const float* o, const T* z, int c, float (&x)[VEC], float (&g)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(o + c);
    x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
  } else {
    x[0] = o[c];
  }
#pragma unroll
  for (int j = 0; j < VEC; ++j) g[j] = 1.f;
  if (z) {
    T e[VEC];
    if constexpr (VEC == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(e) = *reinterpret_cast<const uint2*>(z + c);
    else if constexpr (VEC == 4) *reinterpret_cast<float4*>(e) = *reinterpret_cast<const float4*>(z + c);
    else e[0] = z[c];
#pragma unroll
    for (int j = 0; j < VEC; ++j) g[j] = gate_of<T>(rc_ld(e + j), p.sigmoid);
  }
}

// a group of columns per WARPS warps
template <typename T, int WARPS, int VEC>
__global__ void __launch_bounds__(256) group_norm_kernel(GroupNormParams p) {
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long unit = WARPS == 1 ? (long long)blockIdx.x * 8 + warp : blockIdx.x;
  if (unit >= (long long)p.T * p.groups) return;
  const int t = (int)(unit / p.groups), g = (int)(unit % p.groups), i0 = (WARPS == 1 ? lane : (int)threadIdx.x) * VEC;
  constexpr int STEP = WARPS * 32 * VEC;
  const float* o = p.o + (size_t)unit * p.n;
  const T* z = p.z ? reinterpret_cast<const T*>(p.z) + (size_t)t * p.ldz + (size_t)g * p.n : nullptr;
  float ss = 0.f;
  constexpr int KEEP = VEC == 4 ? 4 : 1;             // columns of this many turns stay in registers
  float kx[KEEP][VEC], kg[KEEP][VEC];
  if (p.n <= KEEP * STEP) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = i0 + i * STEP;
      if (c < p.n) gn_load<T, VEC>(p, o, z, c, kx[i], kg[i]);
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
      if (i0 + i * STEP < p.n)
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          const float x = p.gate_first ? kx[i][j] * kg[i][j] : kx[i][j];
          ss = fmaf(x, x, ss);
        }
  } else {
    for (int c = i0; c < p.n; c += STEP) {
      float x[VEC], gt[VEC];
      gn_load<T, VEC>(p, o, p.gate_first ? z : nullptr, c, x, gt);
#pragma unroll
      for (int j = 0; j < VEC; ++j) { x[j] *= gt[j]; ss = fmaf(x[j], x[j], ss); }
    }
  }
  ss = warp_sum(ss);
  if constexpr (WARPS > 1) {
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) ss += red[i];
  }
  const float f = p.post / sqrtf(ss / (float)p.n + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)g * p.n;
  auto put = [&](int c, const float (&x)[VEC], const float (&gt)[VEC]) {
    const int wc = (int)(((long long)g * p.n + c) % p.w_period);
    T e[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const float v = x[j] * (f * gt[j] * p.w[VEC == 1 ? wc : wc + j]);
      if constexpr (sizeof(T) == 4) e[j] = v;
      else e[j] = __float2bfloat16(v);
    }
    if constexpr (VEC == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(out + c) = *reinterpret_cast<uint2*>(e);
    else if constexpr (VEC == 4) *reinterpret_cast<float4*>(out + c) = *reinterpret_cast<float4*>(e);
    else out[c] = e[0];
  };
  if (p.n <= KEEP * STEP) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
      if (i0 + i * STEP < p.n) put(i0 + i * STEP, kx[i], kg[i]);
  } else {
    for (int c = i0; c < p.n; c += STEP) {
      float x[VEC], gt[VEC];
      gn_load<T, VEC>(p, o, z, c, x, gt);
      put(c, x, gt);
    }
  }
}

// ------------------------------------------------------------------------------------------ minGRU
struct GruParams {
  const void *z, *u, *g;       // [T, ld] before their activations
  float* state;                // [rows, width]
  void* out;                   // [T, ld_out] or null (the state only)
  const int *slots, *q_start, *ctx_len, *no_store;
  long long ld, ld_out;
  int width;
  float2* pairs;               // [B][parts][width]: of each part of a run, the factor of the state before it and the addend; of the first
                               // part the addend alone, with the state before the run in it; or null (a block takes a whole run)
  float* before;               // [B][width]: the states before the runs (with pairs)
  int part, parts;             // tokens per part, parts of the longest run
};
static constexpr int kGruWarps = 8, kGruTok = 8;       // a block takes kGruWarps * kGruTok tokens at a time
static constexpr int kGruPart = 512;

// a gate; bf16: the special function unit's reciprocal (two units in the last place)
template <typename T>
__device__ __forceinline__ float gru_sigmoid(float x) {
  if constexpr (sizeof(T) == 4) return 1.f / (1.f + expf(-x));
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x * -1.4426950408889634f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + r));
  return r;
}
template <typename T>
__device__ __forceinline__ void gru_gate(float z, float u, float& keep, float& add) {
  const float s = gru_sigmoid<T>(z), c = gru_sigmoid<T>(u);
  keep = 1.f - s;
  add = s * (u >= 0.f ? u + 0.5f : c);
}
template <typename T, int VEC> struct alignas(sizeof(T) * VEC) GruVec { T e[VEC]; };
template <typename T, int VEC>
__device__ __forceinline__ GruVec<T, VEC> gru_load(const void* base, size_t at) {
  GruVec<T, VEC> v;
  const T* p = reinterpret_cast<const T*>(base) + at;
  if constexpr (sizeof(T) * VEC == 16) *reinterpret_cast<uint4*>(v.e) = *reinterpret_cast<const uint4*>(p);
  else if constexpr (sizeof(T) * VEC == 8) *reinterpret_cast<uint2*>(v.e) = *reinterpret_cast<const uint2*>(p);
  else if constexpr (sizeof(T) * VEC == 4) *reinterpret_cast<uint32_t*>(v.e) = *reinterpret_cast<const uint32_t*>(p);
  else v.e[0] = *p;
  return v;
}
// vec: the output's rows allow VEC elements as one word; left: elements of the row from c on
template <typename T, int VEC>
__device__ __forceinline__ void gru_store(const GruParams& p, size_t row, int c, const GruVec<T, VEC>& g, const float (&S)[VEC], bool vec,
                                          int left = VEC) {
  T* o = reinterpret_cast<T*>(p.out) + row * p.ld_out + c;
  GruVec<T, VEC> y;
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const float x = rc_ld(g.e + j), v = S[j] * (x * gru_sigmoid<T>(x));
    if constexpr (sizeof(T) == 4) y.e[j] = v;
    else y.e[j] = __float2bfloat16(v);
  }
  if (vec && left >= VEC) {
    *reinterpret_cast<GruVec<T, VEC>*>(o) = y;
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j)
      if (j < left) o[j] = y.e[j];
  }
}

// single tokens: a thread per VEC elements of a sequence
template <typename T, int VEC>
__global__ void __launch_bounds__(128) min_gru_step_kernel(GruParams p, int vec) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * VEC;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0;
  if (n != 1 || c >= p.width) return;
  const size_t at = (size_t)r0 * p.ld + c;
  const auto z = gru_load<T, VEC>(p.z, at), u = gru_load<T, VEC>(p.u, at), g = gru_load<T, VEC>(p.g, at);
  float* st = p.state + (size_t)p.slots[b] * p.width + c;
  const bool fresh = p.ctx_len[b] == 1;
  float S[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    float keep, add;
    gru_gate<T>(rc_ld(z.e + j), rc_ld(u.e + j), keep, add);
    S[j] = fresh ? add : fmaf(keep, st[j], add);
  }
  if (p.out) gru_store<T, VEC>(p, r0, c, g, S, vec);
  if (p.no_store != nullptr && p.no_store[b]) return;
#pragma unroll
  for (int j = 0; j < VEC; ++j) st[j] = S[j];
}

// Runs: a block takes 128 bytes of a row's elements (VEC per lane) over a run, or over a part of it.  Rows come in tiles of kGruWarps *
// kGruTok tokens through a ring in shared memory.  Each warp folds its kGruTok tokens into one pair (factor, addend) per element; the pairs of
// the warps before it and the carry give the state its own tokens start from.  PAIRS: the carry is a pair itself and is all that is
// written (see GruParams::pairs); else the outputs and, by the last part, the state.
static constexpr int kGruStages = 3, kGruTile = kGruWarps * kGruTok;

template <typename T, bool PAIRS>
__global__ void __launch_bounds__(kGruWarps * 32, 3) min_gru_kernel(GruParams p, int vec, int vec_o) {
  constexpr int VEC = 4 / sizeof(T), COLS = 32 * VEC, ARRS = PAIRS ? 2 : 3, CHUNK = 16 / sizeof(T);
  extern __shared__ __align__(128) uint8_t sm8[];                // [stages][z | u | g][tile][COLS]
  __shared__ float2 s_p[kGruWarps][COLS], s_c[2][COLS];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c0 = blockIdx.x * COLS, c = c0 + lane * VEC;
  const int r0 = p.q_start[b], n = p.q_start[b + 1] - r0, from = blockIdx.z * p.part, to = min(n, from + p.part);
  if (n <= 1 || from >= n) return;
  T* ring = reinterpret_cast<T*>(sm8);
  const int tiles = (to - from + kGruTile - 1) / kGruTile;
  auto fill = [&](int i) {
    if (i < tiles) {
      T* dst = ring + (size_t)(i % kGruStages) * ARRS * kGruTile * COLS;
      for (int x = threadIdx.x; x < ARRS * kGruTile * 8; x += kGruWarps * 32) {
        const int part = x & 7, row = x >> 3, t = from + i * kGruTile + row % kGruTile, a = row / kGruTile, col = c0 + part * CHUNK;
        const T* src = reinterpret_cast<const T*>(a == 0 ? p.z : a == 1 ? p.u : p.g) + (size_t)(r0 + min(t, to - 1)) * p.ld + col;
        T* at = dst + row * COLS + part * CHUNK;
        if (vec) {
          const int bytes = t < to ? max(min((p.width - col) * (int)sizeof(T), 16), 0) : 0;
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(at)), "l"(bytes ? (const void*)src : p.z), "r"(bytes) : "memory");
        } else {
#pragma unroll
          for (int e = 0; e < CHUNK; ++e)
            if (t < to && col + e < p.width) at[e] = src[e];
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < kGruStages; ++i) fill(i);
  const bool live = c < p.width;
  float* st = p.state + (size_t)p.slots[b] * p.width + c;
  const bool fresh = p.ctx_len[b] == n;
  if (warp == 0) {
    // the carry: of a part's pair the state before the run in its addend, or nothing; else the state
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      float S = 0.f;
      if (c + j < p.width) {
        if (PAIRS || !p.pairs) {
          if (blockIdx.z == 0 && !fresh) S = st[j];
          if (PAIRS && blockIdx.z == 0) p.before[(size_t)b * p.width + c + j] = S;
        } else if (blockIdx.z == 0) {
          S = p.before[(size_t)b * p.width + c + j];
        } else {
          const float2* pr = p.pairs + (size_t)b * p.parts * p.width + c + j;
          S = pr->y;
#pragma unroll 8
          for (int i = 1; i < blockIdx.z; ++i) {
            const float2 f = pr[(size_t)i * p.width];
            S = fmaf(f.x, S, f.y);
          }
        }
      }
      s_c[0][lane * VEC + j] = make_float2(1.f, S);
    }
  }
  float S[VEC];
  for (int i = 0; i < tiles; ++i) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kGruStages - 1) : "memory");
    __syncthreads();
    const T* tile = ring + (size_t)(i % kGruStages) * ARRS * kGruTile * COLS + (size_t)warp * kGruTok * COLS + lane * VEC;
    const int t0 = from + i * kGruTile + warp * kGruTok;
    float keep[kGruTok][VEC], add[kGruTok][VEC], A[VEC], B[VEC];
    GruVec<T, VEC> gate[PAIRS ? 1 : kGruTok];
#pragma unroll
    for (int j = 0; j < VEC; ++j) { A[j] = 1.f; B[j] = 0.f; }
#pragma unroll
    for (int k = 0; k < kGruTok; ++k) {
      const GruVec<T, VEC> z = *reinterpret_cast<const GruVec<T, VEC>*>(tile + k * COLS), u = *reinterpret_cast<const GruVec<T, VEC>*>(tile + (kGruTile + k) * COLS);
      if constexpr (!PAIRS) gate[k] = *reinterpret_cast<const GruVec<T, VEC>*>(tile + (2 * kGruTile + k) * COLS);
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        gru_gate<T>(rc_ld(z.e + j), rc_ld(u.e + j), keep[k][j], add[k][j]);
        if (t0 + k >= to) { keep[k][j] = 1.f; add[k][j] = 0.f; }          // beyond the run: nothing changes
        A[j] *= keep[k][j];
        B[j] = fmaf(keep[k][j], B[j], add[k][j]);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) s_p[warp][lane * VEC + j] = make_float2(A[j], B[j]);
    __syncthreads();
    float2 carry[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) carry[j] = s_c[i & 1][lane * VEC + j];
#pragma unroll
    for (int w = 0; w < kGruWarps - 1; ++w)
      if (w < warp)
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          const float2 f = s_p[w][lane * VEC + j];
          carry[j] = make_float2(f.x * carry[j].x, fmaf(f.x, carry[j].y, f.y));
        }
    if (warp == kGruWarps - 1)               // the carry after these tokens, as soon as it is known
#pragma unroll
      for (int j = 0; j < VEC; ++j) s_c[(i + 1) & 1][lane * VEC + j] = make_float2(A[j] * carry[j].x, fmaf(A[j], carry[j].y, B[j]));
    fill(i + kGruStages);                    // every warp has read this tile
    if constexpr (!PAIRS) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) S[j] = carry[j].y;
#pragma unroll
      for (int k = 0; k < kGruTok; ++k) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) S[j] = fmaf(keep[k][j], S[j], add[k][j]);
        if (p.out && live && t0 + k < to) gru_store<T, VEC>(p, r0 + t0 + k, c, gate[k], S, vec_o, p.width - c);
      }
    }
  }
  if (warp != kGruWarps - 1 || !live) return;
  if constexpr (PAIRS) {
#pragma unroll
    for (int j = 0; j < VEC; ++j)
      if (c + j < p.width) p.pairs[((size_t)b * p.parts + blockIdx.z) * p.width + c + j] = s_c[tiles & 1][lane * VEC + j];
  } else if (to == n && !(p.no_store != nullptr && p.no_store[b])) {
#pragma unroll
    for (int j = 0; j < VEC; ++j)
      if (c + j < p.width) st[j] = S[j];     // tokens beyond the run changed nothing
  }
}

template <typename T>
static int run_gru(const GruParams& p, int B, int kinds, int vec, int vec16, int vec_o, cudaStream_t s) {
  cudaError_t e = cudaSuccess;
  if (kinds & 1) {
    constexpr int V = 4;
    if (vec) e = launch_pdl(min_gru_step_kernel<T, V>, dim3((p.width + 128 * V - 1) / (128 * V), B), dim3(128), 0, s, p, vec_o);
    else e = launch_pdl(min_gru_step_kernel<T, 1>, dim3((p.width + 127) / 128, B), dim3(128), 0, s, p, 0);
  }
  if (e == cudaSuccess && (kinds & 2)) {
    constexpr int COLS = 128 / sizeof(T);
    constexpr size_t tile = (size_t)kGruStages * kGruTile * 128;          // per array
    const dim3 grid((p.width + COLS - 1) / COLS, B, p.parts), block(kGruWarps * 32);
    static PerDeviceOnce once, once_pairs;
    if (p.pairs) {
      e = once_pairs.smem_limit(min_gru_kernel<T, true>, 2 * tile);
      if (e == cudaSuccess) e = launch_pdl(min_gru_kernel<T, true>, grid, block, 2 * tile, s, p, vec16, 0);
      if (e != cudaSuccess) return (int)e;
    }
    e = once.smem_limit(min_gru_kernel<T, false>, 3 * tile);
    if (e == cudaSuccess) e = launch_pdl(min_gru_kernel<T, false>, grid, block, 3 * tile, s, p, vec16, vec_o);
  }
  return (int)e;
}

// bf16: 4 neighbouring elements of the token's vectors can be read as one 64-bit word
static int words_of_four(const RecParams& p, RecKind kind) {
  auto ok = [](const void* q, long long ld) { return (reinterpret_cast<uintptr_t>(q) & 7) == 0 && ld % 4 == 0; };
  return ok(p.conv, p.ld_conv) && (kind == GATED || p.dk % 4 == 0) && p.dv % 4 == 0 && (kind != DELTA || ok(p.a, p.ld_a));      // HDELTA's are read one by one
}

template <typename T, int DKP, RecKind K>
static int launch_steps(const RecParams& p, int B, cudaStream_t s) {
  constexpr int KL = DKP <= 128 ? 8 : DKP / 16, R = DKP / KL, COLS = kRecWarps * (32 / KL) * 4;
  const int slices = (p.dv + COLS - 1) / COLS;
  auto kern = delta_step_kernel<T, KL, R, 4, K == HDELTA>;
  if constexpr (K == SSM) kern = state_space_step_kernel<T, KL, R, 4>;
  if constexpr (K == GATED) kern = gated_step_kernel<T, KL, R, 4>;
  kern<<<dim3(B * slices, p.heads), kRecWarps * 32, 0, s>>>(p, slices, words_of_four(p, K));
  return (int)cudaGetLastError();
}
template <typename T, int DKP, RecKind K>
static int launch_short_runs(const RecParams& p, int B, cudaStream_t s) {
  constexpr int R = DKP / 8, VPT = R > 32 ? 1 : (sizeof(T) == 4 || R > 16 ? 2 : 4), COLS = kRecWarps * 4 * VPT;
  const int slices = (p.dv + COLS - 1) / COLS;
  const size_t smem = (size_t)2 * kRecTok * ((K == DELTA ? 3 : 2) * DKP + COLS + 4) * 4;
  void (*kern)(RecParams, int);
  if constexpr (K == DELTA || K == HDELTA) kern = delta_rule_kernel<T, R, VPT, K == HDELTA>;
  else kern = state_space_kernel<T, R, VPT, K == GATED>;
  static PerDeviceOnce once;
  cudaError_t e = once.smem_limit(kern, 200 * 1024);
  if (e != cudaSuccess) return (int)e;
  kern<<<dim3(B * slices, p.heads), kRecWarps * 32, smem, s>>>(p, slices);
  return (int)cudaGetLastError();
}
template <typename T, int KL, int R, int VPT, RecKind K>
static int launch_stream(const RecParams& p, int B, cudaStream_t s) {
  constexpr int COLS = kRecWarps * (32 / KL) * VPT;
  const int slices = (p.dv + COLS - 1) / COLS;
  const size_t smem = kRecHead + (size_t)kRecStages * kRecTok * ((K == DELTA ? 3 : 2) * R * KL + (K == GATED ? 0 : K == HDELTA ? kBlockCoef : 4)) * 4;
  void (*kern)(RecParams, int, int);
  if constexpr (K == DELTA) kern = delta_stream_kernel<T, KL, R, VPT>;
  else if constexpr (K == HDELTA) kern = delta_block_kernel<T, KL, R, VPT>;
  else kern = state_space_stream_kernel<T, KL, R, VPT, K == GATED>;
  static PerDeviceOnce once;
  cudaError_t e = once.smem_limit(kern, 220 * 1024);
  if (e != cudaSuccess) return (int)e;
  kern<<<dim3(B * slices, p.heads), (kRecWarps + 1) * 32, smem, s>>>(p, slices, words_of_four(p, K));
  return (int)cudaGetLastError();
}
// 16 columns per warp keep the reductions and the shared-memory reads few; where that gives too few warps to fill the GPU, 4 columns
template <typename T, int DKP, RecKind K>
static int launch_long_runs(const RecParams& p, int B, cudaStream_t s) {
  const unsigned warps4 = (unsigned)(((long long)p.T * p.heads + 3) / 4);
  if constexpr (K == DELTA) delta_records_kernel<T, DKP><<<warps4, 128, 0, s>>>(p);
  else if constexpr (K == HDELTA)
    delta_block_records_kernel<T, DKP><<<(unsigned)(((long long)((p.T + kBlockTok - 1) / kBlockTok) * p.heads + 3) / 4), 128, 0, s>>>(p);
  else if constexpr (K == GATED) gated_records_kernel<T, DKP><<<warps4, 128, 0, s>>>(p);
  else state_space_records_kernel<T, DKP><<<p.T, 128, 0, s>>>(p);
  const int e = (int)cudaGetLastError();
  if (e) return e;
  if constexpr (sizeof(T) == 2 && DKP <= 128)
    if ((long long)B * p.heads * ((p.dv + 15) / 16) >= 4LL * sm_count()) return launch_stream<T, 8, DKP / 8, 4, K>(p, B, s);
  constexpr int KL = DKP >= 64 ? 16 : 8;
  if constexpr (sizeof(T) == 2 && K != DELTA && K != HDELTA && DKP <= 128)     // no reduction between tokens: 8 columns already at half the warps
    if ((long long)B * p.heads * ((p.dv + 7) / 8) >= 2LL * sm_count()) return launch_stream<T, KL, DKP / KL, 4, K>(p, B, s);
  return launch_stream<T, KL, DKP / KL, 2, K>(p, B, s);
}

// kinds: which sequences the step has, bit 0 = single tokens, 1 = short runs, 2 = long runs (with a workspace)
template <typename T, int DKP, RecKind K>
static int run_width(RecParams p, int B, int kinds, cudaStream_t s) {
  int e = 0;
  if (kinds & 1) e = launch_steps<T, DKP, K>(p, B, s);
  if (!e && (kinds & 4)) e = launch_long_runs<T, DKP, K>(p, B, s);
  else p.long_rows = 0x7fffffff;
  if (!e && (kinds & 2)) e = launch_short_runs<T, DKP, K>(p, B, s);
  return e;
}

static int padded_dk(int dk) { return dk <= 32 ? 32 : dk <= 64 ? 64 : dk <= 128 ? 128 : dk <= 256 ? 256 : 512; }
static long long record_bytes(RecKind kind, long long T, int heads, int groups, int dk) {
  const long long n = padded_dk(dk);
  return 4 * (kind == DELTA ? heads * T * (3 * n + 4) : kind == HDELTA ? heads * T * (2 * n + kBlockCoef) : kind == GATED ? heads * T * 2 * n : groups * T * 2 * n + heads * T * 4);
}

template <typename T, RecKind K>
static int run_rec(const RecParams& p, int B, int kinds, long long ws_bytes, cudaStream_t s) {
  if (B == 0) return 0;
  if (B < 0 || p.heads < 1 || p.heads > 65535 || p.groups < 1 || p.heads % p.groups || p.dk < 1 || p.dk > 512 || p.dv < 1)
    return (int)cudaErrorInvalidValue;
  if ((kinds & 4) && (!p.records || !p.out || !p.seq_of_row || p.T < 1 || ws_bytes < record_bytes(K, p.T, p.heads, p.groups, p.dk) ||
                      (reinterpret_cast<uintptr_t>(p.records) & 15)))
    return (int)cudaErrorInvalidValue;
  switch (padded_dk(p.dk)) {
    case 32: return run_width<T, 32, K>(p, B, kinds, s);
    case 64: return run_width<T, 64, K>(p, B, kinds, s);
    case 128: return run_width<T, 128, K>(p, B, kinds, s);
    case 256: return run_width<T, 256, K>(p, B, kinds, s);
    default: return run_width<T, 512, K>(p, B, kinds, s);
  }
}

}  // namespace blz

// Runs of at least this many new tokens are long runs where the caller gives a workspace.
static constexpr int kLongRows = 32;
BLZ_API int blz_rec_long_rows() { return kLongRows; }
// Workspace bytes of a step of T rows (kind: 0 = blz_state_space, 1 = blz_delta_rule, 2 = blz_gated_linear, 3 = blz_delta_rule with one
// decay per head).
BLZ_API long long blz_rec_ws_bytes(int kind, int T, int heads, int groups, int dk) {
  return blz::record_bytes(kind == 1 ? blz::DELTA : kind == 2 ? blz::GATED : kind == 3 ? blz::HDELTA : blz::SSM, T, heads, groups, dk);
}

// Delta rule with channel decays over every sequence of the batch (see RecParams; leading dimensions in elements; conv channels
// [q key_heads * dk | k key_heads * dk | v heads * dv]).  out fp32 [T, heads * dv] or null.  no_store: optional [B], 1 = leave the
// state as it was.  kinds: the sequences with one new token (bit 0), with up to blz_rec_long_rows (bit 1), with more (bit 2, which
// needs out and the workspace ws of blz_rec_ws_bytes; without that bit they count as bit 1's).  dk <= 512.  per_head: one decay per head.
BLZ_API int blz_delta_rule(const void* conv, long long ld_conv, const void* a, long long ld_a, const void* b, long long ld_b, const float* A,
                           const float* dt_bias, float* state, float* out, const int* slots, const int* q_start, const int* ctx_len,
                           const int* no_store, int B, int heads, int key_heads, int dk, int dv, int per_head, const int* seq_of_row, int T,
                           int kinds, float* ws, long long ws_bytes, int f32, cudaStream_t s) {
  using namespace blz;
  const RecParams p = {conv, a, b, A, dt_bias, nullptr, state, out, slots, q_start, ctx_len, no_store, ld_conv, ld_a, ld_b, heads, key_heads,
                       dk, dv, seq_of_row, ws, T, kLongRows, status_word()};
  if (per_head)
    return f32 ? run_rec<float, HDELTA>(p, B, kinds, ws_bytes, s) : run_rec<__nv_bfloat16, HDELTA>(p, B, kinds, ws_bytes, s);
  return f32 ? run_rec<float, DELTA>(p, B, kinds, ws_bytes, s) : run_rec<__nv_bfloat16, DELTA>(p, B, kinds, ws_bytes, s);
}

// State-space duality (conv channels [x heads * dv | B groups * N | C groups * N]); other arguments as above.  N <= 512.
BLZ_API int blz_state_space(const void* conv, long long ld_conv, const void* dt, long long ld_dt, const float* A, const float* dt_bias,
                            const float* D, float* state, float* out, const int* slots, const int* q_start, const int* ctx_len,
                            const int* no_store, int B, int heads, int groups, int N, int dv, const int* seq_of_row, int T, int kinds,
                            float* ws, long long ws_bytes, int f32, cudaStream_t s) {
  using namespace blz;
  const RecParams p = {conv, dt, nullptr, A, dt_bias, D, state, out, slots, q_start, ctx_len, no_store, ld_conv, ld_dt, 0, heads, groups,
                       N, dv, seq_of_row, ws, T, kLongRows, status_word()};
  return f32 ? run_rec<float, SSM>(p, B, kinds, ws_bytes, s) : run_rec<__nv_bfloat16, SSM>(p, B, kinds, ws_bytes, s);
}

// Gated linear attention: q and f_raw [T, heads * dk], v [T, heads * dv] (runs of columns), lower bounds and biases [heads * dk] fp32;
// other arguments as above.  dk <= 512.
BLZ_API int blz_gated_linear(const void* q, long long ld_q, const void* f, long long ld_f, const void* v, long long ld_v, const float* lower,
                             const float* bias, float* state, float* out, const int* slots, const int* q_start, const int* ctx_len,
                             const int* no_store, int B, int heads, int dk, int dv, const int* seq_of_row, int T, int kinds, float* ws,
                             long long ws_bytes, int f32, cudaStream_t s) {
  using namespace blz;
  const RecParams p = {v, f, q, lower, bias, nullptr, state, out, slots, q_start, ctx_len, no_store, ld_v, ld_f, ld_q, heads, heads,
                       dk, dv, seq_of_row, ws, T, kLongRows, status_word()};
  return f32 ? run_rec<float, GATED>(p, B, kinds, ws_bytes, s) : run_rec<__nv_bfloat16, GATED>(p, B, kinds, ws_bytes, s);
}

// Workspace bytes of blz_min_gru for B sequences with up to max_q new tokens (0: none is needed): few long runs are cut into parts.
BLZ_API long long blz_min_gru_ws_bytes(int B, int max_q, int width) {
  using namespace blz;
  const long long blocks = (long long)B * ((width + 63) / 64), parts = (max_q + kGruPart - 1) / kGruPart;
  return parts < 2 || parts > 65535 || blocks >= sm_count() ? 0 : (long long)B * width * (parts * 8 + 4);
}

// minGRU over every sequence of the batch: gate inputs z, candidates u and output gates g [T, ld] (runs of columns, width each), state
// [rows][width] fp32; out [T, ld_out] (activation type) or null.  kinds: bit 0 = some sequences have one new token, bit 1 = some have more
// (max_q at most).  ws: blz_min_gru_ws_bytes, or null.
BLZ_API int blz_min_gru(const void* z, const void* u, const void* g, long long ld, float* state, void* out, long long ld_out, const int* slots,
                        const int* q_start, const int* ctx_len, const int* no_store, int B, int width, int max_q, int kinds, void* ws, int f32,
                        cudaStream_t s) {
  using namespace blz;
  if (B == 0) return 0;
  if (B < 0 || B > 65535 || width < 1 || max_q < 1 || !z || !u || !g || !state || (reinterpret_cast<uintptr_t>(ws) & 7))
    return (int)cudaErrorInvalidValue;
  GruParams p = {z, u, g, state, out, slots, q_start, ctx_len, no_store, ld, ld_out, width, nullptr, nullptr, max_q, 1};
  if (ws) {
    p.part = kGruPart;
    p.parts = (max_q + kGruPart - 1) / kGruPart;
    p.pairs = reinterpret_cast<float2*>(ws);
    p.before = reinterpret_cast<float*>(p.pairs + (size_t)B * p.parts * width);
    if (p.parts > 65535) return (int)cudaErrorInvalidValue;
  }
  const uintptr_t bits = reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(g);
  const int unit = f32 ? 16 : 8, vec = bits % unit == 0 && ld % 4 == 0 && width % 4 == 0, vec16 = bits % 16 == 0 && ld % (f32 ? 4 : 8) == 0;
  const int vec_o = reinterpret_cast<uintptr_t>(out) % unit == 0 && ld_out % 4 == 0;
  return f32 ? run_gru<float>(p, B, kinds, vec, vec16, vec_o, s) : run_gru<__nv_bfloat16>(p, B, kinds, vec, vec16, vec_o, s);
}

// RMS norm of each of `groups` runs of n columns of fp32 rows, with a gate (GroupNormParams), to the activation type.
BLZ_API int blz_group_norm(const float* o, const void* z, long long ldz, const float* w, void* out, long long ld_out, int T, int groups,
                           int n, int w_period, float eps, float post, int sigmoid, int gate_first, int f32, cudaStream_t s) {
  using namespace blz;
  if (T <= 0 || groups < 1 || n < 1 || w_period < 1) return (int)cudaErrorInvalidValue;
  const int esz = f32 ? 4 : 2;
  auto ok = [&](const void* q, long long ld) { return (reinterpret_cast<uintptr_t>(q) % (4 * esz)) == 0 && ld % 4 == 0; };
  const int vec = n % 4 == 0 && w_period % 4 == 0 && (reinterpret_cast<uintptr_t>(o) & 15) == 0 && (!z || ok(z, ldz)) && ok(out, ld_out);
  const GroupNormParams p = {o, z, w, out, ldz, ld_out, T, groups, n, w_period, sigmoid, gate_first, vec, eps, post};
  const long long units = (long long)T * groups;
  const bool wide = n > 1024 || (n > 128 && units < 8LL * sm_count());        // a block per group, else a warp
  const dim3 grid((unsigned)(wide ? units : (units + 7) / 8));
#define BLZ_GN(TT, V) return (int)(wide ? launch_pdl(group_norm_kernel<TT, 8, V>, grid, dim3(256), 0, s, p) \
                                        : launch_pdl(group_norm_kernel<TT, 1, V>, grid, dim3(256), 0, s, p))
  if (f32) { if (vec) { BLZ_GN(float, 4); } BLZ_GN(float, 1); }
  if (vec) { BLZ_GN(__nv_bfloat16, 4); }
  BLZ_GN(__nv_bfloat16, 1);
#undef BLZ_GN
}
