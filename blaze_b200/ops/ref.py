"""Plain PyTorch reference of every fused op (the oracle for the CUDA kernels; also the CPU path).

Semantics follow the reference's kernels: RMSNorm with the residual add rounded to the activation
dtype before the norm and optional zero-centred weights (``kernels/src/cuda/ops_basic.cu:42-67``);
per-head q/k RMSNorm + NeoX rotary on the first ``rotary_dim`` dims, optional ``[q | gate]`` row
layout (``ops_basic.cu:95-164``); softmax → top-k → renormalise routing with lowest-id tie-break
(``ops_basic.cu:196-245``); the Gated DeltaNet recurrence (``kernels/src/cuda/gdn_recurrent.cu:47-92``)
with its causal conv and gates (``ops_basic.cu:301-344``); lowest-index argmax (``ops_basic.cu:249``).
"""
from __future__ import annotations

import math
from typing import List, Optional, Sequence, Tuple

import torch
import torch.nn.functional as F

PAGE = 16


# ----------------------------------------------------------------------------------- norms
def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, residual: Optional[torch.Tensor] = None,
            zero_centered: bool = False) -> Tuple[torch.Tensor, torch.Tensor]:
    """Returns (normed, new_residual); ``new_residual = x + residual`` rounded to x.dtype."""
    if residual is not None:
        x = (x.float() + residual.float()).to(x.dtype)
    xf = x.float()
    var = xf.pow(2).mean(dim=-1, keepdim=True)
    wf = w.float() + 1.0 if zero_centered else w.float()
    y = xf * torch.rsqrt(var + eps) * wf
    return y.to(x.dtype), x


def gated_rmsnorm(x: torch.Tensor, z: torch.Tensor, w: torch.Tensor, eps: float, zero_centered: bool = False,
                  gate: str = "silu") -> torch.Tensor:
    """Per-head RMSNorm of the GDN output, then multiplied by silu(z) (or sigmoid(z))."""
    xf = x.float()
    var = xf.pow(2).mean(dim=-1, keepdim=True)
    wf = w.float() + 1.0 if zero_centered else w.float()
    y = xf * torch.rsqrt(var + eps) * wf
    g = F.silu(z.float()) if gate == "silu" else torch.sigmoid(z.float())
    return (y * g).to(x.dtype)


# ----------------------------------------------------------------------------------- rotary
def rope_cos_sin(positions: torch.Tensor, inv_freq: torch.Tensor, scale: float = 1.0,
                 mrope_section: Optional[Sequence[int]] = None):
    """positions ``[T]`` (or ``[3, T]`` with M-RoPE) → cos, sin ``[T, rotary_dim/2]`` fp32."""
    if positions.dim() == 2:
        ang3 = positions.float().unsqueeze(-1) * inv_freq.float()  # [3, T, half]
        if mrope_section:
            half = inv_freq.numel()
            sel = torch.zeros(half, dtype=torch.long, device=inv_freq.device)
            o = 0
            for i, n in enumerate(mrope_section):
                sel[o:o + n] = i
                o += n
            ang = ang3.gather(0, sel.view(1, 1, half).expand(1, ang3.shape[1], half)).squeeze(0)
        else:
            ang = ang3[0]
    else:
        ang = positions.float().unsqueeze(-1) * inv_freq.float()
    return torch.cos(ang) * scale, torch.sin(ang) * scale


def apply_rope_neox(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """x ``[T, H, D]`` fp32; rotates pairs (i, i + half) over the first ``2*half`` dims."""
    half = cos.shape[-1]
    x1, x2, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    c, s = cos.unsqueeze(1), sin.unsqueeze(1)
    return torch.cat([x1 * c - x2 * s, x2 * c + x1 * s, rest], dim=-1)


def rotate_heads(x: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, interleaved: bool) -> torch.Tensor:
    """x ``[T, H, D]``: the first ``2 * len(freq)`` dimensions of each head turned by position * frequency (fp32)."""
    n, xf = freq.numel(), x.float()
    ang = positions.double().view(-1, 1, 1) * freq.double()
    c, s = torch.cos(ang).float(), torch.sin(ang).float()
    a, b = (xf[..., 0:2 * n:2], xf[..., 1:2 * n:2]) if interleaved else (xf[..., :n], xf[..., n:2 * n])
    ra, rb = a * c - b * s, b * c + a * s
    turned = torch.stack([ra, rb], -1).flatten(-2) if interleaved else torch.cat([ra, rb], -1)
    return torch.cat([turned, xf[..., 2 * n:]], -1)


def hadamard_rotate(x: torch.Tensor) -> torch.Tensor:
    """Randomised Hadamard rotation of the last dimension (a power of two): element i changes sign when bit 15 of
    ``i * 2654435761 mod 2**32`` is set, then a Walsh-Hadamard transform scaled by 1/sqrt(D).  Orthogonal, so the dot
    product of two rotated vectors is the dot product of the originals (reference: ``rht_kernel``,
    kernels/src/cuda/nvfp4_kv.cu :356, behind ``--kv-rotate``)."""
    D = x.shape[-1]
    assert D & (D - 1) == 0
    idx = torch.arange(D, dtype=torch.int64)
    sign = 1.0 - 2.0 * (((idx * 2654435761) % (1 << 32)) >> 15 & 1).to(torch.float32)
    y = x.float() * sign.to(x.device)
    h = 1
    while h < D:
        y = y.reshape(*x.shape[:-1], D // (2 * h), 2, h)
        y = torch.stack([y[..., 0, :] + y[..., 1, :], y[..., 0, :] - y[..., 1, :]], dim=-2)
        h *= 2
    return y.reshape(x.shape) * D ** -0.5


def attn_prep(qkv: torch.Tensor, num_heads: int, num_kv_heads: int, head_dim: int,
              q_norm_w: Optional[torch.Tensor], k_norm_w: Optional[torch.Tensor], eps: float,
              cos: torch.Tensor, sin: torch.Tensor, gated: bool = False, zero_centered: bool = False,
              rotate: bool = False):
    """Split qkv rows, per-head RMSNorm of q and k, rotary, optionally the Hadamard rotation of q and k.
    Returns (q, k, v, gate|None) as [T,H,D]."""
    T = qkv.shape[0]
    dt = qkv.dtype
    qw = num_heads * head_dim * (2 if gated else 1)
    q_raw, k_raw, v_raw = qkv[:, :qw], qkv[:, qw:qw + num_kv_heads * head_dim], qkv[:, qw + num_kv_heads * head_dim:]
    gate = None
    if gated:
        qg = q_raw.view(T, num_heads, 2, head_dim)
        q, gate = qg[:, :, 0], qg[:, :, 1]
    else:
        q = q_raw.view(T, num_heads, head_dim)
    k = k_raw.view(T, num_kv_heads, head_dim)
    v = v_raw.view(T, num_kv_heads, head_dim)

    def hn(x, w):
        if w is None:
            return x.float()
        xf = x.float()
        wf = w.float() + 1.0 if zero_centered else w.float()
        y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * wf
        return y.to(dt).float()

    q = apply_rope_neox(hn(q, q_norm_w), cos, sin)
    k = apply_rope_neox(hn(k, k_norm_w), cos, sin)
    if rotate:
        q, k = hadamard_rotate(q), hadamard_rotate(k)
    return q.to(dt), k.to(dt), v.contiguous(), gate


# ----------------------------------------------------------------------------------- paged KV
def kv_write(k_pool: torch.Tensor, v_pool: torch.Tensor, k: torch.Tensor, v: torch.Tensor,
             slot_mapping: torch.Tensor) -> None:
    """Pools ``[pages, kv_heads, 16, D]``; slot = page * 16 + offset for each of the T new tokens."""
    page, off = slot_mapping.long() // PAGE, slot_mapping.long() % PAGE
    k_pool[page, :, off] = k.to(k_pool.dtype)
    v_pool[page, :, off] = v.to(v_pool.dtype)


def paged_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, block_table: torch.Tensor,
                    slots: Sequence[int], q_start: Sequence[int], ctx_len: Sequence[int], scale: float,
                    tree_mask: Optional[torch.Tensor] = None, allowed: Optional[Sequence] = None, window: int = 0,
                    sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal GQA attention of q ``[T, H, D]`` over the paged pools.  ``window`` > 0: over the last ``window`` positions; ``sink``
    ``[H]``: one more term ``exp(sink)`` in the denominators.

    Sequence ``b`` owns rows ``q_start[b]:q_start[b+1]``; its KV length *including* those rows is
    ``ctx_len[b]``; row i attends to positions ``<= ctx_len - q_len + i``.  With ``tree_mask`` (``[T]`` int32) row i
    sees, among its sequence's own new tokens, only those whose bit is set in its word (a draft tree's ancestors).
    ``allowed[b]`` (bool ``[q_len, ctx_len]`` or None) further restricts what sequence b's rows see (a sparse selection).
    """
    T, H, D = q.shape
    KH, E = k_pool.shape[1], v_pool.shape[3]
    group = H // KH
    out = torch.empty(T, H, E, dtype=torch.float32, device=q.device)
    for b, slot in enumerate(slots):
        r0, r1 = q_start[b], q_start[b + 1]
        ql, n = r1 - r0, ctx_len[b]
        if ql == 0:
            continue
        npg = (n + PAGE - 1) // PAGE
        pages = block_table[slot, :npg].long()
        K = k_pool[pages].float().permute(1, 0, 2, 3).reshape(KH, npg * PAGE, D)[:, :n]
        V = v_pool[pages].float().permute(1, 0, 2, 3).reshape(KH, npg * PAGE, E)[:, :n]
        qq = q[r0:r1].float().view(ql, KH, group, D).permute(1, 2, 0, 3)       # [KH, g, ql, D]
        s = torch.einsum("hgqd,hnd->hgqn", qq, K) * scale
        pos_q = torch.arange(n - ql, n, device=q.device).view(ql, 1)
        pos_k = torch.arange(n, device=q.device).view(1, n)
        mask = pos_k <= pos_q
        if window:
            mask = mask & (pos_k > pos_q - window)
        if tree_mask is not None:
            words = tree_mask[r0:r1].to(torch.int64).view(ql, 1) & 0xFFFFFFFF
            own = ((words >> torch.arange(min(ql, 32), device=q.device).view(1, -1)) & 1).bool()      # [ql, min(ql, 32)]
            mask = mask.clone()
            mask[:, n - ql:n - ql + own.shape[1]] &= own
        if allowed is not None and allowed[b] is not None:
            mask = mask & allowed[b]
        s = s.masked_fill(~mask, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.float().view(KH, group, 1, 1).expand(KH, group, ql, 1)], dim=-1)
        p = torch.softmax(s, dim=-1)[..., :n]
        o = torch.einsum("hgqn,hnd->hgqd", p, V)                               # [KH, g, ql, E]
        out[r0:r1] = o.permute(2, 0, 1, 3).reshape(ql, H, E)
    return out.to(q.dtype)


def diff_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, block_table: torch.Tensor, slots, q_start, ctx_len,
                   scale: float, window: int, lam: float, post: float, eps: float) -> torch.Tensor:
    """Differential attention of q ``[T, H, 2, d]``: per head two causal softmax maps (``window`` > 0: over the last ``window``
    positions) on the keys ``[pages, 2 * G, 16, d]``, both over the values ``[pages, G, 16, e]``; the head's output is the
    RMS-normed ``map 1 - lam * map 2`` times ``post``.  fp32 ``[T, H, e]``."""
    T, H, _, d = q.shape
    G, e = v_pool.shape[1], v_pool.shape[3]
    out = torch.zeros(T, H, e, dtype=torch.float32, device=q.device)
    for b, slot in enumerate(slots):
        r0, r1 = q_start[b], q_start[b + 1]
        ql, n = r1 - r0, ctx_len[b]
        if ql <= 0:
            continue
        lo = max(n - ql - window + 1, 0) // PAGE if window else 0             # first page any of the rows can see
        pages = block_table[slot, lo:(n + PAGE - 1) // PAGE].long()
        m, base = n - lo * PAGE, lo * PAGE
        K = k_pool[pages].float().permute(1, 0, 2, 3).reshape(G, 2, -1, d)[:, :, :m]
        V = v_pool[pages].float().permute(1, 0, 2, 3).reshape(G, -1, e)[:, :m]
        s = torch.einsum("qghmd,gmnd->gmhqn", q[r0:r1].float().view(ql, G, H // G, 2, d), K) * scale
        pq = torch.arange(n - ql, n, device=q.device).view(ql, 1)
        pk = torch.arange(base, n, device=q.device).view(1, m)
        seen = pk <= pq
        if window:
            seen = seen & (pk > pq - window)
        a = torch.einsum("gmhqn,gne->gmhqe", torch.softmax(s.masked_fill(~seen, float("-inf")), -1), V)
        o = a[:, 0] - lam * a[:, 1]                                           # [G, h, q, e]
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * post
        out[r0:r1] = o.permute(2, 0, 1, 3).reshape(ql, H, e)
    return out


def position_vectors(positions: torch.Tensor, freq: torch.Tensor, width: int) -> torch.Tensor:
    """Sines (even columns) and cosines (odd ones) of position * frequency of the column pair, fp32 ``[T, width]``."""
    ang = positions.double().view(-1, 1) * freq.double()
    return torch.stack([torch.sin(ang), torch.cos(ang)], -1).flatten(1)[:, :width].float()


def query_temperature(positions: torch.Tensor, coef: float, every: float) -> torch.Tensor:
    return 1 + coef * torch.log(torch.floor((positions.float() + 1) / every) + 1)


def causal_conv(u: torch.Tensor, before: torch.Tensor, w: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """Causal convolution of each channel over one sequence's rows, ``u [T, C]``, ``w [taps, C]``, ``before [taps - 1, C]`` the rows ahead
    of them; (fp32 rows, the last taps - 1 inputs)."""
    hist = torch.cat([before.to(u.dtype), u])
    return sum(hist[j:j + u.shape[0]].float() * w[j] for j in range(w.shape[0])), hist[u.shape[0]:]


def sigmoid_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, block_table: torch.Tensor, slots, q_start, ctx_len,
                      scale: float, bias: torch.Tensor, pad: int, window: int = 0) -> torch.Tensor:
    """Causal attention of q ``[T, H, d]`` over paged keys and values, whose weights are sigmoids of the scores: ``bias [H, pad + n + ..]``
    holds what is added to the score of a key by its distance (from ``pad`` on; the n-th for every one beyond).  fp32 ``[T, H, e]``."""
    T, H, d = q.shape
    G, e, n_dist = k_pool.shape[1], v_pool.shape[3], bias.shape[1] - 2 * pad
    out = torch.zeros(T, H, e, dtype=torch.float32, device=q.device)
    for b, slot in enumerate(slots):
        r0, r1 = q_start[b], q_start[b + 1]
        ql, n = r1 - r0, ctx_len[b]
        if ql <= 0:
            continue
        pages = block_table[slot, :(n + PAGE - 1) // PAGE].long()
        K = k_pool[pages].float().permute(1, 0, 2, 3).reshape(G, -1, d)[:, :n]
        V = v_pool[pages].float().permute(1, 0, 2, 3).reshape(G, -1, e)[:, :n]
        s = torch.einsum("qghd,gnd->ghqn", q[r0:r1].float().view(ql, G, H // G, d), K) * scale
        dist = torch.arange(n - ql, n, device=q.device).view(ql, 1) - torch.arange(n, device=q.device).view(1, n)
        add = bias[:, pad + dist.clamp(0, n_dist - 1)].masked_fill(dist < 0, float("-inf"))
        if window:
            add = add.masked_fill(dist >= window, float("-inf"))
        o = torch.einsum("ghqn,gne->qghe", torch.sigmoid(s + add.view(G, H // G, ql, n)), V)
        out[r0:r1] = o.reshape(ql, H, e)
    return out


def streams_write(x: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """Residual streams ``[T, S, W]`` after a sublayer: ``mix[from, to]`` of the old ones plus ``out[to] * y``."""
    return torch.einsum("ab,taw->tbw", mix, x) + out.view(1, -1, 1) * y.float()[:, None]


# ----------------------------------------------------------------------------------- MLP / MoE
def clamped_glu(gu: torch.Tensor, limit: float) -> torch.Tensor:
    """``[T, 2I]`` = ``[gate | up]`` -> ``g * sigmoid(1.702 g) * (u + 1)``, g = min(gate, limit), u = up clamped to +-limit."""
    I = gu.shape[-1] // 2
    g, u = gu[..., :I].clamp(max=limit), gu[..., I:].clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def relu2(z: torch.Tensor) -> torch.Tensor:
    return z.float().clamp(min=0).square().to(z.dtype)


def poly_norm(z: torch.Tensor, act: torch.Tensor, eps: float) -> torch.Tensor:
    """``a N(z) + b N(z^2) + c N(z^3) + e``, N dividing a row by its root mean square; ``act`` holds a, b, c, e.  fp32."""
    z = z.float()
    n = lambda x: x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)      # noqa: E731
    return act[0] * n(z) + act[1] * n(z * z) + act[2] * n(z * z * z) + act[3]


def silu_mul(gu: torch.Tensor) -> torch.Tensor:
    """``[T, 2I]`` laid out as ``[gate | up]`` → ``silu(gate) * up`` in the input dtype."""
    I = gu.shape[-1] // 2
    return (F.silu(gu[..., :I].float()) * gu[..., I:].float()).to(gu.dtype)


def router_topk(logits: torch.Tensor, k: int, renorm: bool = True, sigmoid: bool = False):
    """Softmax over all experts (or their sigmoids; fp32), top-k by score, lowest id wins ties."""
    p = torch.sigmoid(logits.float()) if sigmoid else torch.softmax(logits.float(), dim=-1)
    E = p.shape[-1]
    # stable lowest-id tie break: sort by (-p, id)
    order = torch.argsort(-p, dim=-1, stable=True)[..., :k]
    w = torch.gather(p, -1, order)
    if renorm:
        w = w / w.sum(dim=-1, keepdim=True)
    return w, order.to(torch.int32)


def moe_forward(x: torch.Tensor, topk_w: torch.Tensor, topk_id: torch.Tensor, expert_fn, num_experts: int, weigh_input: bool = False):
    """Reference mixture: ``out[t] = sum_j w[t,j] * expert_fn(e_j, x[t])`` evaluated per expert (``weigh_input``:
    ``sum_j expert_fn(e_j, w[t,j] * x[t])``)."""
    out = torch.zeros(x.shape, dtype=torch.float32, device=x.device)
    first = getattr(getattr(expert_fn, "__self__", None), "first", 0)
    count = getattr(getattr(expert_fn, "__self__", None), "count", num_experts)
    for e in range(first, first + count):
        tok, slot = (topk_id == e).nonzero(as_tuple=True)
        if tok.numel() == 0:
            continue
        w = topk_w[tok, slot].float().unsqueeze(-1)
        if weigh_input:
            out.index_add_(0, tok, expert_fn(e, (x[tok].float() * w).to(x.dtype)).float())
            continue
        y = expert_fn(e, x[tok]).float()
        out.index_add_(0, tok, y * w)
    return out.to(x.dtype)


# ----------------------------------------------------------------------------------- Gated DeltaNet
def gdn_conv(x: torch.Tensor, conv_state: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None,
             round_sum: bool = True) -> Tuple[torch.Tensor, torch.Tensor]:
    """Causal depthwise conv + SiLU over one sequence.

    ``x [T, C]``, ``conv_state [C, k-1]`` (the last k-1 inputs), ``w [C, k]``, optional ``bias [C]``.  The conv result is
    rounded to the activation dtype before SiLU (``round_sum``).  Returns (y [T, C], new_state).
    """
    T, C = x.shape
    k = w.shape[1]
    hist = torch.cat([conv_state.t().to(x.dtype), x], dim=0)          # [k-1+T, C]
    win = hist.float().unfold(0, k, 1)                                 # [T, C, k]
    y = (win * w.float().unsqueeze(0)).sum(-1)
    if bias is not None:
        y = y + bias.float()
    if round_sum:
        y = y.to(x.dtype)
    y = F.silu(y.float()).to(x.dtype)
    new_state = hist[-(k - 1):].t().contiguous().to(conv_state.dtype) if k > 1 else conv_state
    return y, new_state


def gdn_gates(a: torch.Tensor, b: torch.Tensor, A_log: torch.Tensor, dt_bias: torch.Tensor):
    """g = -exp(A_log) * softplus(a + dt_bias) (fp32);  beta = sigmoid(b) rounded to b.dtype."""
    g = -torch.exp(A_log.float()) * F.softplus(a.float() + dt_bias.float())
    beta = torch.sigmoid(b.float()).to(b.dtype).float()
    return g, beta


def gdn_recurrent(q, k, v, g, beta, state):
    """Exact token-by-token gated delta rule for one sequence.

    q,k ``[T, Hk, dk]``; v ``[T, Hv, dv]``; g, beta ``[T, Hv]``; state ``[Hv, dk, dv]`` fp32.
    q and k are L2-normalised, q is scaled by dk^-1/2.  Hv is a multiple of Hk (key heads shared).
    """
    T, Hk, dk = q.shape
    Hv, dv = v.shape[1], v.shape[2]
    rep = Hv // Hk
    qf = F.normalize(q.float(), dim=-1, eps=1e-6) * (dk ** -0.5)
    kf = F.normalize(k.float(), dim=-1, eps=1e-6)
    qf = qf.repeat_interleave(rep, dim=1)
    kf = kf.repeat_interleave(rep, dim=1)
    S = state.float().clone()
    out = torch.empty(T, Hv, dv, dtype=torch.float32, device=q.device)
    for t in range(T):
        S = S * torch.exp(g[t]).view(Hv, 1, 1)
        kv = torch.einsum("hk,hkv->hv", kf[t], S)
        delta = (v[t].float() - kv) * beta[t].view(Hv, 1)
        S = S + torch.einsum("hk,hv->hkv", kf[t], delta)
        out[t] = torch.einsum("hk,hkv->hv", qf[t], S)
    return out.to(v.dtype), S


def gdn_chunked(q, k, v, g, beta, state, chunk: int = 64):
    """Chunked (WY / UT-transform) evaluation of the same recurrence; what the GPU kernel computes."""
    T, Hk, dk = q.shape
    Hv, dv = v.shape[1], v.shape[2]
    rep = Hv // Hk
    qf = (F.normalize(q.float(), dim=-1, eps=1e-6) * (dk ** -0.5)).repeat_interleave(rep, dim=1)
    kf = F.normalize(k.float(), dim=-1, eps=1e-6).repeat_interleave(rep, dim=1)
    vf = v.float()
    S = state.float().clone()                                         # [Hv, dk, dv]
    out = torch.empty(T, Hv, dv, dtype=torch.float32, device=q.device)
    for c0 in range(0, T, chunk):
        c1 = min(c0 + chunk, T)
        L = c1 - c0
        Q, K, V = qf[c0:c1].transpose(0, 1), kf[c0:c1].transpose(0, 1), vf[c0:c1].transpose(0, 1)  # [Hv, L, *]
        G = g[c0:c1].t().float().cumsum(dim=1)                         # [Hv, L] cumulative log decay
        B = beta[c0:c1].t().float()                                    # [Hv, L]
        decay = torch.exp(G.unsqueeze(2) - G.unsqueeze(1))             # [Hv, i, j] = exp(G_i - G_j)
        tril = torch.tril(torch.ones(L, L, device=q.device, dtype=torch.bool), -1)
        A = torch.einsum("hik,hjk->hij", K, K) * decay * B.unsqueeze(2)
        A = A.masked_fill(~tril, 0.0)                                  # strictly lower
        eye = torch.eye(L, device=q.device).unsqueeze(0)
        Tm = torch.linalg.solve_triangular(eye + A, eye.expand(Hv, L, L).contiguous(), upper=False)
        # u_i = beta_i (v_i - exp(G_i) k_i^T S0) - sum_{j<i} A_ij u_j
        rhs = B.unsqueeze(2) * (V - torch.exp(G).unsqueeze(2) * torch.einsum("hik,hkv->hiv", K, S))
        U = torch.einsum("hij,hjv->hiv", Tm, rhs)                      # deltas  [Hv, L, dv]
        incl = torch.tril(torch.ones(L, L, device=q.device, dtype=torch.bool), 0)
        QK = (torch.einsum("hik,hjk->hij", Q, K) * decay).masked_fill(~incl, 0.0)
        O = torch.exp(G).unsqueeze(2) * torch.einsum("hik,hkv->hiv", Q, S) + torch.einsum("hij,hjv->hiv", QK, U)
        out[c0:c1] = O.transpose(0, 1)
        GL = G[:, -1]
        S = S * torch.exp(GL).view(Hv, 1, 1) + torch.einsum(
            "hjk,hjv->hkv", K * torch.exp(GL.unsqueeze(1) - G).unsqueeze(2), U)
    return out.to(v.dtype), S


# ----------------------------------------------------------------------------------- recurrences with an fp32 state
def delta_rule(q, k, v, a, b, A, dt_bias, state):
    """Gated delta rule with a decay per head and key channel, one sequence: q, k ``[T, G, dk]``, v ``[T, H, dv]``, decay inputs a
    ``[T, H, dk]`` (``[T, H, 1]``: one per head), write strengths b ``[T, H]`` (before their sigmoid), A ``[H]`` > 0, state ``[H, dk, dv]``.  fp32."""
    T, G, dk = q.shape
    H = v.shape[1]
    unit = lambda x: x.float() * torch.rsqrt(x.float().pow(2).sum(-1, keepdim=True) + 1e-6)      # noqa: E731
    q, k = [unit(x).repeat_interleave(H // G, 1) for x in (q, k)]
    g = torch.exp(-A.view(1, H, 1) * F.softplus(a.float() + dt_bias.view(1, H, -1)))
    beta, v, S = torch.sigmoid(b.float()), v.float(), state.clone()
    out = torch.empty(T, H, v.shape[2], device=q.device)
    for t in range(T):
        S = S * g[t].unsqueeze(-1)
        u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t].unsqueeze(-1) * u.unsqueeze(1)
        out[t] = torch.einsum("hkv,hk->hv", S, q[t]) * dk ** -0.5
    return out, S


def state_space(x, B, C, dt, A, dt_bias, D, state):
    """State-space duality, one sequence: x ``[T, H, dv]``, B, C ``[T, G, N]``, dt ``[T, H]`` before its softplus, A ``[H]`` > 0,
    state ``[H, N, dv]``.  fp32."""
    T, H, _ = x.shape
    x, dt, S = x.float(), F.softplus(dt.float() + dt_bias), state.clone()
    B, C = [y.float().repeat_interleave(H // B.shape[1], 1) for y in (B, C)]
    decay = torch.exp(-A * dt)
    out = torch.empty_like(x)
    for t in range(T):
        S = S * decay[t].view(H, 1, 1) + (dt[t].view(H, 1) * B[t]).unsqueeze(-1) * x[t].unsqueeze(1)
        out[t] = torch.einsum("hnv,hn->hv", S, C[t]) + D.view(H, 1) * x[t]
    return out, S


def gated_linear(q, f, v, lower, bias, state):
    """Gated linear attention (state rows keep a share f and take 1 - f of the value), one sequence: q and the gates' inputs f ``[T, H, dk]`` before
    their activations, v ``[T, H, dv]``, lower bounds and biases ``[H * dk]``, state ``[H, dk, dv]``.  fp32."""
    T, H, dk = q.shape
    lo = lower.view(1, H, dk)
    z = f.float() + bias.view(1, H, dk)
    keep, write = lo + (1 - lo) * torch.sigmoid(z), (1 - lo) * torch.sigmoid(-z)
    q, v, S = F.silu(q.float()), v.float(), state.clone()
    out = torch.empty(T, H, v.shape[2], device=q.device)
    for t in range(T):
        S = S * keep[t].unsqueeze(-1) + write[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out, S


def min_gru(z, u, state):
    """minGRU over one sequence: gate inputs z and candidates u ``[T, n]`` before their activations, state ``[n]``.  fp32."""
    z, u, S = torch.sigmoid(z.float()), u.float(), state.clone()
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    out = torch.empty_like(z)
    for t in range(z.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        out[t] = S
    return out, S


def input_conv(x, state, w):
    """``x + conv(x)`` over one sequence, ``x [T, C]`` fp32, ``w [taps, C]``, ``state [taps - 1, C]`` the inputs before; (y, new state)."""
    hist = torch.cat([state, x])
    y = x.clone()
    for j in range(w.shape[0]):
        y += hist[j:j + x.shape[0]] * w[j]
    return y, hist[x.shape[0]:]


def group_norm(o, z, w, groups: int, eps: float, sigmoid: bool, gate_first: bool, post: float = 1.0):
    """RMS norm of each of ``groups`` equal parts of fp32 rows ``[T, C]`` with a gate (``silu(z)`` or ``sigmoid(z)``; z None: none)
    before or after it and a weight that repeats over the columns.  fp32."""
    gate = torch.ones_like(o) if z is None else torch.sigmoid(z.float()) if sigmoid else F.silu(z.float())
    x = o * gate if gate_first else o
    x = x.view(x.shape[0], groups, -1)
    x = (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)).flatten(1) * w.repeat(o.shape[1] // w.numel())
    return (x if gate_first else x * gate) * post


# ----------------------------------------------------------------------------------- head
def argmax_lowest(logits: torch.Tensor) -> torch.Tensor:
    """Row-wise argmax; the lowest index wins ties."""
    m = logits.max(dim=-1, keepdim=True).values
    idx = torch.arange(logits.shape[-1], device=logits.device).expand_as(logits)
    big = torch.full_like(idx, logits.shape[-1])
    return torch.where(logits == m, idx, big).min(dim=-1).values
