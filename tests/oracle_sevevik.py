"""A plain, slow restatement of the Sevevik decoder, one function per mechanism, for the tests to compare the framework with.

Whole sequences only: no cache, no batch, no kernels, nothing shared with the package.  Weights are a dict of tensors under
the checkpoint's names; everything is computed in the dtype asked for (64-bit unless told otherwise).
"""
import math

import torch


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def clamped_glu(gate, up, limit):
    """min(gate, limit) through z * sigmoid(1.702 z), times the clamped up projection plus one."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, -limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def window_attention(q, k, v, scale, window):
    """One attention map: ``q [T, d]``, ``k [T, d]``, ``v [T, e]``; row i sees keys i - window + 1 .. i (None: all up to i)."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        s = (k[lo:i + 1] @ q[i]) * scale
        p = torch.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[lo:i + 1]
    return out


def mix_weight(lq1, lk1, lq2, lk2, diff):
    """How much of the second map is taken away from the first."""
    return math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + diff


def differential(h, w, prefix, mixer, eps):
    """Two attention maps per head over the same values, the second subtracted from the first, each head normed on its own."""
    H, G, d, e = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    window = (mixer.get("mask") or {}).get("size")
    T = h.shape[0]
    q = (h @ w[prefix + "q"].T).reshape(T, H, 2, d)
    k = (h @ w[prefix + "k"].T).reshape(T, G, 2, d)
    v = (h @ w[prefix + "v"].T).reshape(T, G, e)
    lam = mix_weight(*(w[prefix + n] for n in ("lq1", "lk1", "lq2", "lk2")), mixer["diff"])
    heads = []
    for x in range(H):
        g = x // (H // G)
        a1, a2 = (window_attention(q[:, x, m], k[:, g, m], v[:, g], mixer["scale"], window) for m in (0, 1))
        heads.append(rms(a1 - lam * a2, eps) * (1 - mixer["diff"]))
    return torch.cat(heads, -1) @ w[prefix + "o"].T


def dense_mlp(h, w, prefix, mlp):
    return clamped_glu(h @ w[prefix + "gate"].T, h @ w[prefix + "up"].T, mlp["limit"]) @ w[prefix + "down"].T


def read_streams(xs, w_in):
    """``xs [S, T, W]`` -> the sublayer's input before its norm."""
    return torch.einsum("s,stw->tw", w_in, xs)


def write_streams(xs, w_mix, w_out, y, mult):
    """Every stream anew from the old ones (``w_mix[from, to]``) and the sublayer's output."""
    return torch.einsum("ab,atw->btw", w_mix, xs) + mult * w_out[:, None, None] * y[None]


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]``.  ``cfg`` is config.json's dict; ``layers_out``, a list, gets the sum of the streams after each layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, mult, S = cfg["norm"]["eps"], cfg["residual_mult"], cfg.get("streams", 1)
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    xs = x[None].repeat(S, 1, 1)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{L.get('weights_of', i)}."
        subs = [(1, lambda h: differential(h, w, p + "mix.", L["mixer"], eps))]
        if L["mlp"] is not None:
            subs.append((2, lambda h: dense_mlp(h, w, p + "mlp.", L["mlp"])))
        for n, sub in subs:
            hc = f"{p}hc{n}."
            y = sub(rms(read_streams(xs, w[hc + "in"]), eps, w[f"{p}norm{n}"]))
            xs = write_streams(xs, w[hc + "mix"], w[hc + "out"], y, mult)
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return rms(xs.sum(0), eps, w["final.norm"]) @ w["head"].T
