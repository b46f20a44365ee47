"""A plain, slow restatement of the Rapisun decoder, one function per mechanism, for the tests to compare the framework with.

Whole sequences only: no cache, no batch, no kernels, nothing shared with the package.  Weights are a dict of tensors under
the checkpoint's names; everything is computed in the dtype asked for (64-bit unless told otherwise).
"""
import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    """Mean and spread taken out of each row, then a weight per column (no bias)."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def causal_conv(x, w):
    """Convolution of each channel over time, ``x [T, C]``, ``w [C, taps]`` (the last tap is the current token's)."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


def input_conv(x, w):
    return x + causal_conv(x, w)


# ----------------------------------------------------------------------------------- gated linear attention
def gated_linear(q, f, v):
    """One head, ``q, f [T, d]``, ``v [T, e]``: the state's row i keeps f_i of itself and takes 1 - f_i of the value."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = f[t][:, None] * S + (1 - f[t])[:, None] * v[t][None]
        out[t] = q[t] @ S
    return out


def forget_gate(z, lower):
    return lower + (1 - lower) * sigmoid(z)


def hgrn2(h, w, p, m, eps, shared=None):
    H, d, e, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = silu(h @ w[p + "q"].T).reshape(T, H, d)
    f = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, e)
    o = [rms(gated_linear(q[:, i], f[:, i], v[:, i]), eps) * w[p + "norm"] for i in range(H)]
    return torch.cat(o, 1) @ w[p + "o"].T


# ----------------------------------------------------------------------------------- latent attention
def rotate_half(x, dims, base):
    """``x [T, ..., n]``: dimensions i and i + dims / 2 of the first ``dims`` are turned by position * base^(-2 i / dims)."""
    y, half = x.clone(), dims // 2
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        shape = [-1] + [1] * (x.dim() - 2)
        c, s = torch.cos(a).to(x.dtype).reshape(shape), torch.sin(a).to(x.dtype).reshape(shape)
        u, v = x[..., i], x[..., i + half]
        y[..., i], y[..., i + half] = u * c - v * s, v * c + u * s
    return y


def sink_window_attention(q, k, v, scale, window, sink):
    """One head, ``q, k [T, d]``, ``v [T, e]``: keys lie at most window - 1 positions back (window 0: anywhere before);
    the denominator has one more term ``exp(sink)``."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for i in range(T):
        lo = max(0, i - window + 1) if window else 0
        s = (k[lo:i + 1] @ q[i]) * scale
        top = torch.maximum(s.max(), sink)
        p = torch.exp(s - top)
        out[i] = (p @ v[lo:i + 1]) / (p.sum() + torch.exp(sink - top))
    return out


def latent_keys(h, w, p, m, eps):
    """What a layer caches per token: its normed latent and the key part that all heads share, rotated."""
    z = h @ w[p + "dkv"].T
    r = m["kv_rank"]
    return rms(z[:, :r], eps) * w[p + "dkv.norm"], rotate_half(z[:, r:], m["rot"]["dims"], m["rot"]["base"])


def latent_attention(h, w, p, m, eps, shared):
    """``shared``: latents and rotated key parts of the layers so far, by layer."""
    H, d, r, e, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], h.shape[0]
    q = ((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).reshape(T, H, d + r)
    qr = rotate_half(q[..., d:], m["rot"]["dims"], m["rot"]["base"])
    i = int(p[1:p.index(".")])
    if m.get("kv_from") is None:
        shared[i] = latent_keys(h, w, p, m, eps)
    c, kr = shared[i if m.get("kv_from") is None else m["kv_from"]]
    k, v = (c @ w[p + "uk"].T).reshape(T, H, d), (c @ w[p + "uv"].T).reshape(T, H, e)
    window = (m.get("mask") or {}).get("size") or 0
    o = [sink_window_attention(torch.cat([q[:, x, :d], qr[:, x]], 1), torch.cat([k[:, x], kr], 1), v[:, x], m["scale"], window,
                               w[p + "sink"][x]) for x in range(H)]
    return torch.cat(o, 1) @ w[p + "o"].T


# ----------------------------------------------------------------------------------- feed-forwards
def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


def expert(h, w, p):
    return squared_relu(h @ w[p + "up"].T) @ w[p + "down"].T


def route(z, top):
    """Chosen experts and their weights: the largest softmax scores, divided by their sum."""
    s = torch.softmax(z, -1)
    best = s.argsort(-1, descending=True)[:, :top]
    picked = s.gather(1, best)
    return best, picked / (picked.sum(-1, keepdim=True) + 1e-20)


def mixture(h, w, p, m):
    best, weight = route(h @ w[p + "router"].T, m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows, place = (best == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weight[rows, place][:, None] * expert(h[rows], w, f"{p}e{e}.")
    return out + expert(h, w, p + "shared.") if m.get("shared") else out


def dense(h, w, p, m, eps):
    return poly_norm(h @ w[p + "up"].T, w[p + "act"], eps) @ w[p + "down"].T


MIXERS = {"hgrn2": hgrn2, "latent_attention": latent_attention}


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]``.  ``cfg`` is config.json's dict; ``layers_out``, a list, gets the residual after each layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, shared = cfg["norm"]["eps"], {}
    x = layer_norm(w["embed"][torch.as_tensor(tokens)], w["embed.norm"], eps)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[L["type"]](input_conv(x, w[p + "canon1"]), w, p + "mix.", L["mixer"], eps, shared)
        x = x + layer_norm(y, w[p + "norm1"], eps)
        if L["mlp"] is not None:
            f = dense(x, w, p + "mlp.", L["mlp"], eps) if L["mlp"]["kind"] == "dense" else mixture(x, w, p + "mlp.", L["mlp"])
            x = x + layer_norm(f, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
