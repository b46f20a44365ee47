"""A plain, slow restatement of the Niletar decoder, one function per mechanism, for the tests to compare the framework with.

Whole sequences only: no cache, no batch, no kernels, nothing shared with the package.  Weights are a dict of tensors under
the checkpoint's names; everything is computed in the dtype asked for (64-bit unless told otherwise).
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms(x, eps) * (1 + w)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def short_conv(x, w, bias=None):
    """Causal convolution of each channel over time: ``x [T, C]``, ``w [C, taps]`` (the last tap is the current token's)."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += x[:T - back] * w[:, j]
    return y if bias is None else y + bias


# ----------------------------------------------------------------------------------- softmax attention
def rotary_frequencies(rot):
    """One frequency per rotated pair; with ``scaling``, long wavelengths are stretched and those in between blended."""
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, rot):
    """``x [T, heads, dim]``: neighbouring dimensions of the first ``dims`` are turned by position * frequency."""
    y = x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(rotary_frequencies(rot)):
        c, s = torch.cos(pos * f).to(x.dtype)[:, None], torch.sin(pos * f).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def sink_attention(q, k, v, scale, sink):
    """Causal attention of one head, ``q, k [T, d]``, ``v [T, e]``; the denominator has one more term ``exp(sink)``."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for i in range(T):
        s = (k[:i + 1] @ q[i]) * scale
        m = torch.maximum(s.max(), sink)
        p = torch.exp(s - m)
        out[i] = (p @ v[:i + 1]) / (p.sum() + torch.exp(sink - m))
    return out


def gated_attention(h, w, p, m, eps):
    """The heads' outputs before the output projection, gated by the layer's own input."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = ((h @ w[p + n].T + w[p + n + ".b"]) for n in "qkv")
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, e)
    q, k = (rms(rotate(t, m["rot"]), eps) for t in (q, k))
    heads = [sink_attention(q[:, x], k[:, x // (H // G)], v[:, x // (H // G)], m["scale"], w[p + "sink"][x]) for x in range(H)]
    return torch.cat(heads, 1) * sigmoid(h @ w[p + "g"].T)


# ----------------------------------------------------------------------------------- gated delta rule
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """One head: ``q, k, g [T, d]``, ``v [T, e]``, ``beta [T]``; the state's key rows decay by g, then k's value moves towards v."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = S * g[t][:, None]
        S = S + k[t][:, None] * (beta[t] * (v[t] - S.T @ k[t]))[None]
        out[t] = S.T @ q[t]
    return out


def gated_delta(h, w, p, m, eps):
    """The heads' outputs before the output projection."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q, k = unit(q.reshape(T, G, d)) / math.sqrt(d), unit(k.reshape(T, G, d))
    v = v.reshape(T, H, e)
    beta = sigmoid(h @ w[p + "b"].T)
    a = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, d)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * a)
    z = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, e)
    o = [delta_rule(q[:, x // (H // G)], k[:, x // (H // G)], v[:, x], g[:, x], beta[:, x]) for x in range(H)]
    return torch.cat([rms(o[x], eps) * w[p + "norm"] * z[:, x] for x in range(H)], 1)


def parallel(h, w, p, m, eps):
    left = gated_attention(h, w, p + "left.", m["left"], eps) @ w[p + "left.o"].T
    right = gated_delta(h, w, p + "right.", m["right"], eps) @ w[p + "right.o"].T
    return m["left_scale"] * left + m["right_scale"] * right


# ----------------------------------------------------------------------------------- state-space mixer
def state_space(x, B, C, dt, decay, D):
    """One head: ``x [T, e]``, ``B, C [T, N]``, ``dt, decay [T]``."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=x.dtype)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = decay[t] * S + dt[t] * B[t][:, None] * x[t][None]
        out[t] = S.T @ C[t] + D * x[t]
    return out


def mamba2(h, w, p, m, eps):
    H, e, N, G, P = m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"]
    T, inner = h.shape[0], H * e
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], 1)
    x, B, C = torch.split(silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"])), [inner, G * N, G * N], 1)
    x, B, C = x.reshape(T, H, e), B.reshape(T, G, N), C.reshape(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    y = torch.cat([state_space(x[:, i], B[:, i // (H // G)], C[:, i // (H // G)], dt[:, i], decay[:, i], w[p + "D"][i]) for i in range(H)], 1)
    y = y * silu(z)
    return (rms(y.reshape(T, P, inner // P), eps).reshape(T, inner) * w[p + "norm"]) @ w[p + "o"].T


def dense_mlp(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"mamba2": mamba2, "parallel": parallel}


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]``.  ``cfg`` is config.json's dict; ``layers_out``, a list, gets the residual after each layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{L.get('weights_of', i)}."
        x = centred_norm(alpha * x + MIXERS[L["type"]](x, w, p + "mix.", L["mixer"], eps), w[p + "norm1"], eps)
        if L["mlp"] is not None:
            x = centred_norm(alpha * x + dense_mlp(x, w, p + "mlp."), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T
