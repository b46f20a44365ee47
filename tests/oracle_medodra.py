"""A plain, slow restatement of the Medodra decoder, one function per mechanism, for the tests to compare the framework with.

Whole sequences only: no cache, no batch, no kernels, nothing shared with the package.  Weights are a dict of tensors under
the checkpoint's names; everything is computed in the dtype asked for (64-bit unless told otherwise).
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(x, w):
    """Convolution of each channel over time, ``x [T, C]``, ``w [C, taps]`` (the last tap is the current token's)."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


def position_vectors(positions, width, dtype):
    """Sines (even columns) and cosines (odd columns) of position * 10000^(-2 i / width), i counting the pairs of columns."""
    p = positions.to(torch.float64)
    cols = [(torch.sin if c % 2 == 0 else torch.cos)(p * 10000.0 ** (-2.0 * (c // 2) / width)) for c in range(width)]
    return torch.stack(cols, 1).to(dtype)


def embedding(tokens, table, scale):
    x = table[torch.as_tensor(tokens)] * scale
    return x + position_vectors(torch.arange(x.shape[0]), x.shape[1], x.dtype)


def join_input(x, x0, w):
    """What a pass through the loop starts from: a linear map of the residual beside the embedding."""
    return torch.cat([x, x0], 1) @ w.T


# ----------------------------------------------------------------------------------- delta rule
def delta_rule(q, k, v, g, beta):
    """One head, ``q, k [T, d]``, ``v [T, e]``, decays and write strengths ``[T]``."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - k[t] @ S))
        out[t] = q[t] @ S
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_mixer(h, w, p, m, eps):
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = [silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])).reshape(T, heads, -1) for n, heads in (("q", G), ("k", G), ("v", H))]
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    gate = silu(h @ w[p + "g"].T).reshape(T, H, e)
    o = [rms(delta_rule(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i], beta[:, i]), eps) * w[p + "norm"] * gate[:, i]
         for i in range(H)]
    return torch.cat(o, 1) @ w[p + "o"].T


# ----------------------------------------------------------------------------------- sigmoid attention beside a gated recurrence
def distance_bucket(n, rows, far):
    """Row of a distance table for a key ``n`` tokens back: one each at first, then logarithmically wider up to ``far``."""
    near = rows // 2
    if n < near:
        return n
    return min(rows - 1, near + math.floor(math.log(n / near) / math.log(far / near) * (rows - near) + 1e-9))


def query_temperature(p, coef, every):
    return 1 + coef * math.log(math.floor((p + 1) / every) + 1)


def sigmoid_attention(q, k, v, scale, bias, shift):
    """One head, ``q, k [T, d]``, ``v [T, e]``: weights are sigmoids, not shares; ``bias[n]`` is added to the score of a key n back,
    ``shift`` to every score."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for i in range(T):
        s = (k[:i + 1] @ q[i]) * scale + bias[:i + 1].flip(0) + shift
        out[i] = sigmoid(s) @ v[:i + 1]
    return out


def left_mixer(h, w, p, m, eps):
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = [causal_conv(h @ w[p + n].T + w[p + n + ".b"], w[p + n + ".conv"]).reshape(T, heads, -1)
               for n, heads in (("q", H), ("k", G), ("v", G))]
    temp = torch.tensor([query_temperature(i, m["q_temp"]["coef"], m["q_temp"]["every"]) for i in range(T)], dtype=h.dtype)
    q, v = q * temp[:, None, None], rms(v, eps)
    rel = w[p + "rel"]
    rows = torch.tensor([distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)])
    o = [sigmoid_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], rel[rows, i], w[p + "pb"][i]) for i in range(H)]
    return torch.cat(o, 1) @ w[p + "o"].T + w[p + "o.b"]


def min_gru(z, u):
    """Gates ``z`` in (0, 1) and inputs ``u``, ``[T, n]``: the state keeps 1 - z of itself and takes z of the candidate."""
    cand = torch.where(u >= 0, u + 0.5, sigmoid(u))
    S, out = torch.zeros(z.shape[1], dtype=z.dtype), torch.zeros_like(z)
    for t in range(z.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        out[t] = S
    return out


def right_mixer(h, w, p, m, eps):
    S = min_gru(sigmoid(h @ w[p + "z"].T + w[p + "z.b"]), h @ w[p + "x"].T + w[p + "x.b"])
    return (S * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    left = rms(left_mixer(h, w, p + "left.", m["left"], eps), eps) * w[p + "left.out"]
    right = rms(right_mixer(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return (left + right) / 2


# ----------------------------------------------------------------------------------- feed-forward
def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """Chosen experts and their weights: the largest sigmoid scores, as they are."""
    s = sigmoid(z)
    best = z.argsort(-1, descending=True)[:, :top]
    return best, s.gather(1, best)


def mixture(h, w, p, m):
    """The weight of an expert is on its input."""
    best, weight = route(h @ w[p + "router"].T, m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows, place = (best == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += expert(weight[rows, place][:, None] * h[rows], w, f"{p}e{e}.")
    if m.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return out


MIXERS = {"delta": delta_mixer, "parallel": parallel_mixer}


def layer_runs(cfg):
    """(layer, whether a pass of the loop starts with it) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, z = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, z)] + [(i, False) for i in range(z, n)]


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits ``[T, vocab]``.  ``cfg`` is config.json's dict; ``layers_out``, a list, gets the residual after each layer run."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = embedding(tokens, w["embed"], cfg["embedding"]["scale"])
    for i, starts in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if starts:
            x = join_input(x, x0, w["loop.in"])
        y = MIXERS[L["type"]](norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps)
        if L["mlp"] is not None:
            y = y + mixture(norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"])
        x = x + cfg["residual_mult"] * y
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, w["final.norm"], eps) @ w["head"].T
