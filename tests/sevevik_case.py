"""Small Sevevik configurations with random weights for the tests, as checkpoints on disk, and the engine driven by hand."""
import json
import os

import torch

from blaze_b200.weights import save_safetensors


def mixer(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.3, diff=0.35, window=20):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def layer(ff=96, limit=1.5, weights_of=None, **kw):
    e = {"type": "attention", "mixer": mixer(**kw), "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(layers=None, vocab=320, width=144, streams=3, mult=0.6, eps=1e-5, embed=3.0):
    layers = layers or [layer(), layer(heads=3, kv_heads=1, dim=16, vdim=32, window=33, ff=None), layer(weights_of=0),
                        layer(heads=2, kv_heads=2, dim=32, vdim=16, window=5, ff=128, limit=0.8)]
    return {"architecture": "Sevevik", "embedding": {"scale": embed}, "layers": layers, "norm": {"eps": eps},
            "residual_mult": mult, "streams": streams, "vocab": vocab, "width": width}


def weights(cfg, seed=0, sharp=2.0):
    """Random bf16 weights under the design's names; ``sharp`` scales the query and key maps (larger: fewer keys matter)."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, base=0.0: (torch.randn(*s, generator=g) * std + base).to(torch.bfloat16)   # noqa: E731
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    w = {"embed": rnd(V, W, std=0.3), "head": rnd(V, W, std=W ** -0.5), "final.norm": rnd(W, std=0.2, base=1.0)}
    for i, L in enumerate(cfg["layers"]):
        if "weights_of" in L:
            continue
        m, p = L["mixer"], f"l{i}."
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, r in (("q", H * 2 * d), ("k", G * 2 * d)):
            w[p + "mix." + n] = rnd(r, W, std=sharp * W ** -0.5)
        w[p + "mix.v"], w[p + "mix.o"] = rnd(G * e, W, std=W ** -0.5), rnd(W, H * e, std=(H * e) ** -0.5)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            w[p + "mix." + n] = rnd(d, std=0.4 / d ** 0.25)
        for q in (1, 2) if L["mlp"] else (1,):
            w[f"{p}norm{q}"] = rnd(W, std=0.2, base=1.0)
            w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"] = rnd(S, std=0.4, base=0.5), rnd(S, std=0.4, base=0.7)
            w[f"{p}hc{q}.mix"] = (torch.eye(S) * 0.8 + torch.randn(S, S, generator=g) * 0.2).to(torch.bfloat16)
        if L["mlp"]:
            f = L["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"] = rnd(f, W, std=1.5 * W ** -0.5), rnd(f, W, std=1.5 * W ** -0.5)
            w[p + "mlp.down"] = rnd(W, f, std=f ** -0.5)
    return w


def save(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(os.path.join(path, "model.safetensors"), w)
    return str(path)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def cut(n, sizes):
    """``n`` tokens as portions of the given sizes in turn."""
    out, k = [], 0
    while sum(out) < n:
        out.append(min(sizes[k % len(sizes)], n - sum(out)))
        k += 1
    return out


def run(eng, seqs, steps):
    """Logits of every token of every request.  ``seqs``: id -> tokens; ``steps``: lists of (id, count).  Requests open at their
    first entry and close with their last token."""
    live, at, out = {}, {i: 0 for i in seqs}, {i: [] for i in seqs}
    for step in steps:
        items = []
        for i, n in step:
            if i not in live:
                live[i] = eng.open_from()
            items.append((live[i], seqs[i][at[i]:at[i] + n], n))
        got = eng.forward(eng.plan(items), "logits").float().cpu()
        r = 0
        for i, n in step:
            out[i].append(got[r:r + n])
            r, at[i] = r + n, at[i] + n
            if at[i] == len(seqs[i]):
                eng.close(live.pop(i))
    eng.check_status()
    return {i: torch.cat(o) for i, o in out.items()}


def error(got, want):
    """Largest row error: difference without its mean over the vocabulary, over the spread of the wanted logits."""
    d = got.double() - want.double()
    d = d - d.mean(1, keepdim=True)
    return float((d.pow(2).mean(1).sqrt() / want.double().std()).max())
