"""Small Medodra configurations with random weights for the tests, as checkpoints on disk."""
import torch

from sevevik_case import cut, error, run, save, tokens        # noqa: F401  (helpers that fit any design)


def moe(experts=6, top=2, ff=40, shared=56):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared}}


def delta(mlp=None, heads=4, kv_heads=2, dim=24, vdim=20, conv=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def parallel(mlp=None, heads=6, kv_heads=3, dim=16, vdim=28, conv=4, scale=0.3, bias_max=50, coef=0.4, every=24, width=88):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "bias_max": bias_max,
                 "q_temp": {"coef": coef, "every": every}},
        "right": {"width": width}}}


def config(layers=None, vocab=320, width=112, eps=1e-5, mult=0.6, scale=0.7, loop=(1, 3, 2)):
    layers = layers or [delta(moe()), parallel(moe(5, 1, 24, 40)), delta(None, 3, 3, 32, 16, 2), parallel(None, 4, 1, 24, 32, 2, 0.5, 33, 0.2, 17, 60)]
    c = {"architecture": "Medodra", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab,
         "width": width}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed=0, sharp=1.0, rows=16):
    """Random bf16 weights under the design's names; decays from a few to hundreds of tokens; ``sharp`` scales the queries, ``rows`` is the
    length of the distance tables."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, base=0.0: (torch.randn(*s, generator=g) * std + base).to(torch.bfloat16)   # noqa: E731
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda r, c, k=1.0: rnd(r, c, std=k * c ** -0.5)      # noqa: E731
    w = {"embed": rnd(V, W), "head": lin(V, W), "final.norm": rnd(W, std=0.2)}
    if cfg.get("loop"):
        w["loop.in"] = lin(W, 2 * W)
    for i, L in enumerate(cfg["layers"]):
        m, f, p = L["mixer"], L["mlp"], f"l{i}.mix."
        if L["type"] == "delta":
            H, G, d, e = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            for n, r in (("q", G * d), ("k", G * d), ("v", H * e)):
                w[p + n], w[p + n + ".conv"] = lin(r, W, 1.5), rnd(r, m["conv"], std=0.5)
            w[p + "b"], w[p + "a"], w[p + "g"], w[p + "o"] = lin(H, W), lin(H, W), lin(H * e, W), lin(W, H * e)
            w[p + "A_log"], w[p + "dt_bias"], w[p + "norm"] = rnd(H, std=0.5), rnd(H, base=-3.0), rnd(e, std=0.3, base=1.0)
        else:
            a, r = m["left"], m["right"]["width"]
            H, G, d, e = (a[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            l = p + "left."
            for n, c, s in (("q", H * d, sharp), ("k", G * d, 1.0), ("v", G * e, 1.0)):
                w[l + n], w[l + n + ".b"], w[l + n + ".conv"] = lin(c, W, s), rnd(c, std=0.3), rnd(c, a["conv"], std=0.6)
            w[l + "rel"], w[l + "pb"] = rnd(rows, H, std=0.8), rnd(H, std=0.5, base=-2.0)
            w[l + "o"], w[l + "o.b"], w[l + "out"] = lin(W, H * e), rnd(W, std=0.3), rnd(W, std=0.3, base=1.0)
            q = p + "right."
            w[q + "z"], w[q + "z.b"], w[q + "x"], w[q + "x.b"] = lin(r, W), rnd(r, base=-2.0), lin(r, W), rnd(r, std=0.4)
            w[q + "g"], w[q + "o"], w[q + "out"] = lin(r, W), lin(W, r), rnd(W, std=0.3, base=1.0)
        for n in (1, 2) if f else (1,):
            w[f"l{i}.norm{n}"] = rnd(W, std=0.2)
        if f:
            p = f"l{i}.mlp."
            w[p + "router"], w[p + "shared.sg"] = lin(f["router"]["experts"], W, 5.0), lin(1, W)
            parts = {f"e{e}.": f["expert"]["ff"] for e in range(f["router"]["experts"])}
            for n, ff in {**parts, "shared.": f["shared"]["ff"]}.items():
                w[p + n + "gate"], w[p + n + "up"], w[p + n + "down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)
    return w
