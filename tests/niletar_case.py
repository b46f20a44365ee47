"""Small Niletar configurations with random weights for the tests, as checkpoints on disk."""
import torch

from sevevik_case import cut, error, run, save, tokens        # noqa: F401  (helpers that fit any design)


def mamba(ff=96, weights_of=None, **kw):
    m = {"heads": 4, "vdim": 24, "state": 20, "groups": 2, "norm_groups": 3, "conv": 4, **kw}
    return _entry("mamba2", m, ff, weights_of)


def parallel(ff=80, weights_of=None, left=None, right=None, rot=None, left_scale=0.7, right_scale=0.45):
    r = {"dims": 16, "base": 2000.0, "scaling": {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 96}} if rot is None else rot
    m = {"left": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.35, "rot": r, **(left or {})}, "left_scale": left_scale,
         "right": {"heads": 6, "kv_heads": 3, "dim": 20, "vdim": 28, "conv": 3, **(right or {})}, "right_scale": right_scale}
    return _entry("parallel", m, ff, weights_of)


def _entry(kind, mixer, ff, weights_of):
    e = {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(layers=None, vocab=320, width=144, alpha=1.7, eps=1e-5):
    layers = layers or [parallel(), mamba(), mamba(weights_of=1),
                        parallel(ff=None, left={"heads": 3, "kv_heads": 1, "dim": 16, "vdim": 32}, rot={"dims": 12, "base": 1e4},
                                 right={"heads": 2, "kv_heads": 2, "dim": 32, "vdim": 16, "conv": 2}, left_scale=0.5, right_scale=0.9),
                        parallel(weights_of=0)]
    return {"architecture": "Niletar", "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha, "vocab": vocab, "width": width}


def weights(cfg, seed=0, ranks=(6, 10)):
    """Random bf16 weights under the design's names; decays from a token or two to hundreds of tokens."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, base=0.0: (torch.randn(*s, generator=g) * std + base).to(torch.bfloat16)   # noqa: E731
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda r, c: rnd(r, c, std=c ** -0.5)      # noqa: E731
    w = {"embed": rnd(V, W), "head": rnd(V, W, std=W ** -0.5), "final.norm": rnd(W, std=0.2)}
    for i, L in enumerate(cfg["layers"]):
        if "weights_of" in L:
            continue
        m, p = L["mixer"], f"l{i}.mix."
        if L["type"] == "mamba2":
            inner, bc, H = m["heads"] * m["vdim"], 2 * m["groups"] * m["state"], m["heads"]
            w[p + "in"] = lin(2 * inner + bc + H, W)
            w[p + "conv"], w[p + "conv.b"] = rnd(inner + bc, m["conv"], std=0.6), rnd(inner + bc, std=0.3)
            w[p + "dt_bias"], w[p + "A_log"], w[p + "D"] = rnd(H, std=1.5, base=-2.5), rnd(H, std=1.5), rnd(H, std=0.5)
            w[p + "norm"], w[p + "o"] = rnd(inner, std=0.3, base=1.0), lin(W, inner)
        else:
            l, r = m["left"], m["right"]
            H, G, d, e = (l[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            for n, k in (("q", H * d), ("k", G * d), ("v", G * e)):
                w[f"{p}left.{n}"], w[f"{p}left.{n}.b"] = lin(k, W), rnd(k, std=0.5)
            w[p + "left.sink"], w[p + "left.g"], w[p + "left.o"] = rnd(H, std=2.0, base=1.0), lin(H * e, W), lin(W, H * e)
            H, G, d, e, p = r["heads"], r["kv_heads"], r["dim"], r["vdim"], p + "right."
            for n, k in (("q", G * d), ("k", G * d), ("v", H * e)):
                w[p + n], w[f"{p}{n}.conv"] = lin(k, W), rnd(k, r["conv"], std=0.7)
            w[p + "b"], w[p + "A_log"], w[p + "norm"] = lin(H, W), rnd(H, std=1.5), rnd(e, std=0.3, base=1.0)
            for n, rank, k in (("a", ranks[0], H * d), ("g", ranks[1], H * e)):
                w[f"{p}{n}1"], w[f"{p}{n}2"] = lin(rank, W), lin(k, rank)
            w[p + "dt_bias"], w[p + "o"] = rnd(H * d, std=1.5, base=-3.0), lin(W, H * e)
        for n in (1, 2) if L["mlp"] else (1,):
            w[f"l{i}.norm{n}"] = rnd(W, std=0.2)
        if L["mlp"]:
            f = L["mlp"]["ff"]
            w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = lin(f, W), lin(f, W), lin(W, f)
    return w
