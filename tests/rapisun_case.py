"""Small Rapisun configurations with random weights for the tests, as checkpoints on disk."""
import torch

from sevevik_case import cut, error, run, save, tokens        # noqa: F401  (helpers that fit any design)


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40, shared=56):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": None if not shared else {"ff": shared}}


def hgrn2(mlp=None, heads=3, dim=20, vdim=28):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def latent(mlp=None, kv_from=None, window=20, heads=4, dim=24, rot_dim=8, vdim=40, q_rank=36, kv_rank=48, scale=0.3, base=500.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def config(layers=None, vocab=320, width=144, taps=4, eps=1e-5):
    layers = layers or [latent(dense()), hgrn2(moe()), latent(moe(), window=33, heads=3, dim=16, rot_dim=16, vdim=32, kv_rank=64),
                        latent(None, kv_from=2, window=9, heads=5, dim=12, rot_dim=16, vdim=24, kv_rank=64, q_rank=20, scale=0.5),
                        hgrn2(moe(shared=0, top=3), heads=2, dim=32, vdim=16), latent(dense(72), kv_from=0, window=50, heads=2, kv_rank=48)]
    return {"architecture": "Rapisun", "canon": {"taps": taps}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def weights(cfg, seed=0, sharp=1.0):
    """Random bf16 weights under the design's names; forget gates from a token or two to hundreds of tokens; ``sharp`` scales the
    queries (larger: fewer keys matter)."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, std=1.0, base=0.0: (torch.randn(*s, generator=g) * std + base).to(torch.bfloat16)   # noqa: E731
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda r, c, k=1.0: rnd(r, c, std=k * c ** -0.5)      # noqa: E731
    w = {"embed": rnd(V, W), "embed.norm": rnd(W, std=0.2, base=1.0), "head": lin(V, W), "final.norm": rnd(W, std=0.2, base=1.0)}
    for i, L in enumerate(cfg["layers"]):
        m, f, p = L["mixer"], L["mlp"], f"l{i}.mix."
        w[f"l{i}.canon1"] = rnd(W, cfg["canon"]["taps"], std=0.3)
        H = m["heads"]
        if L["type"] == "hgrn2":
            n, e = H * m["dim"], m["vdim"]
            w[p + "q"], w[p + "f"], w[p + "v"] = lin(n, W), lin(n, W), lin(H * e, W)
            w[p + "f.b"], w[p + "lower"] = rnd(n, std=2.0, base=1.0), torch.sigmoid(rnd(n, std=2.0).float()).to(torch.bfloat16)
            w[p + "norm"], w[p + "o"] = rnd(e, std=0.3, base=1.0), lin(W, H * e)
        else:
            d, r, e, qr, kr = (m[k] for k in ("dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            w[p + "dq"], w[p + "dq.norm"], w[p + "uq"] = lin(qr, W), rnd(qr, std=0.3, base=1.0), lin(H * (d + r), qr, sharp)
            if "kv_from" not in m:
                w[p + "dkv"], w[p + "dkv.norm"] = lin(kr + r, W), rnd(kr, std=0.3, base=1.0)
            w[p + "uk"], w[p + "uv"], w[p + "o"] = lin(H * d, kr), lin(H * e, kr), lin(W, H * e)
            w[p + "sink"] = rnd(H, std=2.0, base=1.0)
        for n in (1, 2) if f else (1,):
            w[f"l{i}.norm{n}"] = rnd(W, std=0.2, base=0.6)
        p = f"l{i}.mlp."
        parts = {}
        if f and f["kind"] == "dense":
            parts[""], w[p + "act"] = f["ff"], rnd(4, std=0.6)
        elif f:
            w[p + "router"] = lin(f["router"]["experts"], W, 1.5)
            parts = {f"e{e}.": f["expert"]["ff"] for e in range(f["router"]["experts"])}
            if f["shared"]:
                parts["shared."] = f["shared"]["ff"]
        for n, ff in parts.items():
            w[p + n + "up"], w[p + n + "down"] = lin(ff, W), lin(W, ff)
    return w
