"""The Medodra design for :mod:`blaze_b200.benchmarks.design`: its configuration beside a Qwen3-Next hybrid with experts of equal size
(recurrent states, attention heads, experts), and its kernels beside the like ones."""
from __future__ import annotations

import copy
from typing import Callable, Dict

import torch

from ..config import DeltaSpec, LayerSpec, MinGruSpec, ModelConfig, MoeSpec, SigmoidAttnSpec, _unrolled
from . import rapisun
from .rapisun import EXPERTS, TOP

ROWS, FAR = 32, 256          # distance table: rows, distance of the last


def configs(W: int, H: int, G: int, ff: int, window: int, layers: int, vocab: int) -> Dict[str, ModelConfig]:
    """Delta-rule layers and parallel ones in turn; the middle ones are a loop of one pass, so that every layer has weights of its own."""
    moe = MoeSpec(EXPERTS, TOP, W // 4, W // 4, "swiglu", "sigmoid", False, True, True)
    attn = SigmoidAttnSpec(H, G, 128, 128, 128 ** -0.5, FAR, True, 4, True, 0.2, 1024.0)
    delta = DeltaSpec(W // 128, W // 128, 128, 128, 4, head_decay=True, gate="silu")
    specs = [LayerSpec(attn, moe, None, MinGruSpec(W)) if i % 2 else LayerSpec(None, moe, None, delta) for i in range(layers)]
    if layers > 2:
        specs = _unrolled(specs, {"start": layers // 4, "stop": layers - layers // 4, "times": 1})
    one = ModelConfig.of_layers(specs, architecture="Medodra", model_type="medodra", vocab_size=vocab, hidden_size=W, zero_centered_norm=True,
                                residual_mult=0.5, embed_scale=1.0)
    two = rapisun.configs(W, H, G, ff, window, layers, vocab)["qwen3-next (moe)"]
    return {"medodra": one, "qwen3-next (moe)": two}


def _attn_mixer(a: SigmoidAttnSpec):
    from ..models.qwen3 import Mixer, SigmoidAttn
    M = Mixer()
    M.attn = SigmoidAttn(a, "cuda", torch.randn(ROWS, a.heads), torch.randn(a.heads) - 4, torch.randn(a.conv_dim, a.conv))
    at = [a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim]
    M.cols = {"q": 0, "k": at[0], "v": at[0] + at[1]}
    return M, sum(at)


def kernels(sizes, window: int, add: Callable, graph_ms: Callable, like_attention: Callable, like_recurrence: Callable, ops) -> None:
    """Timings through ``add(kernel, model, ms, bytes, flops)``; ``like_*`` time the relative's kernels."""
    from ..models.qwen3 import Branches, Mixer, Recurrence
    W, H, G, ff = sizes
    both = configs(W, H, G, ff, window, 2, 1024)
    own, rel = both.values()
    names = list(both)
    rec, a, gru = own.layer_specs[0].rec, own.layer_specs[1].attn, own.layer_specs[1].rec
    one, bf = ModelConfig.of_layers([LayerSpec(a)], architecture="Medodra"), 2.0
    M, width = _attn_mixer(a)
    for label, B, qlen, ctx, copies in (("decode 256x1024", 256, 1, 1024, 2), ("decode 32x1024", 32, 1, 1024, 8),
                                        ("prefill 4x1024", 4, 1024, 1024, 4), ("prefill 1x8192", 1, 8192, 8192, 2)):
        kvs, batch = rapisun._sequences(one, B, qlen, ctx, copies)
        T = B * qlen
        q, out = torch.randn(T, H * a.dim, device="cuda").bfloat16(), torch.empty(T, H * a.vdim, dtype=torch.bfloat16, device="cuda")
        keys = sum(range(ctx - qlen + 1, ctx + 1))
        add("attention " + label, names[0], graph_ms([lambda kv=kv: ops.sigmoid_attend(q, M, batch, kv, 0, out) for kv in kvs]),
            B * ctx * G * (a.dim + a.vdim) * bf + T * H * (a.dim + a.vdim) * bf, 2.0 * B * H * keys * (a.dim + a.vdim))
        if B == 256 or qlen == 1024:
            proj = torch.randn(T, width, device="cuda").bfloat16()
            add("page write " + label, names[0], graph_ms([lambda kv=kv: ops.conv_prep_pages(proj, M, batch, kv, 0, 1e-6) for kv in kvs]),
                2 * T * width * bf + B * 6 * width * bf)
        del kvs, q, out
        torch.cuda.empty_cache()
        like_attention(label, B, qlen, ctx, rel, names[1])
    # the delta rule, then the elementwise recurrence
    cfg = ModelConfig.of_layers([LayerSpec(rec=rec)], architecture="Medodra")
    R, M = Recurrence(rec, "delta", rec.heads), Mixer()
    C, nv = rec.conv_dim, rec.heads * rec.vdim
    M.rec, M.cols = R, {"conv": 0, "z": C, "beta": C + nv, "decay": C + nv + rec.heads}
    R.conv_w, R.A, R.dt_bias = torch.randn(C, 4, device="cuda").bfloat16(), torch.ones(rec.heads, device="cuda"), torch.full((rec.heads,), -4.0, device="cuda")
    R.norm_w = torch.ones(rec.vdim, device="cuda")
    gcfg, E = ModelConfig.of_layers([LayerSpec(rec=gru)], architecture="Medodra"), Mixer()
    E.rec, E.cols = Recurrence(gru, "mingru", 1), {"zg": 0, "u": W, "g": 2 * W}
    for label, B, qlen, copies in (("decode 256", 256, 1, 3), ("decode 8", 8, 1, 16), ("prefill 8x1024", 8, 1024, 2), ("prefill 1x8192", 1, 8192, 2)):
        kvs, batch = rapisun._sequences(cfg, B, qlen, qlen + 8, copies)
        T = B * qlen
        proj, y = torch.randn(T, C + nv + 2 * rec.heads, device="cuda").bfloat16(), torch.randn(T, C, device="cuda").bfloat16()
        o, out = torch.empty(T, nv, device="cuda"), torch.empty(T, nv, dtype=torch.bfloat16, device="cuda")
        io = T * C * bf
        add("convolution " + label, names[0], graph_ms([lambda kv=kv: ops.short_conv(proj, M, batch, kv, 0) for kv in kvs]), 2 * io)
        add("recurrence " + label, names[0], graph_ms([lambda kv=kv: ops.recur(y, proj, None, M, batch, kv, 0, o) for kv in kvs]),
            io + T * rec.heads * 4.0 + B * nv * rec.dim * 8.0 + 4.0 * T * nv, 6.0 * T * nv * rec.dim)
        add("norm " + label, names[0], graph_ms([lambda: ops.gated_norm(o, proj, M, 1e-6, out)] * copies), T * nv * 8.0)
        del kvs, proj, y, o, out
        kvs, batch = rapisun._sequences(gcfg, B, qlen, qlen + 8, copies)
        proj, out = torch.randn(T, 3 * W, device="cuda").bfloat16(), torch.empty(T, W, dtype=torch.bfloat16, device="cuda")
        add("elementwise recurrence " + label, names[0], graph_ms([lambda kv=kv: ops.min_gru(proj, E, batch, kv, 0, out) for kv in kvs]),
            T * W * 8.0 + B * W * 8.0)
        del kvs, proj, out
        torch.cuda.empty_cache()
        like_recurrence(label, B, qlen, copies, rel, names[1])
    _feed_forward(own, rel, names, W, add, graph_ms, ops)
    for T in (256, 8192):
        c = max(2, int(400e6 // (T * W * 16)))
        y, z, w = torch.randn(T, W, device="cuda").bfloat16(), torch.randn(T, W, device="cuda").bfloat16(), torch.ones(W, device="cuda")
        xs = [torch.randn(T, W, device="cuda") for _ in range(c)]
        br = Branches((y, z), (w, w), None, 0.5)
        add(f"residual + norms, {T} rows", names[0], graph_ms([lambda x=x: ops.branch_step(x, br, 1e-6, torch.bfloat16, w, w) for x in xs]), T * W * 16.0)
        rs = [torch.randn(T, W, device="cuda").bfloat16() for _ in range(c)]
        add(f"residual + norms, {T} rows", names[1], graph_ms([lambda r=r: ops.norm(y, r, w.bfloat16(), 1e-6) for r in rs]), T * W * 8.0)
        del xs, rs


def _feed_forward(own: ModelConfig, rel: ModelConfig, names, W: int, add, graph_ms, ops) -> None:
    """A layer's router, routed experts, the shared one, the sum over the chosen ones, the residual and the next norm."""
    from ..models.medodra import Medodra
    from ..models.qwen3 import Branches, Model
    for T in (256, 8192):
        h = torch.randn(T, W, device="cuda").bfloat16()
        x, w, y = torch.zeros(T, W, device="cuda"), torch.ones(W, device="cuda"), torch.zeros(T, W, device="cuda").bfloat16()
        for name, cls, cfg in ((names[0], Medodra, own), (names[1], Model, rel)):
            c = copy.copy(cfg)
            if cfg is own:
                c.layer_specs, c.num_layers, c.layer_types = cfg.layer_specs[:1], 1, cfg.layer_types[:1]
            else:
                c.num_layers, c.layer_types = 1, cfg.layer_types[1:2]
            ms = [cls.random_init(c, seed=i, device="cuda", ops=ops) for i in range(3)]
            per = 3 * W * own.layer_specs[0].mlp.ff      # weights of an expert
            hit = EXPERTS if T * TOP >= EXPERTS * 8 else EXPERTS * (1 - (1 - TOP / EXPERTS) ** T)
            nb, fl = (hit + 1) * per * 2.0 + T * W * 4.0, 2.0 * T * (TOP + 1) * per
            if cfg is own:
                calls = [lambda m=m: ops.branch_step(x, Branches(y, None, m._mlp(m.layers[0].mlp, h)[0], 0.5), 1e-6, torch.bfloat16, w) for m in ms]
                nb += T * W * 10.0
            else:
                res = torch.zeros(T, W, device="cuda").bfloat16()
                calls = [lambda m=m: ops.norm(m._mlp(m.layers[0].mlp, h)[0], res, w.bfloat16(), 1e-6) for m in ms]
                nb += T * W * 4.0
            add(f"experts + residual + norm, {T} rows", name, graph_ms(calls), nb, fl)
            del ms, calls
            torch.cuda.empty_cache()
