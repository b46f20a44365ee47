"""The Rapisun design for :mod:`blaze_b200.benchmarks.design`: its configuration beside a Qwen3-Next hybrid with experts of equal size
(recurrent states, projections of the attention, bytes of all experts), and its kernels beside the like ones."""
from __future__ import annotations

import copy
from typing import Callable, Dict

import torch

from ..config import (GatedLinearSpec, LatentAttnSpec, LayerSpec, ModelConfig, MoeSpec, PolyNormSpec, RopeConfig, RotarySpec)

EXPERTS, TOP = 32, 4


def configs(W: int, H: int, G: int, ff: int, window: int, layers: int, vocab: int) -> Dict[str, ModelConfig]:
    def latent(**kw):
        return LatentAttnSpec(**{**dict(heads=W // 64, dim=64, rot_dim=32, vdim=64, q_rank=3 * W // 8, kv_rank=256, scale=96 ** -0.5,
                                        rot=RotarySpec(32, 1.0e5, False), sink=True, window=window), **kw})
    moe, rec = MoeSpec(EXPERTS, TOP, 3 * W // 8, 3 * W // 8), GatedLinearSpec(W // 128, 128, 128)
    specs = [LayerSpec(None, moe if i else PolyNormSpec(ff), None, rec) if i % 2 == 0 else LayerSpec(latent(kv_from=1 if i == 5 else None), moe)
             for i in range(layers)]
    one = ModelConfig.of_layers(specs, architecture="Rapisun", model_type="rapisun", vocab_size=vocab, hidden_size=W, input_conv=4)
    two = ModelConfig(architecture="Qwen3NextForCausalLM", model_type="qwen3_next", vocab_size=vocab, hidden_size=W, num_layers=layers,
                      num_heads=H, num_kv_heads=G, head_dim=128, intermediate_size=ff, num_experts=EXPERTS, num_experts_per_tok=TOP,
                      moe_intermediate_size=W // 4, shared_expert_intermediate_size=W // 4, rope=RopeConfig(theta=5e5),
                      linear_num_key_heads=W // 128, linear_num_value_heads=W // 128, linear_key_head_dim=128, linear_value_head_dim=128,
                      attn_output_gate=True, zero_centered_norm=True, layer_types=[("linear_attention", "full_attention")[i % 2] for i in range(layers)])
    return {"rapisun": one, "qwen3-next (moe)": two}


def _sequences(cfg: ModelConfig, B: int, qlen: int, ctx: int, copies: int):
    """Caches of one layer with scattered pages, and the batch of a step that brings every sequence's last ``qlen`` tokens."""
    from ..batch import SeqChunk, build_batch
    from ..kv import KVCache
    per = (ctx + 15) // 16 + 1
    kvs = [KVCache(cfg, 1 + B * per, B, per, "bf16", "cuda", "tiles") for _ in range(copies)]
    for kv in kvs:
        perm = torch.randperm(B * per, generator=torch.Generator().manual_seed(0)).tolist()
        for b in range(B):
            kv.set_pages(b, [1 + p for p in perm[b * per:(b + 1) * per]])
        for t in (*kv.kv.values(), *kv.rec_state.values(), *kv.conv_state.values(), *kv.qkv_state.values(), *kv.input_state.values()):
            t.normal_()
        _ = kv.block_table
    return kvs, build_batch([SeqChunk(b, [0] * qlen, ctx - qlen) for b in range(B)], kvs[0].block_table_host, "cuda")


def _latent_mixer(a: LatentAttnSpec):
    from ..linear import Linear
    from ..models.qwen3 import LatentAttn, Mixer
    M, A = Mixer(), LatentAttn(a, "cuda")
    M.attn, M.cols = A, {"q": 0, "kv": a.q_rank}
    A.sink, A.q_norm, A.c_norm = torch.randn(a.heads, device="cuda"), torch.ones(a.q_rank, device="cuda"), torch.ones(a.kv_rank, device="cuda")
    A.uq = Linear.from_dense(torch.randn(a.heads * (a.dim + a.rot_dim), a.q_rank, device="cuda") * a.q_rank ** -0.5)
    A.set_maps(*[torch.randn(a.heads * k, a.kv_rank, device="cuda") * a.kv_rank ** -0.5 for k in (a.dim, a.vdim)], torch.bfloat16)
    return M


def kernels(sizes, window: int, add: Callable, graph_ms: Callable, like_attention: Callable, like_recurrence: Callable, ops) -> None:
    """Timings through ``add(kernel, model, ms, bytes, flops)``; ``like_*`` time the relative's kernels."""
    W, H, G, ff = sizes
    both = configs(W, H, G, ff, window, 2, 1024)
    own, rel = both.values()
    names = list(both)
    a, rec = own.layer_specs[1].attn, own.layer_specs[0].rec
    one = ModelConfig.of_layers([LayerSpec(a)], architecture="Rapisun")
    Hl, D, bf = a.heads, a.kv_rank + a.rot_dim, 2.0
    M = _latent_mixer(a)
    for label, B, qlen, ctx, copies in (("decode 256x1024", 256, 1, 1024, 3), ("decode 32x1024", 32, 1, 1024, 16),
                                        ("prefill 4x1024", 4, 1024, 1024, 4), ("prefill 1x8192", 1, 8192, 8192, 2)):
        kvs, batch = _sequences(one, B, qlen, ctx, copies)
        T = B * qlen
        q = torch.randn(T, Hl * (a.dim + a.rot_dim), device="cuda").bfloat16()
        out = torch.empty(T, Hl * a.vdim, dtype=torch.bfloat16, device="cuda")
        keys = sum(min(i + 1, window) for i in range(ctx - qlen, ctx))
        first = max(ctx - qlen - window + 1, 0)
        seen = B * (ctx - first)                         # cached vectors that are read
        io = T * Hl * (a.dim + a.rot_dim + a.vdim) * bf
        if qlen == 1:
            nb = seen * D * bf + T * Hl * (D + a.kv_rank) * bf
            qe, lat = torch.randn(T, Hl, D, device="cuda").bfloat16(), torch.empty(T, Hl * a.kv_rank, dtype=torch.bfloat16, device="cuda")
            core = [lambda kv=kv: ops.latent_rows(qe, M, batch, kv, 0, 1, 1, lat) for kv in kvs]
            add("attention " + label, names[0], graph_ms(core), nb, 2.0 * B * Hl * keys * (D + a.kv_rank))
            add("attention with the maps " + label, names[0], graph_ms([lambda kv=kv: ops.latent_attend(q, M, batch, kv, 0, out) for kv in kvs]),
                seen * D * bf + io + Hl * (a.dim + a.vdim) * a.kv_rank * bf, 2.0 * B * Hl * (keys * (D + a.kv_rank) + (a.dim + a.vdim) * a.kv_rank))
        else:
            fl = 2.0 * B * Hl * keys * (a.dim + a.rot_dim + a.vdim)
            x = ops._expand_latents(M, batch, kvs[0], 0, ops.LATENT_SHORT)
            add("attention " + label, names[0], graph_ms([lambda kv=kv: ops._expanded_attention(q, M, batch, kv, x, ops.LATENT_SHORT, out) for kv in kvs]),
                seen * Hl * (a.dim + a.rot_dim + a.vdim) * bf + io, fl)
            wide = seen * Hl * (a.dim + a.vdim)
            add("keys and values by head " + label, names[0], graph_ms([lambda kv=kv: ops._expand_latents(M, batch, kv, 0, ops.LATENT_SHORT) for kv in kvs]),
                seen * D * bf + (wide + seen * Hl * a.rot_dim) * bf + Hl * (a.dim + a.vdim) * a.kv_rank * bf, 2.0 * wide * a.kv_rank)
        if B == 256 or qlen == 1024:
            proj = torch.randn(T, a.q_rank + D, device="cuda").bfloat16()
            nb = 2 * T * (a.q_rank + D) * bf
            add("page write " + label, names[0], graph_ms([lambda kv=kv: ops.latent_prep(proj, M, batch, kv, 0, 1e-6) for kv in kvs]), nb)
        del kvs, q, out
        torch.cuda.empty_cache()
        like_attention(label, B, qlen, ctx, rel, names[1])
    from ..models.qwen3 import Mixer, Recurrence
    cfg = ModelConfig.of_layers([LayerSpec(rec=rec)], architecture="Rapisun", hidden_size=W, input_conv=4)
    R, M = Recurrence(rec, "gated", rec.heads), Mixer()
    n = rec.heads * rec.dim
    M.rec, M.cols = R, {"q": 0, "f": n, "v": 2 * n}
    R.A, R.dt_bias, R.norm_w = torch.rand(n, device="cuda"), torch.full((n,), 3.0, device="cuda"), torch.ones(rec.vdim, device="cuda")
    taps = torch.randn(4, W, device="cuda")
    for label, B, qlen, copies in (("decode 256", 256, 1, 3), ("decode 8", 8, 1, 16), ("prefill 8x1024", 8, 1024, 2), ("prefill 1x8192", 1, 8192, 2)):
        kvs, batch = _sequences(cfg, B, qlen, qlen + 8, copies)
        T = B * qlen
        proj, o = torch.randn(T, 2 * n + rec.heads * rec.vdim, device="cuda").bfloat16(), torch.empty(T, rec.heads * rec.vdim, device="cuda")
        out, x = torch.empty(T, rec.heads * rec.vdim, dtype=torch.bfloat16, device="cuda"), torch.randn(T, W, device="cuda")
        nv = T * rec.heads * rec.vdim
        add("recurrence " + label, names[0], graph_ms([lambda kv=kv: ops.recur(None, proj, None, M, batch, kv, 0, o) for kv in kvs]),
            proj.numel() * bf + B * n * rec.vdim * 8.0 + 4.0 * nv, 4.0 * nv * rec.dim)
        add("norm " + label, names[0], graph_ms([lambda: ops.gated_norm(o, proj, M, 1e-6, out)] * copies), nv * 6.0)
        add("convolution " + label, names[0], graph_ms([lambda kv=kv: ops.input_conv(x, taps, batch, kv, 0, torch.bfloat16) for kv in kvs]),
            T * W * 6.0 + B * W * 24.0)
        del kvs, proj, o, out, x
        torch.cuda.empty_cache()
        like_recurrence(label, B, qlen, copies, rel, names[1])
    _feed_forward(own, rel, names, W, ff, add, graph_ms, ops)
    for T in (256, 8192):
        c = max(2, int(400e6 // (T * W * 16)))
        y, w = torch.randn(T, W, device="cuda").bfloat16(), torch.ones(W, device="cuda")
        xs = [torch.randn(T, W, device="cuda") for _ in range(c)]
        add(f"residual + norm, {T} rows", names[0], graph_ms([lambda x=x: ops.branch_norm(x, y, w, 1e-6) for x in xs]), T * W * 12.0)
        rs = [torch.randn(T, W, device="cuda").bfloat16() for _ in range(c)]
        add(f"residual + norm, {T} rows", names[1], graph_ms([lambda r=r: ops.norm(y, r, w.bfloat16(), 1e-6) for r in rs]), T * W * 8.0)
        del xs, rs


def _feed_forward(own: ModelConfig, rel: ModelConfig, names, W: int, ff: int, add, graph_ms, ops) -> None:
    """A layer's routed experts with the shared one and the sum over the chosen ones, and the dense activations."""
    from ..models.qwen3 import Model
    from ..models.rapisun import Rapisun
    for T in (256, 8192):
        h = torch.randn(T, W, device="cuda").bfloat16()
        x, w = torch.zeros(T, W, device="cuda"), torch.ones(W, device="cuda")
        for name, cls, cfg in ((names[0], Rapisun, own), (names[1], Model, rel)):
            c = copy.copy(cfg)
            if cfg is own:
                c.layer_specs, c.num_layers, c.layer_types = cfg.layer_specs[1:2], 1, cfg.layer_types[1:2]
            else:
                c.num_layers, c.layer_types = 1, cfg.layer_types[1:2]
            ms = [cls.random_init(c, seed=i, device="cuda", ops=ops) for i in range(3)]
            e = own.layer_specs[1].mlp
            per = 2 * W * e.ff                           # weights of an expert: the relative's three matrices are as large
            hit = EXPERTS if T * TOP >= EXPERTS * 8 else EXPERTS * (1 - (1 - TOP / EXPERTS) ** T)
            nb, fl = (hit + 1) * per * 2.0 + T * W * 4.0, 2.0 * T * (TOP + 1) * per
            if cfg is own:
                calls = [lambda m=m: ops.branch_norm(x, m._mlp(m.layers[0].mlp, h)[0], w, 1e-6) for m in ms]
                nb += T * W * 8.0
            else:
                res = torch.zeros(T, W, device="cuda").bfloat16()
                calls = [lambda m=m: ops.norm(m._mlp(m.layers[0].mlp, h)[0], res, w.bfloat16(), 1e-6) for m in ms]
                nb += T * W * 4.0
            add(f"experts + residual + norm, {T} rows", name, graph_ms(calls), nb, fl)
            del ms, calls
            torch.cuda.empty_cache()
        z, act = [torch.randn(T, ff, device="cuda").bfloat16() for _ in range(max(2, int(300e6 // (T * ff * 2))))], torch.ones(4, device="cuda")
        add(f"dense activation, {T} rows", names[0], graph_ms([lambda t=t: ops.poly_norm(t, act, 1e-6) for t in z]), T * ff * 4.0)
        gu = [torch.randn(T, 2 * ff, device="cuda").bfloat16() for _ in range(len(z))]
        add(f"dense activation, {T} rows", names[1], graph_ms([lambda t=t: ops.silu_mul(t) for t in gu]), T * ff * 6.0)
        del z, gu
        torch.cuda.empty_cache()
