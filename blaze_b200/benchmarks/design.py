"""A model design beside its closest relative at equal size: prefill and decode throughput of a few layers of real size (random
weights, bf16), and every kernel that is the design's own beside the like kernel of the relative, with fractions of the measured
peaks.  ``bench.py --design <name>`` runs it: Sevevik against the Qwen3 decoder (equal width, heads, projections and
feed-forward), Niletar against the Qwen3-Next hybrid with a dense feed-forward (Gated DeltaNet layers with a state as large as the
state-space layers', gated attention layers with heads as the parallel ones'), Rapisun and Medodra against the Qwen3-Next hybrid with experts
(see :mod:`blaze_b200.benchmarks.rapisun` and :mod:`blaze_b200.benchmarks.medodra`); the relatives keep FP8 pages, their only format on a GPU.

Device-timed with CUDA events; kernels in captured graphs over buffers that together exceed L2.
"""
from __future__ import annotations

import copy
from typing import Callable, Dict, List

import numpy as np
import torch

from ..config import (DeltaSpec, DiffAttnSpec, GluSpec, LayerSpec, ModelConfig, RopeConfig, RotarySpec, SoftAttnSpec,
                      StateSpaceSpec)
from . import medodra, rapisun
from .kernels import peaks

# width, query heads, key/value heads, feed-forward
SIZES = {"2048": (2048, 16, 8, 6144), "4096": (4096, 32, 8, 12288)}
WINDOW = 1024


RELATIVE = {"sevevik": "qwen3", "niletar": "qwen3-next (dense)", "rapisun": "qwen3-next (moe)", "medodra": "qwen3-next (moe)"}
OWN = {"rapisun": rapisun, "medodra": medodra}          # designs whose kernels are timed in a module of their own


def configs(design: str, size: str, layers: int, vocab: int) -> Dict[str, ModelConfig]:
    """The design's configuration and its relative's."""
    W, H, G, ff = SIZES[size]
    if design in OWN:
        return OWN[design].configs(W, H, G, ff, WINDOW, layers, vocab)
    if design == "niletar":
        attn = SoftAttnSpec(H, G, 128, 128, 128 ** -0.5, RotarySpec(128, 5.0e5, True, 8.0, 1.0, 4.0, 8192.0), True, True, True, True,
                            out_scale=0.7)
        par = LayerSpec(attn, GluSpec(ff), None, DeltaSpec(H, H, 128, 128, 4, out_scale=0.7))
        ssm = LayerSpec(None, GluSpec(ff), None, StateSpaceSpec(heads=2 * W // 64, vdim=64, state=128, groups=8, norm_groups=8, conv=4))
        one = ModelConfig.of_layers([(ssm, par)[i % 2] for i in range(layers)], architecture="Niletar", model_type="niletar",
                                    vocab_size=vocab, hidden_size=W, residual_alpha=2.0, zero_centered_norm=True)
        two = ModelConfig(architecture="Qwen3NextForCausalLM", model_type="qwen3_next", vocab_size=vocab, hidden_size=W, num_layers=layers,
                          num_heads=H, num_kv_heads=G, head_dim=128, intermediate_size=ff, rope=RopeConfig(theta=5e5),
                          linear_num_key_heads=W // 128, linear_num_value_heads=2 * W // 128, linear_key_head_dim=128,
                          linear_value_head_dim=128, attn_output_gate=True, zero_centered_norm=True,
                          layer_types=[("linear_attention", "full_attention")[i % 2] for i in range(layers)])
        return {design: one, RELATIVE[design]: two}
    a = DiffAttnSpec(heads=H, kv_heads=G, dim=64, vdim=128, scale=0.125, diff=0.5, window=WINDOW)
    sev = ModelConfig.of_layers([LayerSpec(a, GluSpec(ff, 7.0)) for _ in range(layers)], architecture="Sevevik", model_type="sevevik",
                                vocab_size=vocab, hidden_size=W, streams=4)
    qwen = ModelConfig(vocab_size=vocab, hidden_size=W, num_layers=layers, num_heads=H, num_kv_heads=G, head_dim=128,
                       intermediate_size=ff, rope=RopeConfig(theta=1e6), layer_types=["full_attention"] * layers)
    return {"sevevik": sev, "qwen3": qwen}


def _events(fn: Callable[[], None], reps: int) -> float:
    """Median milliseconds of ``fn``."""
    fn()
    torch.cuda.synchronize()
    t = []
    for _ in range(reps):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        t.append(a.elapsed_time(b))
    return sorted(t)[len(t) // 2]


def throughput(cfg: ModelConfig, steps: int, warmup: int, batch: int = 256, ctx: int = 1024) -> Dict[str, float]:
    """Prefill tokens/s (8 prompts of 1024 in one step; one prompt of 8192) and decode tokens/s at ``batch`` x ``ctx``."""
    from ..llm import LLM
    longest = 8192
    llm = LLM(cfg, device="cuda", kv_tokens=max(batch * (ctx + steps + warmup + 64), 2 * longest), max_seqs=batch, max_model_len=longest + 64,
              enable_prefix_caching=False, seed=1, chunk=8192)
    eng, V = llm.engine, cfg.vocab_size
    g = torch.Generator().manual_seed(1)
    out: Dict[str, float] = {}

    def prefill(n_seqs, n):
        prompts = torch.randint(0, V, (n_seqs, n), generator=g).tolist()

        def once():
            seqs = [eng.open_from() for _ in range(n_seqs)]
            eng.forward(eng.plan([(s, p, 1) for s, p in zip(seqs, prompts)]), "greedy")
            for s in seqs:
                eng.close(s)
        ms = _events(once, 5)
        return {"ms": round(ms, 3), "tok_s": round(n_seqs * n / ms * 1e3)}
    out["prefill_8x1024"] = prefill(8, 1024)
    out["prefill_1x8192"] = prefill(1, 8192)
    seqs = [eng.open_from() for _ in range(batch)]
    for i in range(0, batch, 8):
        part = seqs[i:i + 8]
        eng.forward(eng.plan([(s, torch.randint(0, V, (ctx,), generator=g).tolist(), 0) for s in part]), "none")
    zeros = [0]

    def decode(feedback):
        return eng.forward(eng.plan([(s, zeros, 1) for s in seqs]), "greedy", feedback=feedback)
    for k in range(max(warmup, 3)):
        decode(False)
    torch.cuda.synchronize()
    feed = eng.can_feed_back(batch)
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(steps):
        decode(feed)
    b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / steps
    wbytes = llm.model.weight_bytes() - llm.model.embed.numel() * llm.model.embed.element_size()
    out["decode_%dx%d" % (batch, ctx)] = {"ms": round(ms, 4), "tok_s": round(batch / ms * 1e3), "weight_mb": round(wbytes / 1e6), "captured": feed}
    one = seqs[:1]
    for s in seqs[1:]:
        eng.close(s)
    for _ in range(4):
        eng.forward(eng.plan([(one[0], zeros, 1)]), "greedy")
    torch.cuda.synchronize()
    a.record()
    for _ in range(steps):
        eng.forward(eng.plan([(one[0], zeros, 1)]), "greedy", feedback=eng.can_feed_back(1))
    b.record()
    torch.cuda.synchronize()
    out["decode_1x%d" % ctx] = {"ms": round(a.elapsed_time(b) / steps, 4)}
    eng.check_status()
    del llm, eng
    torch.cuda.empty_cache()
    return out


def _graph_ms(calls: List[Callable[[], object]], reps: int = 7) -> float:
    """Milliseconds per call of a captured graph of ``calls`` (each on buffers of its own)."""
    for c in calls:
        c()
    torch.cuda.synchronize()
    keep = []
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in calls:
            keep.append(c())
    return _events(graph.replay, reps) / len(calls)


def _attention(ops, cfg: ModelConfig, B: int, qlen: int, ctx: int, copies: int):
    """(attention calls, page-write calls, bytes of keys and values read, flops, bytes of the rows before the page write) of one
    attention layer."""
    from ..batch import SeqChunk, build_batch
    from ..kv import KVCache
    own = bool(cfg.layer_specs)
    sev = own and cfg.layer_specs[0].attn is not None and cfg.layer_specs[0].attn.maps == 2
    per = (ctx + 15) // 16 + 1
    if own:
        cfg = ModelConfig.of_layers([next(LayerSpec(s.attn) for s in cfg.layer_specs if s.attn is not None)], architecture=cfg.architecture)
    else:
        cfg = copy.copy(cfg)
        cfg.num_layers, cfg.layer_types = 1, ["full_attention"]
    kvs = [KVCache(cfg, 1 + B * per, B, per, "bf16" if own else "fp8", "cuda", "tiles" if own else "umma") for _ in range(copies)]
    G = cfg.num_kv_heads
    for kv in kvs:
        perm = torch.randperm(B * per, generator=torch.Generator().manual_seed(0)).tolist()
        for b in range(B):
            kv.set_pages(b, [1 + p for p in perm[b * per:(b + 1) * per]])
        if own:
            kv.kv[0].normal_()
        else:
            kv.kv[0].copy_(torch.randint(0, 120, kv.kv[0].shape, dtype=torch.uint8, device="cuda"))
    chunks = [SeqChunk(b, [0] * qlen, ctx - qlen) for b in range(B)]
    batch = build_batch(chunks, kvs[0].block_table_host, "cuda", attn_group=0 if own else cfg.num_heads // G)
    T, H = B * qlen, cfg.num_heads
    seen = lambda i: min(i + 1, WINDOW) if sev else i + 1      # noqa: E731
    keys = sum(seen(i) for i in range(ctx - qlen, ctx))        # of one sequence's rows
    first = max(ctx - qlen - WINDOW + 1, 0) if sev else 0
    for kv in kvs:
        _ = kv.block_table
    if sev:
        class A:
            spec, lam = cfg.layer_specs[0].attn, 0.6
        a = A.spec
        qkv = torch.randn(T, a.heads * 2 * a.dim + a.kv_heads * (2 * a.dim + a.vdim), device="cuda").bfloat16()
        calls = [lambda kv=kv: ops.diff_attention(qkv, A, batch, kv, 0, 1e-6, store=False) for kv in kvs]
        write = [lambda kv=kv: ops.diff_store(qkv, A, batch, kv, 0) for kv in kvs]
        flops = 2.0 * B * H * keys * (2 * a.dim + 2 * a.vdim)
        return calls, write, B * (ctx - first) * G * (2 * a.dim + a.vdim) * 2.0, flops, T * qkv.shape[1] * 2.0
    D = cfg.head_dim
    if own:
        from ..models.qwen3 import Mixer, SoftAttn
        a, M = cfg.layer_specs[0].attn, Mixer()
        M.attn = SoftAttn(a, "cuda", torch.randn(H))
        at = [H * D, G * D, G * a.vdim, H * a.vdim]
        M.cols = {n: sum(at[:i]) for i, n in enumerate(("q", "k", "v", "gate"))}
        proj, q = torch.randn(T, sum(at), device="cuda").bfloat16(), torch.randn(T, H * D, device="cuda").bfloat16()
        out = torch.empty(T, H * a.vdim, dtype=torch.bfloat16, device="cuda")
        calls = [lambda kv=kv: ops.soft_attend(q, proj, M, batch, kv, 0, out) for kv in kvs]
        write = [lambda kv=kv: ops.attn_prep_pages(proj, M, batch, kv, 0, 1e-6) for kv in kvs]
        return calls, write, B * ctx * G * (D + a.vdim) * 2.0 + T * H * a.vdim * 2.0, 2.0 * B * H * keys * (D + a.vdim), T * sum(at[:3]) * 2.0

    class M:
        inv_freq, rope_scale, kv_rotate = torch.ones(D // 2, device="cuda"), 1.0, False

    class N:
        heads, kv_heads, q_norm, k_norm = H, G, torch.ones(D, device="cuda").bfloat16(), torch.ones(D, device="cuda").bfloat16()
    M.cfg = cfg
    q = torch.randn(T, H, D, device="cuda").bfloat16()
    qkv = torch.randn(T, (H * (2 if cfg.attn_output_gate else 1) + 2 * G) * D, device="cuda").bfloat16()
    calls = [lambda kv=kv: ops.attention(q, M, batch, kv, 0, D ** -0.5) for kv in kvs]
    write = [lambda kv=kv: ops.attn_prep_store(qkv, N, M, batch, kv, 0, None) for kv in kvs]
    return calls, write, B * ctx * G * 2.0 * D, 4.0 * B * H * keys * D, T * qkv.shape[1] * 2.0


def _recurrence(ops, cfg: ModelConfig, rec, B: int, qlen: int, copies: int):
    """(convolution, recurrence, gated norm) calls and the bytes and flops of each, of one recurrent layer: ``rec`` is the design's
    spec, or None for the relative's Gated DeltaNet with the value heads ``cfg`` names.  The products counted are those of the
    recurrence as it is written (three with the state per token for the delta rule, two for the state space)."""
    from ..batch import SeqChunk, build_batch
    from ..kv import KVCache
    from ..models.qwen3 import Gdn, Mixer, Recurrence
    T, bf, cuda = B * qlen, torch.bfloat16, dict(device="cuda")
    if rec is not None:
        cfg = ModelConfig.of_layers([LayerSpec(rec=rec)], architecture=cfg.architecture)
    else:
        cfg = copy.copy(cfg)
        cfg.num_layers, cfg.layer_types = 1, ["linear_attention"]
    kvs = [KVCache(cfg, 2, B, 1, "bf16", "cuda", "tiles" if rec is not None else "logical") for _ in range(copies)]
    for kv in kvs:
        kv.rec_state[0].normal_()
    batch = build_batch([SeqChunk(b, [0] * qlen, 0) for b in range(B)], np.zeros((B, (qlen + 15) // 16), np.int32), "cuda")
    batch.ctx_len.fill_(qlen + 8)                       # none of them starts here
    C, state = kvs[0].conv_state[0].shape[1], kvs[0].rec_state[0]
    H, dk, dv = state.shape[1:]
    io, st = T * C * 2.0, B * H * dk * dv * 8.0
    if rec is None:
        G = Gdn()
        G.k_heads, G.v_heads = cfg.linear_num_key_heads, H
        G.conv_w, G.norm_w = torch.randn(C, 4, **cuda).to(bf), torch.ones(dv, **cuda).to(bf)
        G.A_log, G.dt_bias = torch.zeros(H, **cuda), torch.full((H,), -4.0, **cuda)
        x, y, ab = torch.randn(T, C, **cuda).to(bf), torch.randn(T, C, **cuda).to(bf), torch.randn(2, T, H, **cuda).to(bf)
        o, z = torch.empty(T, H, dv, dtype=bf, **cuda), torch.randn(T, H * dv, **cuda).to(bf)

        class M:
            pass
        M.cfg = cfg
        calls = ([lambda kv=kv: ops.gdn_conv(x, G, batch, kv, 0) for kv in kvs],
                 [lambda kv=kv: ops.gdn_rule(y, ab[0], ab[1], G, M, batch, kv, 0, o) for kv in kvs],
                 [lambda: ops.gdn_norm(o, z, G, cfg)] * copies)
        gates, out_bytes, prods = T * H * 4.0, 2.0, 3
    else:
        delta = isinstance(rec, DeltaSpec)
        R, M = Recurrence(rec, "delta" if delta else "ssm", H if delta else rec.norm_groups), Mixer()
        M.rec, M.cols = R, {"conv": 0, "beta": C, "dt": C, "z": 0}
        R.conv_w, R.conv_b = torch.randn(C, rec.conv, **cuda).to(bf), None if delta else torch.randn(C, **cuda)
        R.A, R.dt_bias = torch.ones(H, **cuda), torch.full((H * (dk if delta else 1),), -4.0, **cuda)
        R.D, R.norm_w = torch.ones(H, **cuda), torch.ones(dv if delta else H * dv, **cuda)
        x, y = torch.randn(T, C + H, **cuda).to(bf), torch.randn(T, C, **cuda).to(bf)
        low, o = torch.randn(T, H * (dk + dv), **cuda).to(bf), torch.empty(T, H * dv, **cuda)
        out = torch.empty(T, H * dv, dtype=bf, **cuda)
        calls = ([lambda kv=kv: ops.short_conv(x, M, batch, kv, 0) for kv in kvs],
                 [lambda kv=kv: ops.recur(y, x, low, M, batch, kv, 0, o) for kv in kvs],
                 [lambda: ops.gated_norm(o, x if not delta else low, M, 1e-6, out)] * copies)
        gates, out_bytes, prods = T * H * (dk + 1 if delta else 1) * 2.0, 4.0, 3 if delta else 2
    n = T * H * dv
    return calls, ((2 * io, 0.0), (io + gates + st + out_bytes * n, 2.0 * prods * n * dk), (n * (out_bytes + 4.0), 0.0))


def kernels(design: str, size: str) -> List[Dict]:
    from ..linear import Linear
    from ..models.sevevik import StaticStreams
    from ..ops import get_ops
    ops, pk = get_ops("cuda"), peaks()
    W, H, G, ff = SIZES[size]
    rows: List[Dict] = []

    def add(name, model, ms, nbytes=0.0, flops=0.0):
        bound = max(nbytes / pk["hbm_gbs"] / 1e6, flops / pk["bf16_tflops"] / 1e9)
        rows.append({"kernel": name, "model": model, "us": round(ms * 1e3, 2), "roofline_frac": round(bound / ms, 3),
                     "bound": "hbm" if nbytes / pk["hbm_gbs"] / 1e6 >= flops / pk["bf16_tflops"] / 1e9 else "bf16 tensor"})
    if design in OWN:
        def like_attention(label, B, qlen, ctx, cfg, model):
            calls, write, kvb, flops, rowb = _attention(ops, cfg, B, qlen, ctx, 2 if B == 256 else 8 if qlen == 1 else 4)
            add("attention " + label, model, _graph_ms(calls), kvb + B * qlen * H * 128 * 4.0, flops)
            if B == 256 or qlen == 1024:
                add("page write " + label, model, _graph_ms(write), 2 * rowb)
            del calls, write
            torch.cuda.empty_cache()

        def like_recurrence(label, B, qlen, copies, cfg, model):
            calls, cost = _recurrence(ops, cfg, None, B, qlen, copies)
            for part, c, (nbytes, flops) in zip(("convolution", "recurrence", "norm"), calls, cost):
                add(f"{part} {label}", model, _graph_ms(c), nbytes, flops)
            del calls
            torch.cuda.empty_cache()
        OWN[design].kernels(SIZES[size], WINDOW, add, _graph_ms, like_attention, like_recurrence, ops)
        assert ops.take_status() == 0
        return rows
    for name, B, qlen, ctx, copies in (("attention decode 256x1024", 256, 1, 1024, 2), ("attention decode 32x1024", 32, 1, 1024, 8),
                                       ("attention prefill 4x1024", 4, 1024, 1024, 4), ("attention prefill 1x8192", 1, 8192, 8192, 2)):
        for model, cfg in configs(design, size, 2, 1024).items():
            calls, write, kvb, flops, rowb = _attention(ops, cfg, B, qlen, ctx, copies)
            out = B * qlen * H * 128 * 2.0
            add(name, model, _graph_ms(calls), kvb + out + B * qlen * H * 128 * 2.0, flops)
            if qlen == 1024 or B == 256:
                add("page write " + name.split(" ", 1)[1], model, _graph_ms(write), 2 * rowb if model != "sevevik" else 2.0 * B * qlen * G * 256 * 2)
            del calls, write
            torch.cuda.empty_cache()
    if design == "niletar":
        cfgs = configs(design, size, 2, 1024)
        own, rel = cfgs[design], cfgs[RELATIVE[design]]
        for label, B, qlen, copies in (("decode 256", 256, 1, 2), ("decode 8", 8, 1, 8), ("prefill 8x1024", 8, 1024, 2), ("prefill 1x8192", 1, 8192, 2)):
            for kind, spec in (("state space", own.layer_specs[0].rec), ("delta rule", own.layer_specs[1].rec)):
                like = copy.copy(rel)
                if kind == "delta rule":
                    like.linear_num_value_heads = like.linear_num_key_heads
                for model, cfg, rec in ((design, own, spec), (RELATIVE[design], like, None)):
                    calls, cost = _recurrence(ops, cfg, rec, B, qlen, copies)
                    for part, c, (nbytes, flops) in zip(("convolution", "recurrence", "gated norm"), calls, cost):
                        add(f"{part} ({kind}) {label}", model, _graph_ms(c), nbytes, flops)
                    del calls
                    torch.cuda.empty_cache()
    for T in (256, 8192):
        n = max(2, int(400e6 // (T * W * 16)))
        S = 4
        if design == "niletar":
            y, w = torch.randn(T, W, device="cuda").bfloat16(), torch.ones(W, device="cuda")
            xs = [torch.randn(T, W, device="cuda") for _ in range(n)]
            add(f"residual + norm, {T} rows", design, _graph_ms([lambda x=x: ops.residual_norm(x, 2.0, y, w, 1e-6) for x in xs]), T * W * (4 + 2 + 4 + 2))
            rs = [torch.randn(T, W, device="cuda").bfloat16() for _ in range(n)]
            add(f"residual + norm, {T} rows", RELATIVE[design], _graph_ms([lambda r=r: ops.norm(y, r, w.bfloat16(), 1e-6) for r in rs]), T * W * 8)
            del xs, rs
            continue
        w = StaticStreams(torch.randn(S), torch.randn(S, S), torch.randn(S), 1.0, "cuda", torch.bfloat16)
        nw = torch.ones(W, device="cuda")
        y = torch.randn(T, W, device="cuda").bfloat16()
        xs = [torch.randn(T, S, W, device="cuda") for _ in range(n)]
        add(f"streams + norm, {T} rows", "sevevik", _graph_ms([lambda x=x: ops.streams_step(x, y, w, w, nw, 1e-6) for x in xs]),
            T * W * (2 * 4 * S + 2 + 2))
        del xs
        n = max(2, int(400e6 // (T * W * 4)))
        rs = [torch.randn(T, W, device="cuda").bfloat16() for _ in range(n)]
        nb = nw.bfloat16()
        add(f"residual + norm, {T} rows", "qwen3", _graph_ms([lambda r=r: ops.norm(y, r, nb, 1e-6) for r in rs]), T * W * (2 + 2 + 2 + 2))
        del rs
        x = torch.randn(T, W, device="cuda").bfloat16()
        ws = torch.randn(2 * ff, W, device="cuda") * 0.02
        copies = max(1, min(8, int(300e6 // (2 * ff * W * 2)) + 1))
        for model in ("sevevik", "qwen3"):
            lins = [Linear.from_dense(ws) for _ in range(copies)]
            f = (lambda l: ops.linear_glu(l, x, 7.0)) if model == "sevevik" else (lambda l: ops.linear_swiglu(l, x))
            add(f"gate/up GEMM + activation, {T} rows", model, _graph_ms([lambda l=l: f(l) for l in lins]),
                2.0 * (2 * ff * W + T * W + T * ff), 4.0 * T * ff * W)
            del lins
        del ws
        torch.cuda.empty_cache()
    assert ops.take_status() == 0
    return rows


def run(design: str, sizes, steps: int, warmup: int, layers: int = 8, vocab: int = 32768, kernels_only: bool = False) -> Dict:
    res: Dict = {"design": design, "beside": f"{RELATIVE[design]} (equal size, bf16 weights, FP8 pages)", "layers": layers, "vocab": vocab,
                 "window": WINDOW if design in ("sevevik", "rapisun") else None, "data": "synthetic token ids, random-init weights", "throughput": {}, "kernels": {}}
    for size in sizes:
        res["kernels"][size] = kernels(design, size)
        if not kernels_only:
            res["throughput"][size] = {m: throughput(c, steps, warmup) for m, c in configs(design, size, layers, vocab).items()}
    return res
