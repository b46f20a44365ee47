"""Sevevik: a decoder of differential-attention layers (sliding window, no rotation) and clamped gated feed-forwards on static
residual streams, described layer by layer in its configuration (``ModelConfig.layer_specs``).

Every sublayer reads a weighted sum of the streams and is written back through a mix of all of them; weights are per layer, not
per token (:class:`StaticStreams`).  The streams, their mixes and all norms are fp32.  A layer may use another layer's tensors,
with keys and values of its own.  Tensor names: ``embed``, ``l<i>.{norm1,norm2}``, ``l<i>.mix.{q,k,v,o,lq1,lk1,lq2,lk2}``,
``l<i>.mlp.{gate,up,down}``, ``l<i>.{hc1,hc2}.{in,out,mix}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..batch import StepBatch
from ..config import ModelConfig
from ..kv import KVCache
from ..linear import Linear
from ..quant import Format
from . import qwen3
from .qwen3 import ClampedGlu, DiffAttn, Layer, Model, TPInfo


class StaticStreams:
    """Weights of one sublayer on the residual streams: ``read [S]``, ``mix [S, S]`` (from, to) and ``out [S]`` (the residual
    multiplier included), fp32; ``dtype`` is the activations'."""

    def __init__(self, read, mix, out, mult: float, device, dtype):
        self.read = read.float().to(device).contiguous()
        self.mix = mix.float().to(device).contiguous()
        self.out = (out.float() * mult).to(device).contiguous()
        self.dtype = dtype


class Sevevik(Model):
    kernel_sources = ("host", "fused_ops", "gemm_tc", "gemm_sk", "gemm_wide", "moe_gemm", "gemm_simple", "streams", "attn_maps",
                      "attn_maps_tc", "sampling")
    cuda_dtypes = (torch.bfloat16, torch.float32)
    fp8_pages = False

    @classmethod
    def _supports(cls, cfg: ModelConfig) -> None:
        if not cfg.layer_specs:
            raise ValueError("a Sevevik configuration lists its layers")
        if not 1 <= cfg.streams <= 16:
            raise ValueError(f"{cfg.streams} residual streams: 1 to 16 are supported")

    def __init__(self, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None,
                 first_layer: int = 0, last_layer: Optional[int] = None):
        super().__init__(cfg, device, dtype, tp, ops, first_layer, last_layer)
        if self.tp.world > 1 or not (self.is_first_stage and self.is_last_stage):
            raise ValueError("Sevevik models run on one rank (no tensor or pipeline parallelism)")
        if dtype not in self.cuda_dtypes:
            raise ValueError(f"Sevevik models run in bfloat16 or float32, not {dtype}")

    # ================================================================== construction
    @classmethod
    def random_init(cls, cfg: ModelConfig, fmt: Format = Format.DENSE, seed: int = 0, device="cpu", dtype=torch.bfloat16,
                    tp: Optional[TPInfo] = None, std: float = 0.02, ops=None, first_layer: int = 0,
                    last_layer: Optional[int] = None, **_) -> "Sevevik":
        """Random weights under the checkpoint's tensor names (``std`` of the matrices; mixes near an average and an identity)."""
        if fmt != Format.DENSE:
            raise ValueError("Sevevik weights are bf16 or fp32 (weight format 'dense')")
        m = cls(cfg, device, dtype, tp, ops, first_layer, last_layer)
        gen = torch.Generator(device=device).manual_seed(seed)
        S, W = cfg.streams, cfg.hidden_size

        def rnd(*shape, s=std, base=0.0):
            return torch.randn(*shape, generator=gen, device=device) * s + base

        def get(name: str) -> torch.Tensor:
            leaf = name.rsplit(".", 1)[-1]
            if name in ("embed", "head"):
                return rnd(cfg.vocab_size, W)
            if leaf in ("norm1", "norm2", "norm"):
                return rnd(W, s=0.1, base=1.0)
            spec = cfg.layer_specs[int(name[1:name.index(".")])]
            if ".hc" in name:
                return {"in": lambda: rnd(S, s=0.2, base=1.0 / S), "out": lambda: rnd(S, s=0.2, base=1.0),
                        "mix": lambda: rnd(S, S, s=0.1) + torch.eye(S, device=device)}[leaf]()
            a = spec.attn
            shapes = {"q": (a.heads * 2 * a.dim, W), "k": (a.kv_heads * 2 * a.dim, W), "v": (a.kv_heads * a.vdim, W), "o": (W, a.heads * a.vdim)}
            if ".mix." in name:
                return rnd(*shapes[leaf]) if leaf in shapes else rnd(a.dim, s=0.1)
            return rnd(W, spec.mlp.ff) if leaf == "down" else rnd(spec.mlp.ff, W)
        return m._assemble(get, lambda name: True)

    @classmethod
    def load(cls, model_dir: str, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None, first_layer: int = 0,
             last_layer: Optional[int] = None, cfg: Optional[ModelConfig] = None) -> "Sevevik":
        from ..weights import Checkpoint
        ck = Checkpoint.open(model_dir)
        m = cls(cfg or ModelConfig.load(model_dir), device, dtype, tp, ops, first_layer, last_layer)
        return m._assemble(ck.get, ck.__contains__)

    def _assemble(self, get, has) -> "Sevevik":
        """The layers from tensors by name (``get``; ``has``: is there one)."""
        cfg, dev, dt = self.cfg, self.device, self.dtype
        S, W = cfg.streams, cfg.hidden_size

        def tensor(name: str, *shape: int) -> torch.Tensor:
            t = get(name)
            if tuple(t.shape) != shape:
                raise ValueError(f"tensor {name} is {tuple(t.shape)}, the configuration asks for {shape}")
            return t

        def linear(names: List[str], rows: List[int], cols: int) -> Linear:
            lin = Linear.from_dense(torch.cat([tensor(n, r, cols).to(dev, dt) for n, r in zip(names, rows)]), dtype=dt)
            lin.name = "+".join(names)
            return lin

        def norm(name: str) -> torch.Tensor:
            return tensor(name, W).to(dev, torch.float32).contiguous()

        def streams(prefix: str) -> StaticStreams:
            if S == 1 and not has(prefix + "mix"):            # one stream without mixes: the plain residual sum
                one = torch.ones(1)
                return StaticStreams(one, one.view(1, 1), one, cfg.residual_mult, dev, dt)
            return StaticStreams(tensor(prefix + "in", S), tensor(prefix + "mix", S, S), tensor(prefix + "out", S), cfg.residual_mult, dev, dt)

        self.embed = tensor("embed", cfg.vocab_size, W).to(dev, dt).contiguous()
        for i, spec in enumerate(cfg.layer_specs):
            if spec.weights_of is not None:
                self.layers.append(None)
                continue
            L, p, a = Layer(), f"l{i}.", spec.attn
            L.kind = cfg.layer_type(i)
            L.input_norm, L.hc_attn = norm(p + "norm1"), streams(p + "hc1.")
            A = L.attn = DiffAttn(a)
            A.qkv = linear([p + "mix.q", p + "mix.k", p + "mix.v"], [a.heads * 2 * a.dim, a.kv_heads * 2 * a.dim, a.kv_heads * a.vdim], W)
            A.o = linear([p + "mix.o"], [W], a.heads * a.vdim)
            A.lam = DiffAttn.map_weight(*(tensor(p + "mix." + n, a.dim) for n in ("lq1", "lk1", "lq2", "lk2")), a.diff)
            if spec.mlp is not None:
                L.post_norm, L.hc_mlp = norm(p + "norm2"), streams(p + "hc2.")
                M = L.mlp = ClampedGlu(spec.mlp.limit)
                M.gate_up = linear([p + "mlp.gate", p + "mlp.up"], [spec.mlp.ff] * 2, W)
                M.down = linear([p + "mlp.down"], [W], spec.mlp.ff)
            self.layers.append(L)
        for i, spec in enumerate(cfg.layer_specs):
            if spec.weights_of is not None:
                self.layers[i] = self.layers[spec.weights_of]
        self.final_norm = norm("final.norm")
        self.lm_head = linear(["head"], [cfg.vocab_size], W)
        return self

    # ================================================================== forward
    def forward(self, batch: StepBatch, kv: KVCache, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The sum of the streams after the last layer, fp32 ``[T, hidden]`` (before the final norm)."""
        if hidden_in is not None or batch.embed_over:
            raise ValueError("Sevevik models take token ids only")
        ops, eps = self.ops, self.cfg.rms_norm_eps
        x = ops.streams_begin(self.embed, batch.tokens, self.cfg.embed_scale, self.cfg.streams)
        y = last = None
        dump = qwen3._DUMP_DIR and not (self.device.type == "cuda" and torch.cuda.is_current_stream_capturing())
        for gi, L in enumerate(self.layers):
            x, h = ops.streams_step(x, y, last, L.hc_attn, L.input_norm, eps)
            y, last = self._diff_attention(L.attn, h, batch, kv, gi), L.hc_attn
            if L.mlp is not None:
                x, h = ops.streams_step(x, y, last, L.hc_mlp, L.post_norm, eps)
                y, last = self._mlp(L.mlp, h, None, gi)[0], L.hc_mlp
            if dump:
                qwen3._dump(f"layer{gi:03d}_streams_sum", ops.streams_sum(x, y, last))
        if dump:
            qwen3._dump_step[0] += 1
        return ops.streams_sum(x, y, last)

    def final_hidden(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return self.ops.norm_rows(x, rows, self.final_norm, self.cfg.rms_norm_eps, self.dtype)
