"""Niletar: a post-norm decoder whose layers mix tokens with a state-space recurrence (Mamba-2), or with a gated softmax attention and
a gated delta rule side by side, described layer by layer in its configuration (``ModelConfig.layer_specs``).

``x <- norm(alpha * x + sublayer(x))`` after every sublayer; the sums, norms and recurrent states are fp32.  A layer may use another
layer's tensors, with a cache and a state of its own.  Tensor names: ``embed``, ``l<i>.{norm1,norm2}``; of a state-space mixer
``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``; of a parallel one ``l<i>.mix.left.{q,k,v}[.b]``, ``.left.{sink,g,o}``,
``l<i>.mix.right.{q,k,v}[.conv]``, ``.right.{b,A_log,norm,a1,a2,dt_bias,g1,g2,o}``; ``l<i>.mlp.{gate,up,down}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import List, Optional, Sequence, Tuple

import torch

from ..batch import StepBatch
from ..config import ModelConfig
from ..kv import KVCache
from ..linear import Linear
from ..quant import Format
from . import qwen3
from .qwen3 import DenseMlp, Layer, Mixer, Model, Recurrence, SoftAttn, TPInfo


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class Niletar(Model):
    kernel_sources = ("host", "fused_ops", "gemm_tc", "gemm_sk", "gemm_wide", "moe_gemm", "gemm_simple", "streams", "attn_maps",
                      "attn_maps_tc", "gdn", "recurrent", "sampling")
    cuda_dtypes = (torch.bfloat16, torch.float32)
    fp8_pages = False

    @classmethod
    def _supports(cls, cfg: ModelConfig) -> None:
        if not cfg.layer_specs:
            raise ValueError("a Niletar configuration lists its layers")
        for i, s in enumerate(cfg.layer_specs):
            if s.rec is not None and (s.rec.conv > 8 or s.rec.state > 512):
                raise ValueError(f"layer {i}: convolutions of up to 8 taps and states of up to 512 rows are supported")
            if s.attn is not None and s.attn.vdim > 1024:
                raise ValueError(f"layer {i}: values of up to 1024 columns are supported")

    def __init__(self, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None,
                 first_layer: int = 0, last_layer: Optional[int] = None):
        super().__init__(cfg, device, dtype, tp, ops, first_layer, last_layer)
        if self.tp.world > 1 or not (self.is_first_stage and self.is_last_stage):
            raise ValueError("Niletar models run on one rank (no tensor or pipeline parallelism)")
        if dtype not in self.cuda_dtypes:
            raise ValueError(f"Niletar models run in bfloat16 or float32, not {dtype}")

    # ================================================================== construction
    @classmethod
    def random_init(cls, cfg: ModelConfig, fmt: Format = Format.DENSE, seed: int = 0, device="cpu", dtype=torch.bfloat16,
                    tp: Optional[TPInfo] = None, std: float = 0.02, ops=None, first_layer: int = 0,
                    last_layer: Optional[int] = None, **_) -> "Niletar":
        """Random weights under the checkpoint's tensor names (``std`` of the matrices; decays between a few and many tokens)."""
        if fmt != Format.DENSE:
            raise ValueError("Niletar weights are bf16 or fp32 (weight format 'dense')")
        m = cls(cfg, device, dtype, tp, ops, first_layer, last_layer)
        gen = torch.Generator(device=device).manual_seed(seed)
        rank = lambda i: max(cfg.layer_specs[i].rec.vdim, 16)              # noqa: E731  width of the low-rank inputs

        def get(name: str, shape: Sequence[int]) -> torch.Tensor:
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("a1", "g1", "a2", "g2"):
                r = rank(int(name[1:name.index(".")]))
                shape = [r if n < 0 else n for n in shape]
            t = torch.randn(*shape, generator=gen, device=device)
            if leaf in ("norm1", "norm2") or name == "final.norm":
                return t * 0.1
            if leaf == "conv":
                return t * 0.3
            if leaf in ("norm", "D"):
                return t * 0.1 + 1.0
            if leaf == "A_log":
                return t.abs()
            if leaf == "dt_bias":
                return t - 4.0
            return t * std
        return m._assemble(get)

    @classmethod
    def load(cls, model_dir: str, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None, first_layer: int = 0,
             last_layer: Optional[int] = None, cfg: Optional[ModelConfig] = None) -> "Niletar":
        from ..weights import Checkpoint
        ck = Checkpoint.open(model_dir)
        m = cls(cfg or ModelConfig.load(model_dir), device, dtype, tp, ops, first_layer, last_layer)
        return m._assemble(lambda name, shape: ck.get(name))

    def _assemble(self, get) -> "Niletar":
        """The layers from tensors by name; ``get`` is told the shape the configuration asks for (-1: the tensor's own)."""
        cfg, dev, dt, W = self.cfg, self.device, self.dtype, self.cfg.hidden_size

        def tensor(name: str, *shape: int) -> torch.Tensor:
            t = get(name, shape)
            if t.dim() != len(shape) or any(n not in (-1, s) for n, s in zip(shape, t.shape)):
                raise ValueError(f"tensor {name} is {tuple(t.shape)}, the configuration asks for {shape}")
            return t.to(dev)

        def f32(name: str, *shape: int) -> torch.Tensor:
            return tensor(name, *shape).float().contiguous()

        def dense(w: torch.Tensor, name: str, bias: Optional[torch.Tensor] = None) -> Linear:
            lin = Linear.from_dense(w.to(dt), dtype=dt)
            lin.name, lin.bias = name, None if bias is None else bias.to(dt)
            return lin

        def norm(name: str) -> torch.Tensor:
            return 1.0 + f32(name, W)                    # stored around zero

        self.embed = tensor("embed", cfg.vocab_size, W).to(dt).contiguous()
        for i, spec in enumerate(cfg.layer_specs):
            if spec.weights_of is not None:
                self.layers.append(None)
                continue
            L, p = Layer(), f"l{i}."
            L.kind = cfg.layer_type(i)
            L.mixer, L.mixer_norm = self._assemble_mixer(spec, p + "mix.", tensor, f32, dense), norm(p + "norm1")
            if spec.mlp is not None:
                L.mlp_norm, L.mlp = norm(p + "norm2"), DenseMlp()
                gu = [tensor(p + "mlp." + n, spec.mlp.ff, W) for n in ("gate", "up")]
                L.mlp.gate_up = dense(torch.cat(gu), p + "mlp.gate+up")
                L.mlp.down = dense(tensor(p + "mlp.down", W, spec.mlp.ff), p + "mlp.down")
            self.layers.append(L)
        for i, spec in enumerate(cfg.layer_specs):
            if spec.weights_of is not None:
                self.layers[i] = self.layers[spec.weights_of]
        self.final_norm = norm("final.norm")
        self.lm_head = dense(tensor("head", cfg.vocab_size, W), "head")
        return self

    def _assemble_mixer(self, spec, p: str, tensor, f32, dense) -> Mixer:
        M, W = Mixer(), self.cfg.hidden_size
        parts: List[Tuple[torch.Tensor, Optional[torch.Tensor]]] = []       # rows of the input projection with their biases
        at = 0

        def rows(col: str, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> None:
            """Append the rows of a part, which starts at a multiple of 8 columns (16 bytes of bf16)."""
            nonlocal at
            M.cols[col] = at
            pad = _up(w.shape[0], 8) - w.shape[0]
            parts.append((torch.cat([w, w.new_zeros(pad, W)]), None if bias is None else torch.cat([bias, bias.new_zeros(pad)])))
            at += w.shape[0] + pad

        outs = []
        a, r = spec.attn, spec.rec
        if a is not None:
            l = p + "left."
            for n, k in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                rows(n, tensor(l + n, k, W), tensor(l + n + ".b", k))
            rows("gate", tensor(l + "g", a.heads * a.vdim, W))
            M.attn = SoftAttn(a, self.device, sink=tensor(l + "sink", a.heads))
            outs.append(tensor(l + "o", W, a.heads * a.vdim))
            p = p + "right."
        if spec.kind.endswith("delta_rule"):
            R, nk, nv = Recurrence(r, "delta", r.heads), r.kv_heads * r.dim, r.heads * r.vdim
            names, sizes = ("q", "k", "v"), (nk, nk, nv)
            rows("conv", torch.cat([tensor(p + n, k, W) for n, k in zip(names, sizes)]))
            R.conv_w = torch.cat([tensor(p + n + ".conv", k, r.conv) for n, k in zip(names, sizes)]).to(self.dtype).contiguous()
            rows("beta", tensor(p + "b", r.heads, W))
            # the two low-rank maps share a product: [decay inputs | norm gates] from [a1 | g1], a block diagonal weight
            a1, a2, g1, g2 = tensor(p + "a1", -1, W), tensor(p + "a2", r.heads * r.dim, -1), tensor(p + "g1", -1, W), tensor(p + "g2", nv, -1)
            if a1.shape[0] != a2.shape[1] or g1.shape[0] != g2.shape[1]:
                raise ValueError(f"{p}: low-rank inputs of {a1.shape[0]} / {g1.shape[0]} rows for {a2.shape[1]} / {g2.shape[1]} columns")
            ra, rg = _up(a1.shape[0], 16), _up(g1.shape[0], 16)
            rows("low", torch.cat([a1, a1.new_zeros(ra - a1.shape[0], W), g1, g1.new_zeros(rg - g1.shape[0], W)]))
            M.low_width = ra + rg
            low = a2.new_zeros(a2.shape[0] + nv, ra + rg)
            low[:a2.shape[0], :a2.shape[1]] = a2
            low[a2.shape[0]:, ra:ra + g2.shape[1]] = g2
            R.low = dense(low, p + "a2+g2")
            R.dt_bias, R.norm_w = f32(p + "dt_bias", r.heads * r.dim), f32(p + "norm", r.vdim)
            outs.append(tensor(p + "o", W, nv))
        else:
            R = Recurrence(r, "ssm", r.norm_groups)
            z, conv, dt = torch.split(tensor(p + "in", r.inner + r.conv_dim + r.heads, W), [r.inner, r.conv_dim, r.heads])
            rows("z", z)
            rows("conv", conv)
            rows("dt", dt)
            R.conv_w = tensor(p + "conv", r.conv_dim, r.conv).to(self.dtype).contiguous()
            R.conv_b = f32(p + "conv.b", r.conv_dim)
            R.dt_bias, R.D, R.norm_w = f32(p + "dt_bias", r.heads), f32(p + "D", r.heads), f32(p + "norm", r.inner)
            outs.append(tensor(p + "o", W, r.inner))
        R.A = torch.exp(f32(p + "A_log", r.heads)).contiguous()
        M.rec = R
        bias = None
        if any(b is not None for _, b in parts):
            bias = torch.cat([w.new_zeros(w.shape[0]) if b is None else b for w, b in parts])
        M.in_proj = dense(torch.cat([w for w, _ in parts]), p + "in", bias)
        M.o = dense(torch.cat(outs, 1), p + "o")
        return M

    # ================================================================== forward
    def forward(self, batch: StepBatch, kv: KVCache, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The residual after the last layer, fp32 ``[T, hidden]`` (before the final norm)."""
        if hidden_in is not None or batch.embed_over:
            raise ValueError("Niletar models take token ids only")
        ops, eps, alpha = self.ops, self.cfg.rms_norm_eps, self.cfg.residual_alpha
        x = h = ops.embed(self.embed, batch.tokens)
        dump = qwen3._DUMP_DIR and not (self.device.type == "cuda" and torch.cuda.is_current_stream_capturing())
        for gi, L in enumerate(self.layers):
            x, h = ops.residual_norm(x, alpha, self._mixer(L.mixer, h, batch, kv, gi), L.mixer_norm, eps)
            if L.mlp is not None:
                x, h = ops.residual_norm(x, alpha, self._mlp(L.mlp, h, None, gi)[0], L.mlp_norm, eps)
            if dump:
                qwen3._dump(f"layer{gi:03d}_residual", x)
        if dump:
            qwen3._dump_step[0] += 1
        return x.float()

    def final_hidden(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return self.ops.norm_rows(x, rows, self.final_norm, self.cfg.rms_norm_eps, self.dtype)
