"""Rapisun: a decoder that adds the layer-normed output of every sublayer to its residual, described layer by layer in its
configuration (``ModelConfig.layer_specs``).

Mixers are a linear attention with forget gates whose complements weigh the incoming values (HGRN2) and a windowed latent attention
with a sink, whose latents a later layer may read; a causal convolution over time is added to what a mixer reads.  Feed-forwards have no gate: a
dense one activated by a sum of normed powers, or routed experts with squared ReLUs and a shared one.  The residual, the norms, the
inputs of the convolutions and the recurrent states are fp32.  Tensor names: ``embed[.norm]``, ``l<i>.{norm1,norm2,canon1}``,
``l<i>.mix.{q,f,f.b,lower,v,norm,o}`` or ``l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,o}``, ``l<i>.mlp.{up,down,act}`` or
``l<i>.mlp.{router,e<j>.up,e<j>.down,shared.up,shared.down}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ..batch import StepBatch
from ..config import GatedLinearSpec, ModelConfig, MoeSpec
from ..kv import KVCache
from ..linear import Linear
from ..quant import Format
from . import qwen3
from .qwen3 import Experts, LatentAttn, Layer, Mixer, Model, MoeMlp, PlainMlp, Recurrence, TPInfo


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class Rapisun(Model):
    kernel_sources = ("host", "fused_ops", "gemm_tc", "gemm_sk", "gemm_wide", "moe_gemm", "gemm_simple", "streams", "attn_maps",
                      "attn_maps_tc", "latent", "recurrent", "moe", "sampling")
    cuda_dtypes = (torch.bfloat16, torch.float32)
    fp8_pages = False

    @classmethod
    def _supports(cls, cfg: ModelConfig) -> None:
        if not cfg.layer_specs:
            raise ValueError("a Rapisun configuration lists its layers")
        for i, s in enumerate(cfg.layer_specs):
            if s.rec is not None and s.rec.state > 512:
                raise ValueError(f"layer {i}: states of up to 512 rows are supported")
            if s.attn is not None and s.attn.kv_rank > 1024:
                raise ValueError(f"layer {i}: latents of up to 1024 columns are supported")
            if isinstance(s.mlp, MoeSpec) and (s.mlp.experts > 512 or s.mlp.top > 32):
                raise ValueError(f"layer {i}: up to 512 experts and 32 per token are supported")

    def __init__(self, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None,
                 first_layer: int = 0, last_layer: Optional[int] = None):
        super().__init__(cfg, device, dtype, tp, ops, first_layer, last_layer)
        if self.tp.world > 1 or not (self.is_first_stage and self.is_last_stage):
            raise ValueError("Rapisun models run on one rank (no tensor or pipeline parallelism)")
        if dtype not in self.cuda_dtypes:
            raise ValueError(f"Rapisun models run in bfloat16 or float32, not {dtype}")
        self.embed_norm_w: torch.Tensor = None

    # ================================================================== construction
    @classmethod
    def random_init(cls, cfg: ModelConfig, fmt: Format = Format.DENSE, seed: int = 0, device="cpu", dtype=torch.bfloat16,
                    tp: Optional[TPInfo] = None, std: float = 0.02, ops=None, first_layer: int = 0,
                    last_layer: Optional[int] = None, **_) -> "Rapisun":
        """Random weights under the checkpoint's tensor names (``std`` of the matrices; forget gates over a few to many tokens)."""
        if fmt != Format.DENSE:
            raise ValueError("Rapisun weights are bf16 or fp32 (weight format 'dense')")
        m = cls(cfg, device, dtype, tp, ops, first_layer, last_layer)
        gen = torch.Generator(device=device).manual_seed(seed)

        def get(name: str, shape: Sequence[int]) -> torch.Tensor:
            leaf = name.rsplit(".", 1)[-1]
            t = torch.randn(*shape, generator=gen, device=device)
            if leaf in ("norm", "norm1", "norm2"):
                return t * 0.1 + 1.0
            if leaf == "canon1":
                return t * 0.2
            if leaf == "lower":
                return torch.sigmoid(t)
            if leaf == "b":
                return t + 2.0
            if leaf in ("sink", "act"):
                return t * 0.5
            return t * (std if name != "embed" else 1.0)
        return m._assemble(get)

    @classmethod
    def load(cls, model_dir: str, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None, first_layer: int = 0,
             last_layer: Optional[int] = None, cfg: Optional[ModelConfig] = None) -> "Rapisun":
        from ..weights import Checkpoint
        ck = Checkpoint.open(model_dir)
        m = cls(cfg or ModelConfig.load(model_dir), device, dtype, tp, ops, first_layer, last_layer)
        return m._assemble(lambda name, shape: ck.get(name))

    def _assemble(self, get) -> "Rapisun":
        """The layers from tensors by name; ``get`` is told the shape the configuration asks for."""
        cfg, dt, W = self.cfg, self.dtype, self.cfg.hidden_size

        def tensor(name: str, *shape: int) -> torch.Tensor:
            t = get(name, shape)
            if tuple(t.shape) != shape:
                raise ValueError(f"tensor {name} is {tuple(t.shape)}, the configuration asks for {shape}")
            return t.to(self.device)

        def f32(name: str, *shape: int) -> torch.Tensor:
            return tensor(name, *shape).float().contiguous()

        def dense(w: torch.Tensor, name: str) -> Linear:
            lin = Linear.from_dense(w.to(dt), dtype=dt)
            lin.name = name
            return lin

        def linear(name: str, rows: int, cols: int) -> Linear:
            return dense(tensor(name, rows, cols), name)

        self.embed = tensor("embed", cfg.vocab_size, W).to(dt).contiguous()
        self.embed_norm_w = f32("embed.norm", W)
        for i, spec in enumerate(cfg.layer_specs):
            L, p = Layer(), f"l{i}."
            L.kind = cfg.layer_type(i)
            if cfg.input_conv:
                L.in_conv = f32(p + "canon1", W, cfg.input_conv).t().contiguous()
            L.mixer, L.mixer_norm = self._assemble_mixer(spec, p + "mix.", tensor, f32, dense, linear), f32(p + "norm1", W)
            if spec.mlp is not None:
                L.mlp_norm, L.mlp = f32(p + "norm2", W), self._assemble_mlp(spec.mlp, p + "mlp.", f32, linear)
            self.layers.append(L)
        self.final_norm = f32("final.norm", W)
        self.lm_head = linear("head", cfg.vocab_size, W)
        return self

    def _assemble_mlp(self, spec, p: str, f32, linear):
        W = self.cfg.hidden_size

        def plain(p: str, ff: int, poly=None) -> PlainMlp:
            M = PlainMlp(poly)
            M.up, M.down = linear(p + "up", ff, W), linear(p + "down", W, ff)
            return M
        if not isinstance(spec, MoeSpec):
            return plain(p, spec.ff, f32(p + "act", 4))
        M, E = MoeMlp(), Experts()
        M.top_k, M.renorm, M.rows_out, M.experts = spec.top, True, True, E
        M.router = linear(p + "router", spec.experts, W)
        E.act, E.num_experts, E.count = "relu2", spec.experts, spec.experts
        for e in range(spec.experts):
            E.gate_up.append(linear(f"{p}e{e}.up", spec.ff, W))
            E.down.append(linear(f"{p}e{e}.down", W, spec.ff))
        if spec.shared_ff:
            M.shared = plain(p + "shared.", spec.shared_ff)
        return M

    def _assemble_mixer(self, spec, p: str, tensor, f32, dense, linear) -> Mixer:
        M, W, a, r = Mixer(), self.cfg.hidden_size, spec.attn, spec.rec
        parts: List[torch.Tensor] = []                   # rows of the input projection
        at = 0

        def rows(col: str, w: torch.Tensor) -> None:
            """Append the rows of a part, which starts at a multiple of 8 columns (16 bytes of bf16)."""
            nonlocal at
            M.cols[col] = at
            pad = _up(w.shape[0], 8) - w.shape[0]
            parts.append(torch.cat([w, w.new_zeros(pad, W)]))
            at += w.shape[0] + pad

        if isinstance(r, GatedLinearSpec):
            nk, nv = r.heads * r.dim, r.heads * r.vdim
            for n, k in (("q", nk), ("f", nk), ("v", nv)):
                rows(n, tensor(p + n, k, W))
            R = M.rec = Recurrence(r, "gated", r.heads)
            R.A, R.dt_bias, R.norm_w = f32(p + "lower", nk), f32(p + "f.b", nk), f32(p + "norm", r.vdim)
            n_out = nv
        else:
            A = M.attn = LatentAttn(a, self.device)
            rows("q", tensor(p + "dq", a.q_rank, W))
            if a.kv_from is None:
                rows("kv", tensor(p + "dkv", a.kv_rank + a.rot_dim, W))
                A.c_norm = f32(p + "dkv.norm", a.kv_rank)
            A.q_norm, A.uq = f32(p + "dq.norm", a.q_rank), linear(p + "uq", a.heads * (a.dim + a.rot_dim), a.q_rank)
            A.set_maps(tensor(p + "uk", a.heads * a.dim, a.kv_rank), tensor(p + "uv", a.heads * a.vdim, a.kv_rank), self.dtype)
            A.sink = f32(p + "sink", a.heads) if a.sink else None
            n_out = a.heads * a.vdim
        M.in_proj, M.o = dense(torch.cat(parts), p + "in"), linear(p + "o", W, n_out)
        return M

    # ================================================================== forward
    def forward(self, batch: StepBatch, kv: KVCache, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The residual after the last layer, fp32 ``[T, hidden]`` (before the final norm)."""
        if hidden_in is not None or batch.embed_over:
            raise ValueError("Rapisun models take token ids only")
        ops, eps, dt = self.ops, self.cfg.rms_norm_eps, self.dtype
        x = ops.embed_norm(self.embed, batch.tokens, self.embed_norm_w, eps)
        dump = qwen3._DUMP_DIR and not (self.device.type == "cuda" and torch.cuda.is_current_stream_capturing())
        for gi, L in enumerate(self.layers):
            if L.in_conv is not None:
                if batch.gdn_defer is not None and self.cfg.input_conv > 1:
                    self.conv_records[gi] = x.clone()
                h = ops.input_conv(x, L.in_conv, batch, kv, gi, dt)
            else:
                h = x.to(dt)
            x, h = ops.branch_norm(x, self._mixer(L.mixer, h, batch, kv, gi), L.mixer_norm, eps, copy=L.mlp is not None)
            if L.mlp is not None:
                x, _ = ops.branch_norm(x, self._mlp(L.mlp, h, None, gi)[0], L.mlp_norm, eps, copy=False)
            if dump:
                qwen3._dump(f"layer{gi:03d}_residual", x)
        if dump:
            qwen3._dump_step[0] += 1
        return x

    def final_hidden(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return self.ops.norm_rows(x, rows, self.final_norm, self.cfg.rms_norm_eps, self.dtype, centre=True)
