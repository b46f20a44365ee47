"""Medodra: a decoder whose layers add a mixer and a feed-forward, both of the same residual, described layer by layer in its
configuration (``ModelConfig.layer_specs``).

Mixers are a gated delta rule with one decay per head, or a sigmoid attention (weights are not shares; distances enter as learned
terms of the scores) beside an elementwise gated recurrence (minGRU).  Feed-forwards route tokens to experts by sigmoid scores that weigh
the experts' inputs, beside a gated shared expert.  A run of layers may be passed several times with the same tensors, each pass with a
cache and states of its own and a linear map of the residual beside the embedding ahead of it.  The residual, the norms, the router and the
recurrent states are fp32.  Tensor names: ``embed``, ``loop.in``, ``l<i>.{norm1,norm2}``; of a delta mixer
``l<i>.mix.{q,k,v}[.conv]``, ``.{b,a,A_log,dt_bias,norm,g,o}``; of a parallel one ``l<i>.mix.left.{q,k,v}[.b|.conv]``, ``.left.{rel,pb,o,o.b,out}``,
``l<i>.mix.right.{z,z.b,x,x.b,g,o,out}``; ``l<i>.mlp.{router,e<j>.{gate,up,down},shared.{gate,up,down,sg}}``, ``final.norm``, ``head``.
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
from .qwen3 import Branches, DenseMlp, Experts, Layer, Mixer, Model, MoeMlp, Recurrence, SigmoidAttn, TPInfo


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class Medodra(Model):
    kernel_sources = ("host", "fused_ops", "gemm_tc", "gemm_sk", "gemm_wide", "moe_gemm", "gemm_simple", "streams", "attn_maps",
                      "attn_maps_tc", "gdn", "recurrent", "moe", "sampling")
    cuda_dtypes = (torch.bfloat16, torch.float32)
    fp8_pages = False

    @classmethod
    def _supports(cls, cfg: ModelConfig) -> None:
        if not cfg.layer_specs:
            raise ValueError("a Medodra configuration lists its layers")
        for i, s in enumerate(cfg.layer_specs):
            if s.rec is not None and (s.rec.conv > 8 or s.rec.state > 512):
                raise ValueError(f"layer {i}: convolutions of up to 8 taps and states of up to 512 rows are supported")
            if s.attn is not None and (s.attn.conv > 8 or s.attn.vdim > 1024):
                raise ValueError(f"layer {i}: convolutions of up to 8 taps and values of up to 1024 columns are supported")
            if s.mlp is not None and (s.mlp.experts > 512 or s.mlp.top > 32):
                raise ValueError(f"layer {i}: up to 512 experts and 32 per token are supported")

    def __init__(self, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None,
                 first_layer: int = 0, last_layer: Optional[int] = None):
        super().__init__(cfg, device, dtype, tp, ops, first_layer, last_layer)
        if self.tp.world > 1 or not (self.is_first_stage and self.is_last_stage):
            raise ValueError("Medodra models run on one rank (no tensor or pipeline parallelism)")
        if dtype not in self.cuda_dtypes:
            raise ValueError(f"Medodra models run in bfloat16 or float32, not {dtype}")
        W = cfg.hidden_size
        self.pos_freq = qwen3._two_floats([10000.0 ** (-2.0 * i / W) for i in range((W + 1) // 2)], self.device)
        self.loop_in: Optional[Linear] = None

    # ================================================================== construction
    @classmethod
    def random_init(cls, cfg: ModelConfig, fmt: Format = Format.DENSE, seed: int = 0, device="cpu", dtype=torch.bfloat16,
                    tp: Optional[TPInfo] = None, std: float = 0.02, ops=None, first_layer: int = 0,
                    last_layer: Optional[int] = None, **_) -> "Medodra":
        """Random weights under the checkpoint's tensor names (``std`` of the matrices; decays between a few and many tokens)."""
        if fmt != Format.DENSE:
            raise ValueError("Medodra weights are bf16 or fp32 (weight format 'dense')")
        m = cls(cfg, device, dtype, tp, ops, first_layer, last_layer)
        gen = torch.Generator(device=device).manual_seed(seed)

        def get(name: str, shape: Sequence[int]) -> torch.Tensor:
            leaf = name.rsplit(".", 1)[-1]
            t = torch.randn(*(32 if n < 0 else n for n in shape), generator=gen, device=device)
            if leaf in ("norm1", "norm2") or name == "final.norm":
                return t * 0.1
            if leaf in ("norm", "out"):
                return t * 0.1 + 1.0
            if leaf == "conv":
                return t * 0.3
            if leaf == "A_log":
                return t.abs()
            if leaf in ("dt_bias", "pb"):
                return t - 4.0
            if leaf == "rel":
                return t * 0.5
            return t * (std if name != "embed" else 1.0)
        return m._assemble(get)

    @classmethod
    def load(cls, model_dir: str, device="cpu", dtype=torch.bfloat16, tp: Optional[TPInfo] = None, ops=None, first_layer: int = 0,
             last_layer: Optional[int] = None, cfg: Optional[ModelConfig] = None) -> "Medodra":
        from ..weights import Checkpoint
        ck = Checkpoint.open(model_dir)
        m = cls(cfg or ModelConfig.load(model_dir), device, dtype, tp, ops, first_layer, last_layer)
        return m._assemble(lambda name, shape: ck.get(name))

    def _assemble(self, get) -> "Medodra":
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
        if any(s.joins for s in cfg.layer_specs):
            self.loop_in = dense(tensor("loop.in", W, 2 * W), "loop.in")
        for i, spec in enumerate(cfg.layer_specs):
            if spec.weights_of is not None:
                self.layers.append(self.layers[spec.weights_of])
                continue
            L, p = Layer(), f"l{i if spec.number is None else spec.number}."
            L.kind = cfg.layer_type(i)
            L.mixer, L.mixer_norm = self._assemble_mixer(spec, p + "mix.", tensor, f32, dense), norm(p + "norm1")
            if spec.mlp is not None:
                L.mlp_norm, L.mlp = norm(p + "norm2"), self._assemble_mlp(spec.mlp, p + "mlp.", tensor, dense)
            self.layers.append(L)
        self.final_norm = norm("final.norm")
        self.lm_head = dense(tensor("head", cfg.vocab_size, W), "head")
        return self

    def _assemble_mlp(self, spec, p: str, tensor, dense) -> MoeMlp:
        W = self.cfg.hidden_size

        def glu(p: str, ff: int) -> Tuple[Linear, Linear]:
            gate_up = torch.cat([tensor(p + n, ff, W) for n in ("gate", "up")])
            return dense(gate_up, p + "gate+up"), dense(tensor(p + "down", W, ff), p + "down")
        M, E = MoeMlp(), Experts()
        M.top_k, M.renorm, M.sigmoid, M.rows_out, M.experts = spec.top, spec.renorm, spec.scores == "sigmoid", True, E
        E.act, E.weigh_input, E.fused_act, E.num_experts, E.count = spec.act, spec.weigh_input, True, spec.experts, spec.experts
        for e in range(spec.experts):
            gate_up, down = glu(f"{p}e{e}.", spec.ff)
            E.gate_up.append(gate_up)
            E.down.append(down)
        # the router's rows and the shared expert's gate are one product, rounded up to 8 rows
        router = [tensor(p + "router", spec.experts, W)]
        if spec.shared_ff:
            M.shared = DenseMlp()
            M.shared.gate_up, M.shared.down = glu(p + "shared.", spec.shared_ff)
            if spec.shared_gate:
                M.gate_row = spec.experts
                router.append(tensor(p + "shared.sg", 1, W))
        rows = sum(r.shape[0] for r in router)
        if M.gate_row is not None:
            router.append(router[0].new_zeros(_up(rows, 8) - rows, W))
        M.router = dense(torch.cat(router), p + "router")
        return M

    def _assemble_mixer(self, spec, p: str, tensor, f32, dense) -> Mixer:
        M, W, a, r = Mixer(), self.cfg.hidden_size, spec.attn, spec.rec
        parts: List[Tuple[torch.Tensor, Optional[torch.Tensor]]] = []       # rows of the input projection with their biases
        at = 0

        def rows(col: str, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> None:
            """Append the rows of a part, which starts at a multiple of 8 columns (16 bytes of bf16)."""
            nonlocal at
            M.cols[col] = at
            pad = _up(w.shape[0], 8) - w.shape[0]
            parts.append((torch.cat([w, w.new_zeros(pad, W)]), w.new_zeros(w.shape[0] + pad) if bias is None else
                          torch.cat([bias, bias.new_zeros(pad)])))
            at += w.shape[0] + pad

        if a is None:
            R, nk, nv = Recurrence(r, "delta", r.heads), r.kv_heads * r.dim, r.heads * r.vdim
            names, sizes = ("q", "k", "v"), (nk, nk, nv)
            rows("conv", torch.cat([tensor(p + n, k, W) for n, k in zip(names, sizes)]))
            R.conv_w = torch.cat([tensor(p + n + ".conv", k, r.conv) for n, k in zip(names, sizes)]).to(self.dtype).contiguous()
            rows("z", tensor(p + "g", nv, W))
            rows("beta", tensor(p + "b", r.heads, W))
            rows("decay", tensor(p + "a", r.heads, W))
            R.A, R.dt_bias, R.norm_w = torch.exp(f32(p + "A_log", r.heads)).contiguous(), f32(p + "dt_bias", r.heads), f32(p + "norm", r.vdim)
            M.rec, M.o = R, dense(tensor(p + "o", W, nv), p + "o")
            M.in_proj = dense(torch.cat([w for w, _ in parts]), p + "in")
            return M
        l, g = p + "left.", p + "right."
        sizes = (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim))
        for n, k in sizes:
            rows(n, tensor(l + n, k, W), tensor(l + n + ".b", k))
        conv = torch.cat([tensor(f"{l}{n}.conv", k, a.conv) for n, k in sizes]) if a.conv else None
        M.attn = SigmoidAttn(a, self.device, tensor(l + "rel", -1, a.heads), tensor(l + "pb", a.heads), conv)
        rows("zg", tensor(g + "z", r.width, W), tensor(g + "z.b", r.width))
        rows("u", tensor(g + "x", r.width, W), tensor(g + "x.b", r.width))
        rows("g", tensor(g + "g", r.width, W))
        M.rec = Recurrence(r, "mingru", 1)
        M.o = dense(tensor(l + "o", W, a.heads * a.vdim), l + "o", tensor(l + "o.b", W))
        M.o_rec = dense(tensor(g + "o", W, r.width), g + "o")
        M.out_norms = (f32(l + "out", W), f32(g + "out", W))
        M.in_proj = dense(torch.cat([w for w, _ in parts]), p + "in", torch.cat([b for _, b in parts]))
        return M

    # ================================================================== forward
    def forward(self, batch: StepBatch, kv: KVCache, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The residual after the last layer, fp32 ``[T, hidden]`` (before the final norm)."""
        if hidden_in is not None or batch.embed_over:
            raise ValueError("Medodra models take token ids only")
        ops, cfg, dt, W = self.ops, self.cfg, self.dtype, self.cfg.hidden_size
        eps = cfg.rms_norm_eps
        # rows of the map ahead of a pass: [residual | embedding]
        join = torch.empty(batch.tokens.numel(), 2 * W, dtype=dt, device=self.device) if self.loop_in is not None else None
        x = ops.embed_positions(self.embed, batch.tokens, batch.positions, cfg.embed_scale, self.pos_freq, None if join is None else join[:, W:])
        dump = qwen3._DUMP_DIR and not (self.device.type == "cuda" and torch.cuda.is_current_stream_capturing())
        br: Optional[Branches] = None                    # what the layer before leaves to be added
        for gi, (L, spec) in enumerate(zip(self.layers, cfg.layer_specs)):
            if spec.joins:
                x, _, _ = ops.branch_step(x, br, eps, dt, copy=join[:, :W])
                if dump and br is not None:
                    qwen3._dump(f"layer{gi - 1:03d}_residual", x)
                x, br = ops.linear(self.loop_in, join, out_dtype=torch.float32), None
            x, h1, h2 = ops.branch_step(x, br, eps, dt, L.mixer_norm, L.mlp_norm)
            if dump and br is not None:
                qwen3._dump(f"layer{gi - 1:03d}_residual", x)
            y = self._mixer(L.mixer, h1, batch, kv, gi)
            br = Branches(y, L.mixer.out_norms, self._mlp(L.mlp, h2, None, gi)[0] if L.mlp is not None else None, cfg.residual_mult)
        x, _, _ = ops.branch_step(x, br, eps, dt)
        if dump:
            qwen3._dump(f"layer{len(self.layers) - 1:03d}_residual", x)
            qwen3._dump_step[0] += 1
        return x

    def final_hidden(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return self.ops.norm_rows(x, rows, self.final_norm, self.cfg.rms_norm_eps, self.dtype)

    def weight_bytes(self) -> int:
        return super().weight_bytes() + (self.loop_in.nbytes() if self.loop_in is not None else 0)
