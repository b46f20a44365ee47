"""Model configuration: the keys of a Hugging Face ``config.json`` that the runtime reads.

Covers the same surface as the reference's ``crates/blaze/src/config.rs:117-273``
(``text_config`` nesting, ``layer_types`` / ``full_attention_interval``, Gated DeltaNet dims,
MoE dims, RoPE with YaRN / partial rotary / M-RoPE sections, MTP layer count, eos ids), and
adds the plain Qwen3 / Qwen3-MoE architectures (ungated attention, no shared expert, norms
that are not zero-centred) which the reference refuses to load.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import asdict, dataclass, field, replace
from typing import Any, Dict, List, Optional, Union


@dataclass
class RopeConfig:
    theta: float = 1.0e4
    partial_rotary_factor: float = 1.0
    mrope_section: Optional[List[int]] = None
    # YaRN
    yarn_factor: float = 1.0
    yarn_original_max_position: int = 0
    yarn_beta_fast: float = 32.0
    yarn_beta_slow: float = 1.0
    yarn_attention_factor: Optional[float] = None

    def rope_scale(self) -> float:
        """Multiplier of sin/cos under YaRN (1 when YaRN is off)."""
        if self.yarn_factor <= 1.0:
            return 1.0
        if self.yarn_attention_factor is not None:
            return float(self.yarn_attention_factor)
        return 0.1 * math.log(self.yarn_factor) + 1.0


@dataclass
class DiffAttnSpec:
    """Differential attention of one layer: two attention maps per head over the same values, the second subtracted from the
    first with a learned weight."""
    heads: int
    kv_heads: int
    dim: int                    # per map and head, queries and keys
    vdim: int                   # per head, values
    scale: float                # of the scores
    diff: float                 # constant part of the second map's weight; the normed output is scaled by 1 - diff
    window: int = 0             # a row sees itself and the window - 1 tokens before it (0: every token before it)

    maps = 2                    # query / key maps per head

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads


@dataclass
class RotarySpec:
    """Rotary positions on the first ``dims`` dimensions of a head.  ``factor`` > 1 slows frequencies down by their wavelength:
    those longer than ``original / low`` tokens by the whole factor, those shorter than ``original / high`` not at all, the ones
    between by a blend."""
    dims: int
    base: float
    interleaved: bool = True    # pairs (2i, 2i + 1); else (i, i + dims / 2)
    factor: float = 1.0
    low: float = 1.0
    high: float = 4.0
    original: float = 0.0       # 0: no scaling

    def frequencies(self) -> List[float]:
        out = []
        for i in range(self.dims // 2):
            f = self.base ** (-2.0 * i / self.dims)
            if self.original:
                turns = self.original * f / (2 * math.pi)          # full turns over the original context
                if turns < self.low:
                    f /= self.factor
                elif turns <= self.high:
                    keep = (turns - self.low) / (self.high - self.low) if self.high > self.low else 1.0
                    f *= keep + (1 - keep) / self.factor
            out.append(f)
        return out


@dataclass
class SoftAttnSpec:
    """Softmax attention of one layer over bf16 / fp32 pages, with the options of its designs."""
    heads: int
    kv_heads: int
    dim: int                    # queries and keys
    vdim: int                   # values
    scale: float                # of the scores
    rot: Optional[RotarySpec] = None
    bias: bool = False          # q, k and v projections have biases
    unit_rms: bool = False      # q and k heads divided by their root mean square after the rotation
    sink: bool = False          # a learned term per head in the softmax's denominator
    gate: bool = False          # heads multiplied by sigmoid of a projection of the layer's input
    window: int = 0             # as in DiffAttnSpec
    out_scale: float = 1.0      # of the mixer's output
    maps = 1

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads


@dataclass
class SigmoidAttnSpec:
    """Attention of one layer whose weights are sigmoids of the scores, not shares of a sum, with the options of its designs; scores have
    a learned term per head and distance bucket (a table of the checkpoint) and one per head."""
    heads: int
    kv_heads: int
    dim: int                    # queries and keys
    vdim: int                   # values
    scale: float                # of the scores, before the learned terms
    far: float                  # distance from which all keys share the table's last row
    bias: bool = False          # q, k, v and output projections have biases
    conv: int = 0               # taps of a causal convolution of the projected q, k and v over time (0: none)
    unit_v: bool = False        # value heads divided by their root mean square
    temp_coef: float = 0.0      # queries at position p times 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
    temp_every: float = 1.0
    window = 0                  # as in DiffAttnSpec
    out_scale = 1.0
    maps = 1

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads

    @property
    def conv_dim(self) -> int:
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)

    def bucket(self, n: int, rows: int) -> int:
        """Row of a table of ``rows`` rows for a key ``n`` tokens back: the first half of the rows for one distance each, the others
        for ranges that grow logarithmically up to ``far``."""
        near = rows // 2
        if n < near:
            return n
        # distances where the logarithms' ratio is a whole number fall into the upper bucket, whatever the rounding
        return min(rows - 1, near + math.floor(math.log(n / near) / math.log(self.far / near) * (rows - near) + 1e-9))


@dataclass
class LatentAttnSpec:
    """Softmax attention whose keys and values are linear maps of one cached vector per token (a normed latent of ``kv_rank``
    numbers), beside a rotated key part that all heads share; queries come through a latent of their own."""
    heads: int
    dim: int                    # per head, queries and keys without rotation
    rot_dim: int                # rotated query / key columns
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float                # of the scores
    rot: Optional[RotarySpec] = None
    sink: bool = False          # as in SoftAttnSpec
    window: int = 0             # as in DiffAttnSpec
    kv_from: Optional[int] = None          # the layer whose latents and rotated key parts this one reads instead of its own
    maps = 1
    kv_heads = 1                # what is cached is one key / value head of kv_rank + rot_dim columns

    @property
    def group(self) -> int:
        return self.heads


@dataclass
class GatedLinearSpec:
    """Linear attention with a forget gate per head and query channel, whose complement weighs the incoming value (HGRN2); normed per
    head."""
    heads: int
    dim: int
    vdim: int
    conv = 0                    # no convolution of its own
    out_scale = 1.0

    @property
    def state(self) -> int:
        return self.dim


@dataclass
class DeltaSpec:
    """Gated delta rule with one decay per head and key channel (or one per head), and a gated norm per head."""
    heads: int
    kv_heads: int               # heads of q and k
    dim: int
    vdim: int
    conv: int                   # taps of the convolution before it
    out_scale: float = 1.0
    head_decay: bool = False    # one decay per head, its input and the gate's projected from the layer's input as they are; else one per
                                # key channel, both inputs through low-rank maps
    gate: str = "sigmoid"       # of the normed output: "sigmoid" | "silu"

    @property
    def conv_dim(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def state(self) -> int:
        return self.dim


@dataclass
class MinGruSpec:
    """Elementwise recurrence with a gated output (minGRU): its gate and its candidate depend on the token's input, not on the state."""
    width: int
    conv = 0                    # no convolution of its own
    heads = state = 1
    out_scale = 1.0

    @property
    def vdim(self) -> int:
        return self.width


@dataclass
class StateSpaceSpec:
    """Mamba-2 (state-space duality) mixer."""
    heads: int
    vdim: int
    state: int
    groups: int                 # B / C pairs, each for heads / groups heads
    norm_groups: int
    conv: int
    out_scale: float = 1.0

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_dim(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass
class GluSpec:
    """Dense gated feed-forward: with a clamped gate and a clamped up projection, or (no ``limit``) ``silu(gate) * up``."""
    ff: int
    limit: Optional[float] = None


@dataclass
class PolyNormSpec:
    """Dense feed-forward without a gate, activated by a sum of normed powers (``a N(z) + b N(z^2) + c N(z^3) + e``)."""
    ff: int


@dataclass
class MoeSpec:
    """Routed experts weighted by their scores, and a shared one.  An expert is ``down(relu(up h)^2)`` or
    ``down(silu(gate h) * up h)``."""
    experts: int
    top: int
    ff: int                     # per expert
    shared_ff: int = 0          # 0: no shared expert
    act: str = "relu2"          # or "swiglu"
    scores: str = "softmax"     # or "sigmoid"
    renorm: bool = True         # weights divided by their sum over the chosen experts
    weigh_input: bool = False   # the weight multiplies an expert's input, not its output
    shared_gate: bool = False   # the shared expert's output times sigmoid of a projection to one number


@dataclass
class LayerSpec:
    """One entry of a configuration that describes its layers one by one: an attention, a recurrence, or both side by side."""
    attn: Union[DiffAttnSpec, SoftAttnSpec, SigmoidAttnSpec, LatentAttnSpec, None] = None
    mlp: Union[GluSpec, PolyNormSpec, MoeSpec, None] = None        # None: the layer has no feed-forward
    weights_of: Optional[int] = None       # the layer whose tensors this one uses (with a cache and a state of its own)
    rec: Union[DeltaSpec, StateSpaceSpec, GatedLinearSpec, MinGruSpec, None] = None
    number: Optional[int] = None           # of the layer in the checkpoint, where that is not its place in the list (looped layers)
    joins: bool = False         # a pass of a loop starts here: the residual is first mapped from itself beside the embedding

    @property
    def kind(self) -> str:
        names = {DiffAttnSpec: "diff_attention", SoftAttnSpec: "soft_attention", SigmoidAttnSpec: "sigmoid_attention",
                 LatentAttnSpec: "latent_attention", DeltaSpec: "delta_rule", StateSpaceSpec: "state_space", GatedLinearSpec: "gated_linear",
                 MinGruSpec: "min_gru"}
        return "+".join(names[type(m)] for m in (self.attn, self.rec) if m is not None)


@dataclass
class ModelConfig:
    architecture: str = "Qwen3ForCausalLM"
    model_type: str = "qwen3"
    vocab_size: int = 1024
    hidden_size: int = 256
    num_layers: int = 2
    num_heads: int = 4
    num_kv_heads: int = 2
    head_dim: int = 64
    intermediate_size: int = 512
    rms_norm_eps: float = 1e-6
    tie_word_embeddings: bool = False
    max_position_embeddings: int = 32768
    rope: RopeConfig = field(default_factory=RopeConfig)
    # layer pattern: "full_attention" | "linear_attention"
    layer_types: List[str] = field(default_factory=list)
    # attention variants
    attn_output_gate: bool = False          # q_proj rows are [q | gate] per head
    qk_norm: bool = True                    # per-head RMSNorm on q and k
    zero_centered_norm: bool = False        # weights stored as (w - 1)
    attention_bias: bool = False
    # Gated DeltaNet
    linear_num_key_heads: int = 0
    linear_num_value_heads: int = 0
    linear_key_head_dim: int = 0
    linear_value_head_dim: int = 0
    linear_conv_kernel_dim: int = 4
    # MoE
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    shared_expert_intermediate_size: int = 0
    norm_topk_prob: bool = True
    # MTP
    mtp_num_hidden_layers: int = 0
    # Qwen4-Exp extras (``crates/blaze/src/config.rs:56-80``, :181-212): hyper-connections, per-layer n-gram embedding,
    # sparse-attention indexer
    hc_count: int = 0                       # residual streams (0 or 1: plain pre-norm residual)
    hc_lowrank: int = 16
    ple_layers: List[int] = field(default_factory=list)      # decoder layers that add an n-gram embedding (0-based)
    ngram_size: int = 3
    heads_per_ngram: int = 0
    ple_embed_dim: int = 0
    ple_conv_kernel: int = 4
    gdn_output_gate: str = "silu"           # activation of the Gated DeltaNet output gate: "silu" | "sigmoid"
    indexer_heads: int = 0                  # > 0: the checkpoint carries a sparse-attention indexer (not used: dense attention)
    indexer_head_dim: int = 0
    indexer_budget: int = 0
    indexer_compress_ratio: int = 0
    # models whose configuration lists its layers one by one, each with sizes of its own (Sevevik, Niletar, Rapisun, Medodra); the sizes above
    # then hold those of the first layer
    layer_specs: List[LayerSpec] = field(default_factory=list)
    streams: int = 1                        # residual streams joined by learned static mixes
    residual_mult: float = 1.0              # of every sublayer's output
    embed_scale: float = 1.0
    residual_alpha: float = 1.0             # post-norm residual: x <- norm(alpha * x + sublayer)
    input_conv: int = 0                     # taps of a causal convolution that is added to every mixer's input (0: none)
    # tokens
    eos_token_ids: List[int] = field(default_factory=list)
    bos_token_id: Optional[int] = None
    # quantisation block of config.json (raw), resolved by quant.QuantConfig
    quantization_config: Optional[Dict[str, Any]] = None
    torch_dtype: str = "bfloat16"
    # vision tower (raw dict), if any
    vision_config: Optional[Dict[str, Any]] = None

    # ------------------------------------------------------------------ derived
    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def has_gdn(self) -> bool:
        return any(t == "linear_attention" for t in self.layer_types)

    @property
    def has_hc(self) -> bool:
        return self.hc_count > 1

    @property
    def rotary_dim(self) -> int:
        rd = int(self.head_dim * self.rope.partial_rotary_factor)
        return rd - (rd % 2)

    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    def layer_type(self, i: int) -> str:
        if self.layer_specs:
            return self.layer_specs[i].kind
        return self.layer_types[i] if self.layer_types else "full_attention"

    def to_dict(self) -> Dict[str, Any]:
        return asdict(self)

    # ------------------------------------------------------------------ loading
    @classmethod
    def load(cls, model_dir: str) -> "ModelConfig":
        with open(os.path.join(model_dir, "config.json")) as f:
            raw = json.load(f)
        cfg = cls.from_json(raw)
        # eos ids may also live in generation_config.json / tokenizer_config.json
        for name in ("generation_config.json",):
            p = os.path.join(model_dir, name)
            if os.path.exists(p):
                try:
                    with open(p) as f:
                        g = json.load(f)
                    cfg._add_eos(g.get("eos_token_id"))
                except (OSError, ValueError):
                    pass
        hq = os.path.join(model_dir, "hf_quant_config.json")
        if cfg.quantization_config is None and os.path.exists(hq):
            with open(hq) as f:
                cfg.quantization_config = {"hf_quant_config": json.load(f)}
        return cfg

    def _add_eos(self, v) -> None:
        if v is None:
            return
        ids = v if isinstance(v, list) else [v]
        for i in ids:
            if isinstance(i, int) and i not in self.eos_token_ids:
                self.eos_token_ids.append(i)

    @classmethod
    def from_json(cls, raw: Dict[str, Any]) -> "ModelConfig":
        if raw.get("architecture") == "Sevevik":
            return cls._from_sevevik(raw)
        if raw.get("architecture") == "Niletar":
            return cls._from_niletar(raw)
        if raw.get("architecture") == "Rapisun":
            return cls._from_rapisun(raw)
        if raw.get("architecture") == "Medodra":
            return cls._from_medodra(raw)
        archs = raw.get("architectures") or ["Qwen3ForCausalLM"]
        t = raw.get("text_config", raw)
        g = lambda k, d=None: t.get(k, raw.get(k, d))  # noqa: E731
        model_type = g("model_type", "qwen3")
        n_layers = int(g("num_hidden_layers", 2))
        heads = int(g("num_attention_heads", 4))
        hidden = int(g("hidden_size", 256))
        cfg = cls(
            architecture=archs[0],
            model_type=model_type,
            vocab_size=int(g("vocab_size", 1024)),
            hidden_size=hidden,
            num_layers=n_layers,
            num_heads=heads,
            num_kv_heads=int(g("num_key_value_heads", heads)),
            head_dim=int(g("head_dim", hidden // heads)),
            intermediate_size=int(g("intermediate_size", 4 * hidden)),
            rms_norm_eps=float(g("rms_norm_eps", 1e-6)),
            tie_word_embeddings=bool(g("tie_word_embeddings", False)),
            max_position_embeddings=int(g("max_position_embeddings", 32768)),
            attention_bias=bool(g("attention_bias", False)),
            linear_num_key_heads=int(g("linear_num_key_heads", 0) or 0),
            linear_num_value_heads=int(g("linear_num_value_heads", 0) or 0),
            linear_key_head_dim=int(g("linear_key_head_dim", 0) or 0),
            linear_value_head_dim=int(g("linear_value_head_dim", 0) or 0),
            linear_conv_kernel_dim=int(g("linear_conv_kernel_dim", 4) or 4),
            num_experts=int(g("num_experts", 0) or 0),
            num_experts_per_tok=int(g("num_experts_per_tok", 0) or 0),
            moe_intermediate_size=int(g("moe_intermediate_size", 0) or 0),
            shared_expert_intermediate_size=int(g("shared_expert_intermediate_size", 0) or 0),
            norm_topk_prob=bool(g("norm_topk_prob", True)),
            mtp_num_hidden_layers=int(g("mtp_num_hidden_layers", 0) or 0),
            bos_token_id=g("bos_token_id"),
            quantization_config=raw.get("quantization_config", t.get("quantization_config")),
            torch_dtype=str(g("torch_dtype", g("dtype", "bfloat16"))),
            vision_config=raw.get("vision_config"),
        )
        cfg._add_eos(g("eos_token_id"))
        hc = int(g("hc_count", 0) or 0)
        if hc > 1:
            cfg.hc_count, cfg.hc_lowrank = hc, int(g("hc_lowrank", 16) or 16)
        ple_ids = g("ple_layer_ids")
        if ple_ids:
            # the checkpoint counts layers from 1 (SGLang: layer_id + 1 in ple_layer_ids)
            cfg.ple_layers = [int(i) - 1 for i in ple_ids if int(i) >= 1]
            cfg.ngram_size = int(g("ngram_size"))
            cfg.heads_per_ngram = int(g("heads_per_ngram"))
            cfg.ple_embed_dim = int(g("ple_embed_dim"))
            cfg.ple_conv_kernel = int(g("ple_conv_kernel_size", 4) or 4)
        cfg.gdn_output_gate = str(g("output_gate_type", "silu") or "silu")
        if g("indexer_n_heads"):
            cfg.indexer_heads, cfg.indexer_head_dim = int(g("indexer_n_heads")), int(g("indexer_head_dim", 0) or 0)
            cfg.indexer_budget, cfg.indexer_compress_ratio = int(g("indexer_budget", 0) or 0), int(g("indexer_compress_ratio", 0) or 0)
        # layer pattern
        lt = g("layer_types")
        if lt:
            cfg.layer_types = [
                "linear_attention" if x in ("linear_attention", "gdn", "linear") else "full_attention" for x in lt
            ]
        else:
            interval = g("full_attention_interval")
            if interval and cfg.linear_num_value_heads > 0:
                interval = int(interval)
                cfg.layer_types = [
                    "full_attention" if (i + 1) % interval == 0 else "linear_attention" for i in range(n_layers)
                ]
            else:
                cfg.layer_types = ["full_attention"] * n_layers
        # architecture family switches
        hybrid = cfg.has_gdn or model_type in ("qwen3_next", "qwen3_5", "qwen3_5_moe", "qwen3_6", "qwen3_8", "qwen4_exp")
        cfg.attn_output_gate = bool(g("attn_output_gate", hybrid))
        cfg.zero_centered_norm = bool(g("zero_centered_norm", hybrid))
        cfg.qk_norm = bool(g("qk_norm", model_type.startswith(("qwen3", "qwen4"))))
        # rope
        rp = g("rope_parameters") or g("rope_scaling") or {}
        rope = RopeConfig(
            theta=float(rp.get("rope_theta", g("rope_theta", 1.0e4))),
            partial_rotary_factor=float(rp.get("partial_rotary_factor", g("partial_rotary_factor", 1.0))),
            mrope_section=rp.get("mrope_section"),
        )
        rtype = rp.get("rope_type", rp.get("type"))
        if rtype == "yarn":
            rope.yarn_factor = float(rp.get("factor", 1.0))
            rope.yarn_original_max_position = int(
                rp.get("original_max_position_embeddings", cfg.max_position_embeddings)
            )
            rope.yarn_beta_fast = float(rp.get("beta_fast", 32.0))
            rope.yarn_beta_slow = float(rp.get("beta_slow", 1.0))
            if rp.get("attention_factor") is not None:
                rope.yarn_attention_factor = float(rp["attention_factor"])
        cfg.rope = rope
        return cfg

    @classmethod
    def _from_sevevik(cls, raw: Dict[str, Any]) -> "ModelConfig":
        """The layer-by-layer configuration of the Sevevik design."""
        specs: List[LayerSpec] = []
        for i, e in enumerate(raw["layers"]):
            if e["type"] != "attention":
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            m = e["mixer"]
            mask = m.get("mask") or {}
            attn = DiffAttnSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                scale=float(m["scale"]), diff=float(m["diff"]), window=int(mask.get("size") or 0))
            specs.append(LayerSpec(attn, _dense_mlp(i, e, limit=True), _weights_of(e)))
        _check_layers(specs)
        return cls.of_layers(specs, architecture="Sevevik", model_type="sevevik", vocab_size=int(raw["vocab"]),
                             hidden_size=int(raw["width"]), rms_norm_eps=float(raw["norm"]["eps"]), streams=int(raw.get("streams", 1)),
                             residual_mult=float(raw.get("residual_mult", 1.0)),
                             embed_scale=float((raw.get("embedding") or {}).get("scale", 1.0)),
                             torch_dtype=str(raw.get("torch_dtype", "bfloat16")))

    @classmethod
    def _from_niletar(cls, raw: Dict[str, Any]) -> "ModelConfig":
        """The layer-by-layer configuration of the Niletar design."""
        specs: List[LayerSpec] = []
        for i, e in enumerate(raw["layers"]):
            m, attn = e["mixer"], None
            if e["type"] == "mamba2":
                rec = StateSpaceSpec(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]),
                                     norm_groups=int(m["norm_groups"]), conv=int(m["conv"]))
            elif e["type"] == "parallel":
                l, r = m["left"], m["right"]
                attn = SoftAttnSpec(heads=int(l["heads"]), kv_heads=int(l["kv_heads"]), dim=int(l["dim"]), vdim=int(l["vdim"]),
                                    scale=float(l["scale"]), rot=_rotary(l.get("rot")), bias=True, unit_rms=True, sink=True, gate=True,
                                    out_scale=float(m["left_scale"]))
                rec = DeltaSpec(heads=int(r["heads"]), kv_heads=int(r["kv_heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]),
                                conv=int(r["conv"]), out_scale=float(m["right_scale"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            specs.append(LayerSpec(attn, _dense_mlp(i, e, limit=False), _weights_of(e), rec))
        _check_layers(specs)
        return cls.of_layers(specs, architecture="Niletar", model_type="niletar", vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]),
                             rms_norm_eps=float(raw["norm"]["eps"]), zero_centered_norm=True, residual_alpha=float(raw["postln_alpha"]),
                             torch_dtype=str(raw.get("torch_dtype", "bfloat16")))

    @classmethod
    def _from_rapisun(cls, raw: Dict[str, Any]) -> "ModelConfig":
        """The layer-by-layer configuration of the Rapisun design."""
        specs: List[LayerSpec] = []
        for i, e in enumerate(raw["layers"]):
            m, attn, rec = e["mixer"], None, None
            if e["type"] == "hgrn2":
                rec = GatedLinearSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
            elif e["type"] == "latent_attention":
                src = m.get("kv_from")
                attn = LatentAttnSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                      q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=_rotary(m.get("rot")),
                                      sink=True, window=int((m.get("mask") or {}).get("size") or 0), kv_from=None if src is None else int(src))
                if attn.rot is not None:
                    attn.rot.interleaved = False
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            specs.append(LayerSpec(attn, _norm_or_moe(i, e), None, rec))
        _check_layers(specs)
        taps = int((raw.get("canon") or {}).get("taps") or 0)
        if taps < 0:
            raise ValueError(f"an input convolution of {taps} taps")
        return cls.of_layers(specs, architecture="Rapisun", model_type="rapisun", vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]),
                             rms_norm_eps=float(raw["norm"]["eps"]), input_conv=taps, torch_dtype=str(raw.get("torch_dtype", "bfloat16")))

    @classmethod
    def _from_medodra(cls, raw: Dict[str, Any]) -> "ModelConfig":
        """The layer-by-layer configuration of the Medodra design."""
        specs: List[LayerSpec] = []
        for i, e in enumerate(raw["layers"]):
            m, attn = e["mixer"], None
            if e["type"] == "delta":
                rec = DeltaSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), conv=int(m["conv"]),
                                head_decay=True, gate="silu")
            elif e["type"] == "parallel":
                l, t = m["left"], m["left"].get("q_temp") or {"coef": 0.0, "every": 1.0}
                attn = SigmoidAttnSpec(heads=int(l["heads"]), kv_heads=int(l["kv_heads"]), dim=int(l["dim"]), vdim=int(l["vdim"]),
                                       scale=float(l["scale"]), far=float(l["bias_max"]), bias=True, conv=int(l["conv"]), unit_v=True,
                                       temp_coef=float(t["coef"]), temp_every=float(t["every"]))
                rec = MinGruSpec(int(m["right"]["width"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            specs.append(LayerSpec(attn, _gated_moe(i, e), None, rec))
        specs = _unrolled(specs, raw.get("loop"))
        _check_layers(specs)
        return cls.of_layers(specs, architecture="Medodra", model_type="medodra", vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]),
                             rms_norm_eps=float(raw["norm"]["eps"]), zero_centered_norm=True, residual_mult=float(raw["residual_mult"]),
                             embed_scale=float(raw["embedding"]["scale"]), torch_dtype=str(raw.get("torch_dtype", "bfloat16")))

    @classmethod
    def of_layers(cls, specs: List[LayerSpec], **kw) -> "ModelConfig":
        """A configuration from its layer list; the model-wide sizes that other parts read are those of the first layer."""
        a = next((s.attn for s in specs if s.attn is not None), None)
        r, mlp = specs[0].rec, specs[0].mlp
        heads = (a.heads, a.kv_heads, a.dim) if a is not None else (r.heads, r.heads, r.vdim)
        return cls(layer_specs=specs, num_layers=len(specs), num_heads=heads[0], num_kv_heads=heads[1], head_dim=heads[2],
                   intermediate_size=mlp.ff if mlp else 0, qk_norm=False, layer_types=[s.kind for s in specs], **kw)


def _weights_of(entry: Dict[str, Any]) -> Optional[int]:
    v = entry.get("weights_of")
    return None if v is None else int(v)


def _dense_mlp(i: int, entry: Dict[str, Any], limit: bool) -> Optional[GluSpec]:
    m = entry.get("mlp")
    if m is None:
        return None
    if m.get("kind", "dense") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {m['kind']!r}")
    return GluSpec(ff=int(m["ff"]), limit=float(m["limit"]) if limit else None)


def _norm_or_moe(i: int, entry: Dict[str, Any]) -> Union[PolyNormSpec, MoeSpec, None]:
    m = entry.get("mlp")
    if m is None:
        return None
    if m.get("kind") == "dense":
        return PolyNormSpec(ff=int(m["ff"]))
    if m.get("kind") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {m.get('kind')!r}")
    shared = m.get("shared")
    return MoeSpec(experts=int(m["router"]["experts"]), top=int(m["router"]["top"]), ff=int(m["expert"]["ff"]),
                   shared_ff=int(shared["ff"]) if shared else 0)


def _gated_moe(i: int, entry: Dict[str, Any]) -> Optional[MoeSpec]:
    m = entry.get("mlp")
    if m is None:
        return None
    if m.get("kind") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {m.get('kind')!r}")
    shared = m.get("shared")
    return MoeSpec(experts=int(m["router"]["experts"]), top=int(m["router"]["top"]), ff=int(m["expert"]["ff"]),
                   shared_ff=int(shared["ff"]) if shared else 0, act="swiglu", scores="sigmoid", renorm=False, weigh_input=True,
                   shared_gate=bool(shared))


def _unrolled(specs: List[LayerSpec], loop: Optional[Dict[str, Any]]) -> List[LayerSpec]:
    """The layers in the order they run: those of ``loop`` (start, stop, times) stand there once per pass, later passes with the tensors
    of the first."""
    if not loop:
        return specs
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start < stop <= len(specs) or times < 1:
        raise ValueError(f"a loop over layers {start} .. {stop - 1} of {len(specs)}, {times} times")
    out = specs[:start]
    for k in range(times):
        out += [replace(s, number=i, joins=i == start, weights_of=i if k else None) for i, s in enumerate(specs[start:stop], start)]
    return out + [replace(s, number=i) for i, s in enumerate(specs[stop:], stop)]


def _rotary(rot: Optional[Dict[str, Any]]) -> Optional[RotarySpec]:
    if not rot:
        return None
    r, sc = RotarySpec(dims=int(rot["dims"]), base=float(rot["base"])), rot.get("scaling")
    if sc:
        r.factor, r.low, r.high, r.original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    return r


def _check_layers(specs: List[LayerSpec]) -> None:
    """Refuse a layer list that no model of the design can have."""
    if not specs:
        raise ValueError("the configuration lists no layers")
    for i, s in enumerate(specs):
        a, r = s.attn, s.rec
        if a is not None:
            if min(a.heads, a.kv_heads, a.dim, a.vdim) < 1 or a.heads % a.kv_heads:
                raise ValueError(f"layer {i}: {a.heads} query heads over {a.kv_heads} key/value heads of {a.dim} / {a.vdim}")
            if a.window < 0:
                raise ValueError(f"layer {i}: a window of {a.window}")
            if isinstance(a, SigmoidAttnSpec) and (a.conv < 0 or a.temp_every <= 0 or a.far <= 0):
                raise ValueError(f"layer {i}: a convolution of {a.conv} taps, distances up to {a.far}, query temperature steps of {a.temp_every}")
            rot, turned = getattr(a, "rot", None), a.rot_dim if isinstance(a, LatentAttnSpec) else a.dim
            if rot is not None and (rot.dims % 2 or not 0 <= rot.dims <= turned):
                raise ValueError(f"layer {i}: rotary positions on {rot.dims} of {turned} dimensions")
            if isinstance(a, LatentAttnSpec):
                if min(a.rot_dim, a.q_rank, a.kv_rank) < 1:
                    raise ValueError(f"layer {i}: latents of {a.q_rank} / {a.kv_rank} and a rotated part of {a.rot_dim} columns")
                if a.kv_from is not None:
                    src = specs[a.kv_from].attn if 0 <= a.kv_from < i else None
                    if not isinstance(src, LatentAttnSpec) or src.kv_from is not None:
                        raise ValueError(f"layer {i} reads the latents of layer {a.kv_from}, which has none of its own before it")
                    if (src.kv_rank, src.rot_dim, src.rot) != (a.kv_rank, a.rot_dim, a.rot):
                        raise ValueError(f"layer {i} reads latents of layer {a.kv_from} that have another size or rotation")
        if r is not None:
            groups = r.groups if isinstance(r, StateSpaceSpec) else r.kv_heads if isinstance(r, DeltaSpec) else r.heads
            taps = r.conv if not isinstance(r, (GatedLinearSpec, MinGruSpec)) else 1
            if min(r.heads, groups, r.state, r.vdim, taps) < 1 or r.heads % groups:
                raise ValueError(f"layer {i}: {r.heads} recurrent heads over {groups} groups, state {r.state} x {r.vdim}, {r.conv} taps")
            if isinstance(r, StateSpaceSpec) and (r.norm_groups < 1 or r.inner % r.norm_groups):
                raise ValueError(f"layer {i}: {r.inner} columns in {r.norm_groups} norm groups")
        if isinstance(s.mlp, MoeSpec) and (not 1 <= s.mlp.top <= s.mlp.experts or s.mlp.ff < 1):
            raise ValueError(f"layer {i}: {s.mlp.top} of {s.mlp.experts} experts of {s.mlp.ff}")
        if s.weights_of is not None:
            src = specs[s.weights_of] if 0 <= s.weights_of < len(specs) else None
            if src is None or src.weights_of is not None:
                raise ValueError(f"layer {i} uses the tensors of layer {s.weights_of}, which has none of its own")
            if (src.attn, src.rec, src.mlp) != (a, r, s.mlp):
                raise ValueError(f"layer {i} differs from layer {s.weights_of}, whose tensors it uses")


def inv_freq(cfg: ModelConfig, yarn_factor_override: Optional[float] = None):
    """Rotary inverse frequencies (fp32 list), with YaRN blending when enabled.

    Same role as the reference's ``inv_freq`` (``crates/blaze/src/model.rs:991``).
    """
    rd = cfg.rotary_dim
    half = rd // 2
    r = cfg.rope
    base = [r.theta ** (-(2.0 * i) / rd) for i in range(half)]
    factor = yarn_factor_override if yarn_factor_override else r.yarn_factor
    if factor <= 1.0:
        return base
    orig = r.yarn_original_max_position or cfg.max_position_embeddings

    def corr_dim(rot):
        return (rd * math.log(orig / (rot * 2 * math.pi))) / (2 * math.log(r.theta))

    low = max(math.floor(corr_dim(r.yarn_beta_fast)), 0)
    high = min(math.ceil(corr_dim(r.yarn_beta_slow)), rd - 1)
    if low == high:
        high += 0.001
    out = []
    for i, f in enumerate(base):
        ramp = min(max((i - low) / (high - low), 0.0), 1.0)
        extrap = 1.0 - ramp  # 1 → keep original frequency
        out.append((f / factor) * (1 - extrap) + f * extrap)
    return out


# ---------------------------------------------------------------------------------- named shapes
def named_config(name: str) -> ModelConfig:
    """Shapes of the benchmark models (random-init; no checkpoint needed)."""
    n = name.lower()
    if n in ("tiny", "tiny-qwen3"):
        c = ModelConfig(vocab_size=1024, hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=64,
                        intermediate_size=512, rope=RopeConfig(theta=1e6))
    elif n in ("tiny-hybrid",):
        # two Gated DeltaNet layers and two gated-attention layers with a small MoE: the Qwen3-Next layer pattern in miniature
        c = ModelConfig(architecture="Qwen3NextForCausalLM", model_type="qwen3_next", vocab_size=1024, hidden_size=256,
                        num_layers=4, num_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=512, num_experts=8,
                        num_experts_per_tok=2, moe_intermediate_size=128, shared_expert_intermediate_size=128,
                        linear_num_key_heads=2, linear_num_value_heads=4, linear_key_head_dim=128, linear_value_head_dim=64,
                        linear_conv_kernel_dim=4, attn_output_gate=True, zero_centered_norm=True,
                        rope=RopeConfig(theta=1e6, partial_rotary_factor=0.25))
        c.layer_types = ["linear_attention", "full_attention", "linear_attention", "full_attention"]
    elif n in ("tiny-qwen4",):
        # the hybrid in miniature with two residual streams and an n-gram embedding on two of its layers
        c = named_config("tiny-hybrid")
        c.architecture, c.model_type = "Qwen4ExpForCausalLM", "qwen4_exp"
        c.hc_count, c.hc_lowrank = 2, 8
        c.ple_layers, c.ngram_size, c.heads_per_ngram, c.ple_embed_dim, c.ple_conv_kernel = [0, 2], 3, 2, 16, 4
        c.eos_token_ids = [1]
    elif n in ("tiny-sevevik",):
        # the Sevevik layer kinds in miniature: unequal layers, one without a feed-forward, one that uses another's tensors
        a = DiffAttnSpec(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.2, diff=0.35, window=40)
        b = DiffAttnSpec(heads=3, kv_heads=1, dim=16, vdim=64, scale=0.25, diff=0.2, window=24)
        layers = [LayerSpec(a, GluSpec(320, 3.0)), LayerSpec(b), LayerSpec(a, GluSpec(320, 3.0), weights_of=0)]
        return ModelConfig.of_layers(layers, architecture="Sevevik", model_type="sevevik", vocab_size=1024, hidden_size=192,
                                     streams=3, residual_mult=0.8, embed_scale=6.0)
    elif n in ("tiny-niletar",):
        # the Niletar layer kinds in miniature, one without a feed-forward, one that uses another's tensors
        def mamba(**kw):
            return StateSpaceSpec(**{**dict(heads=6, vdim=32, state=48, groups=2, norm_groups=3, conv=4), **kw})
        a = SoftAttnSpec(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.2, rot=RotarySpec(24, 1.0e4, factor=4.0, original=256.0), bias=True,
                         unit_rms=True, sink=True, gate=True, out_scale=0.7)
        d = DeltaSpec(heads=4, kv_heads=2, dim=32, vdim=40, conv=3, out_scale=0.4)
        layers = [LayerSpec(a, GluSpec(320), None, d), LayerSpec(None, None, None, mamba()), LayerSpec(a, GluSpec(320), 0, d)]
        return ModelConfig.of_layers(layers, architecture="Niletar", model_type="niletar", vocab_size=1024, hidden_size=192,
                                     zero_centered_norm=True, residual_alpha=1.8)
    elif n in ("tiny-rapisun",):
        # the Rapisun layer kinds in miniature: both mixers, both feed-forwards and none, latents read by a later layer
        def latent(**kw):
            return LatentAttnSpec(**{**dict(heads=4, dim=24, rot_dim=16, vdim=40, q_rank=48, kv_rank=64, scale=0.16,
                                            rot=RotarySpec(16, 1.0e4, False), sink=True, window=40), **kw})
        layers = [LayerSpec(None, PolyNormSpec(288), None, GatedLinearSpec(4, 32, 48)), LayerSpec(latent(), MoeSpec(8, 2, 64, 96)),
                  LayerSpec(latent(heads=6, window=24, kv_from=1)), LayerSpec(None, MoeSpec(8, 2, 64), None, GatedLinearSpec(2, 48, 32))]
        return ModelConfig.of_layers(layers, architecture="Rapisun", model_type="rapisun", vocab_size=1024, hidden_size=192, input_conv=4)
    elif n in ("tiny-medodra",):
        # the Medodra layer kinds in miniature, one without a feed-forward, with a loop over two of three layers
        a = SigmoidAttnSpec(4, 2, 32, 48, 0.2, 100.0, True, 4, True, 0.2, 64.0)
        d = DeltaSpec(4, 2, 32, 40, 3, head_decay=True, gate="silu")
        moe = MoeSpec(8, 2, 64, 96, "swiglu", "sigmoid", False, True, True)
        layers = [LayerSpec(a, moe, None, MinGruSpec(160)), LayerSpec(None, moe, None, d), LayerSpec(a, None, None, MinGruSpec(192))]
        return ModelConfig.of_layers(_unrolled(layers, {"start": 0, "stop": 2, "times": 2}), architecture="Medodra", model_type="medodra",
                                     vocab_size=1024, hidden_size=192, zero_centered_norm=True, residual_mult=0.8, embed_scale=0.5)
    elif n in ("qwen3-8b",):
        c = ModelConfig(vocab_size=151936, hidden_size=4096, num_layers=36, num_heads=32, num_kv_heads=8,
                        head_dim=128, intermediate_size=12288, rope=RopeConfig(theta=1e6))
    elif n in ("qwen3-32b",):
        c = ModelConfig(vocab_size=151936, hidden_size=5120, num_layers=64, num_heads=64, num_kv_heads=8,
                        head_dim=128, intermediate_size=25600, rope=RopeConfig(theta=1e6), mtp_num_hidden_layers=1)
    elif n in ("qwen3-30b-a3b",):
        c = ModelConfig(architecture="Qwen3MoeForCausalLM", model_type="qwen3_moe", vocab_size=151936,
                        hidden_size=2048, num_layers=48, num_heads=32, num_kv_heads=4, head_dim=128,
                        intermediate_size=6144, num_experts=128, num_experts_per_tok=8, moe_intermediate_size=768,
                        norm_topk_prob=True, rope=RopeConfig(theta=1e6))
    elif n in ("qwen3-next-80b-a3b",):
        c = ModelConfig(architecture="Qwen3NextForCausalLM", model_type="qwen3_next", vocab_size=151936,
                        hidden_size=2048, num_layers=48, num_heads=16, num_kv_heads=2, head_dim=256,
                        intermediate_size=5120, num_experts=512, num_experts_per_tok=10, moe_intermediate_size=512,
                        shared_expert_intermediate_size=512, linear_num_key_heads=16, linear_num_value_heads=32,
                        linear_key_head_dim=128, linear_value_head_dim=128, linear_conv_kernel_dim=4,
                        attn_output_gate=True, zero_centered_norm=True,
                        rope=RopeConfig(theta=1e7, partial_rotary_factor=0.25))
        c.layer_types = ["full_attention" if (i + 1) % 4 == 0 else "linear_attention" for i in range(48)]
    else:
        raise ValueError(f"unknown model shape {name!r}")
    if not c.layer_types:
        c.layer_types = ["full_attention"] * c.num_layers
    return c
