"""The Medodra design on the oracle op set: every mechanism and the whole model against the independent restatement in
``oracle_medodra.py``, through the package's loader, cache, engine, scheduler and command line."""
import copy
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import medodra_case as C
import oracle_medodra as O
from blaze_b200.config import DeltaSpec, MinGruSpec, ModelConfig, MoeSpec, SigmoidAttnSpec, named_config
from blaze_b200.llm import LLM
from blaze_b200.models import model_class
from blaze_b200.models.qwen3 import SigmoidAttn
from blaze_b200.ops import ref
from blaze_b200.ops.ref_ops import RefOps
from blaze_b200.sampler import SamplingParams
from test_niletar_cpu import verify_with_rejected_rows
from test_sevevik_cpu import ROOT, SCHEDULES, mixed_steps

EXACT = 1e-4            # fp32 rounding through these random models; a wrong key, state or constant gives 1e-2 and more
SHOWS = 1e-2
V = 320


@pytest.fixture(autouse=True, scope="module")
def few_threads():
    n = torch.get_num_threads()
    torch.set_num_threads(1)             # thousands of tiny products
    yield
    torch.set_num_threads(n)


def _llm(path, dtype=torch.float32, **kw):
    kw = {"kv_tokens": 1024, "max_seqs": 4, "max_model_len": 512, "enable_prefix_caching": False, **kw}
    return LLM(path, device="cpu", dtype=dtype, **kw)


@pytest.fixture(scope="module")
def case(tmp_path_factory):
    cfg = C.config()
    w = C.weights(cfg, seed=3)
    return cfg, w, C.save(tmp_path_factory.mktemp("medodra"), cfg, w)


def rand(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ----------------------------------------------------------------------------------- configuration and loading
def test_configuration_is_read_layer_by_layer():
    cfg = ModelConfig.from_json(C.config())
    assert cfg.architecture == "Medodra" and model_class(cfg).__name__ == "Medodra" and cfg.rms_norm_eps == 1e-5 and cfg.residual_mult == 0.6
    assert cfg.embed_scale == 0.7 and cfg.num_layers == 6
    s = cfg.layer_specs
    assert s[0].rec == DeltaSpec(4, 2, 24, 20, 3, 1.0, True, "silu") and s[0].mlp == MoeSpec(6, 2, 40, 56, "swiglu", "sigmoid", False, True, True)
    assert s[1].attn == SigmoidAttnSpec(6, 3, 16, 28, 0.3, 50.0, True, 4, True, 0.4, 24.0) and s[1].rec == MinGruSpec(88)
    assert [(x.number, x.joins, x.weights_of) for x in s] == [(None, False, None), (1, True, None), (2, False, None), (1, True, 1), (2, False, 2),
                                                              (3, False, None)]
    assert [cfg.layer_type(i) for i in (0, 1)] == ["delta_rule", "sigmoid_attention+min_gru"]
    assert ModelConfig.from_json(C.config(loop=None)).num_layers == 4
    assert [x.joins for x in ModelConfig.from_json(C.config(loop=(0, 4, 1))).layer_specs] == [True, False, False, False]


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"]["left"]["q_temp"].update(every=0),
    lambda c: c["layers"][1]["mixer"]["left"].update(bias_max=0), lambda c: c["layers"][1]["mixer"]["right"].update(width=0),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=7), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c["loop"].update(stop=5), lambda c: c["loop"].update(start=3), lambda c: c["loop"].update(times=0), lambda c: c.update(layers=[])])
def test_configurations_that_make_no_model_are_refused(change):
    c = copy.deepcopy(C.config())
    change(c)
    with pytest.raises(ValueError):
        ModelConfig.from_json(c)


def test_tensors_of_the_wrong_shape_are_refused(tmp_path, case):
    cfg, w, _ = case
    for name in ("l0.mix.a", "l1.mix.left.k.conv", "l1.mix.right.x.b", "l0.mlp.e5.up", "l1.mlp.shared.sg", "loop.in", "l3.mix.left.out"):
        with pytest.raises(ValueError, match="asks for"):
            _llm(C.save(tmp_path, cfg, dict(w, **{name: w[name].new_zeros((*w[name].shape[:-1], w[name].shape[-1] + 1))})))
    with pytest.raises(ValueError, match="distances"):
        _llm(C.save(tmp_path, cfg, dict(w, **{"l1.mix.left.rel": w["l1.mix.left.rel"].repeat(8, 1)})))


def test_pages_and_states_follow_each_layers_sizes(case):
    llm = _llm(case[2])
    kv = llm.engine.kv
    assert sorted(kv.k) == [1, 3, 5] and kv.k[1].shape[1:] == (3, 16, 16) and kv.v[3].shape[1:] == (3, 16, 28) and kv.k[5].shape[1:] == (1, 16, 24)
    assert kv.k[1] is not kv.k[3]                        # every pass keeps its own
    assert kv.rec_state[0].shape[1:] == (4, 24, 20) and kv.rec_state[1].shape[1:] == (1, 1, 88) and kv.rec_state[5].shape[1:] == (1, 1, 60)
    assert sorted(kv.conv_state) == [0, 2, 4] and kv.conv_state[2].shape[1:] == (240, 1)
    assert kv.qkv_state[1].shape[1:] == (3, 6 * 16 + 3 * 44) and kv.qkv_state[5].shape[1:] == (1, 4 * 24 + 56) and kv.state_layers == list(range(6))
    assert all(t.dtype == torch.float32 for t in kv.rec_state.values())
    matrices = [n for n, t in case[1].items() if t.dim() == 2 and not n.endswith(("conv", "rel"))]
    assert llm.model.weight_bytes() >= sum(case[1][n].numel() * 4 for n in matrices)
    assert llm.model.layers[1] is llm.model.layers[3]    # one set of tensors


def test_what_the_design_does_not_have_is_refused(case):
    with pytest.raises(ValueError, match="bf16 or fp32"):
        _llm(case[2], kv_cache_dtype="fp8")
    with pytest.raises(ValueError, match="dense"):
        LLM("tiny-medodra", device="cpu", weight_format="nvfp4")
    with pytest.raises(ValueError, match="drafters"):
        _llm(case[2], spec_method="mtp")


# ----------------------------------------------------------------------------------- mechanisms alone
def test_embedding_with_position_vectors():
    from blaze_b200.models.qwen3 import _two_floats
    for W in (10, 7):
        table, tok = rand(20, W), torch.arange(20)
        freq = _two_floats([10000.0 ** (-2.0 * i / W) for i in range((W + 1) // 2)], "cpu")
        copy = torch.empty(20, W, dtype=torch.bfloat16)
        got = RefOps().embed_positions(table, tok, torch.arange(20), 0.3, freq, copy)
        assert torch.allclose(got.double(), O.embedding(tok, table.double(), 0.3), atol=1e-6) and torch.equal(copy, got.bfloat16())


def test_branches_and_norms():
    from blaze_b200.models.qwen3 import Branches
    x, y, z, f, w1, w2, n1 = rand(5, 24), rand(5, 24, seed=1), rand(5, 24, seed=2), rand(5, 24, seed=3), rand(24, seed=4), rand(24, seed=5), rand(24, seed=6)
    got, a, b = RefOps().branch_step(x, Branches((y, z), (w1, w2), f, 0.7), 1e-2, torch.float32, 1 + n1, None)
    want = x.double() + 0.7 * ((O.rms(y.double(), 1e-2) * w1 + O.rms(z.double(), 1e-2) * w2) / 2 + f)
    assert torch.allclose(got.double(), want, atol=1e-5) and b is None
    assert torch.allclose(a.double(), O.norm(want, n1.double(), 1e-2), atol=1e-5)
    got, a, b = RefOps().branch_step(x, Branches(y, None, None, 0.3), 1e-2, torch.bfloat16, None, w2)
    assert torch.allclose(got, x + 0.3 * y, atol=1e-6) and a is None and b.dtype == torch.bfloat16


@pytest.mark.parametrize("rows,far", [(16, 50), (32, 250), (8, 64), (6, 1000.0), (2, 1.5), (32, 256), (64, 33)])
def test_distance_buckets(rows, far):
    spec = SigmoidAttnSpec(2, 1, 8, 8, 0.5, far)
    rel, pb = rand(rows, 2), rand(2, seed=1)
    A = SigmoidAttn(spec, "cpu", rel, pb)
    for n in range(min(A.reach + 20, 2000)):
        want = rel[O.distance_bucket(n, rows, far)] + pb
        assert torch.allclose(A.bias[:, A.PAD + min(n, A.reach - 1)], want, atol=1e-6), n
    assert A.bias.shape[1] == A.reach + 2 * A.PAD and bool((A.bias[:, :A.PAD] == float("-inf")).all())
    assert torch.equal(A.bias[:, -1], A.bias[:, A.PAD + A.reach - 1])


def test_query_temperature_steps():
    p = torch.arange(200)
    got = ref.query_temperature(p, 0.3, 24.0)
    assert torch.allclose(got.double(), torch.tensor([O.query_temperature(i, 0.3, 24) for i in range(200)], dtype=torch.float64), atol=1e-6)
    assert got[22] == 1 and got[23] > 1.2                # position 23 is the 24th token


def test_convolution_keeps_its_history():
    for taps in (1, 2, 4, 7):
        x, w = rand(30, 12), rand(12, taps, seed=1)
        st, out = torch.zeros(taps - 1, 12), []
        for n in (1, 2, 9, 1, 17):
            y, st = ref.causal_conv(x[sum(map(len, out)):][:n], st, w.t())
            out.append(y)
        assert st.shape == (taps - 1, 12) and torch.allclose(torch.cat(out).double(), O.causal_conv(x.double(), w.double()), atol=1e-5)


def test_sigmoid_attention_sees_one_key_among_many():
    """A key that stands out shows at every distance, with the bias of its distance; weights are no shares."""
    n, d, e, near, spec = 120, 8, 6, 8, SigmoidAttnSpec(1, 1, 8, 6, 0.5, 40.0)
    q, k, v = rand(n, d), rand(n, d, seed=1) * 0.1, rand(n, e, seed=2)
    k[3] = 4 * torch.ones(d)
    q[50] = q[119] = torch.ones(d)
    rel, pb = rand(16, 1, seed=3) * 2, torch.tensor([-3.0])
    A = SigmoidAttn(spec, "cpu", rel, pb)
    pages = lambda t: torch.cat([t, t.new_zeros(8, t.shape[1])]).view(8, 1, 16, -1)      # noqa: E731
    got = ref.sigmoid_attention(q[:, None], pages(k), pages(v), torch.arange(8).view(1, 8), [0], [0, n], [n], 0.5, A.bias, A.PAD)[:, 0]
    bias = torch.stack([rel[O.distance_bucket(i, 16, 40), 0] for i in range(n)]).double()
    want = O.sigmoid_attention(q.double(), k.double(), v.double(), 0.5, bias, pb[0].double())
    assert torch.allclose(got.double(), want, atol=1e-5)
    gone = O.sigmoid_attention(q.double(), torch.cat([k[:3], -k[3:4], k[4:]]).double(), v.double(), 0.5, bias, pb[0].double())
    for i in (50, 119):
        assert (want[i] - gone[i] - v[3].double()).abs().max() < 0.05
    shifted = O.sigmoid_attention(q.double(), k.double(), v.double(), 0.5, bias.roll(1), pb[0].double())
    assert (shifted - want).abs().max() > SHOWS


def test_delta_rule_with_head_decay_in_portions():
    T, H, G, d, e = 40, 4, 2, 12, 10
    q, k, v, a, b = rand(T, G, d), rand(T, G, d, seed=1), rand(T, H, e, seed=2), rand(T, H, 1, seed=3), rand(T, H, seed=4)
    A, bias, S, outs = rand(H, seed=5).abs(), rand(H, seed=6) - 1, torch.zeros(H, d, e), []
    for i, n in ((0, 1), (1, 2), (3, 20), (23, 17)):
        s = slice(i, i + n)
        o, S = ref.delta_rule(q[s], k[s], v[s], a[s], b[s], A, bias, S)
        outs.append(o)
    g = torch.exp(-A.double() * O.softplus(a[..., 0].double() + bias.double()))
    for h in range(H):
        want = O.delta_rule(O.unit(q[:, h // 2].double()) * d ** -0.5, O.unit(k[:, h // 2].double()), v[:, h].double(), g[:, h], O.sigmoid(b[:, h].double()))
        assert torch.allclose(torch.cat(outs)[:, h].double(), want, atol=1e-5)


def test_min_gru_in_portions():
    z, u, S, outs = rand(40, 9) * 2, rand(40, 9, seed=1) * 2, torch.zeros(9), []
    for i, n in ((0, 1), (1, 2), (3, 20), (23, 17)):
        o, S = ref.min_gru(z[i:i + n], u[i:i + n], S)
        outs.append(o)
    assert torch.allclose(torch.cat(outs).double(), O.min_gru(O.sigmoid(z.double()), u.double()), atol=1e-5)


def test_routing_weighs_the_inputs():
    from blaze_b200.models.qwen3 import Experts
    from blaze_b200.linear import Linear
    z = rand(6, 30) * 2
    w, ids = ref.router_topk(z, 5, False, True)
    best, weight = O.route(z.double(), 5)
    assert torch.equal(ids.long(), best) and torch.allclose(w.double(), weight, atol=1e-6)
    assert torch.equal(RefOps().router_topk(torch.cat([z, z + 9], 1), 5, False, sigmoid=True, n_exp=30)[1], ids)
    E, W, ff, p = 3, 16, 8, "m."
    t = {f"{p}e{e}.{n}": rand(*s, seed=7 * e + len(n)) for e in range(E) for n, s in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff)))}
    t.update({p + "router": rand(E, W, seed=50), p + "shared.sg": rand(1, W, seed=51), p + "shared.gate": rand(ff, W, seed=52),
              p + "shared.up": rand(ff, W, seed=53), p + "shared.down": rand(W, ff, seed=54)})
    ex = Experts()
    ex.num_experts = ex.count = E
    ex.weigh_input = True
    for e in range(E):
        ex.gate_up.append(Linear.from_dense(torch.cat([t[f"{p}e{e}.gate"], t[f"{p}e{e}.up"]]), dtype=torch.float32))
        ex.down.append(Linear.from_dense(t[f"{p}e{e}.down"], dtype=torch.float32))
    x = rand(11, W, seed=60)
    w, ids = ref.router_topk(x @ t[p + "router"].t(), 2, False, True)
    shared = O.expert(x, t, p + "shared.")
    got = RefOps().moe_rows(x, w, ids, ex, shared, (x @ t[p + "shared.sg"].t())[:, 0])
    m = {"router": {"experts": E, "top": 2}, "shared": {"ff": ff}}
    assert torch.allclose(got, O.mixture(x, t, p, m), atol=1e-4, rtol=1e-4)


# ----------------------------------------------------------------------------------- the whole model
@pytest.fixture(scope="module")
def reference(case):
    cfg, w, _ = case
    seqs = {"a": C.tokens(150, V, 1), "b": C.tokens(67, V, 2), "c": C.tokens(33, V, 3), "d": C.tokens(1, V, 4), "e": C.tokens(90, V, 5)}
    return seqs, {i: O.forward(cfg, w, t) for i, t in seqs.items()}


@pytest.mark.parametrize("name", SCHEDULES)
def test_logits_do_not_depend_on_how_a_prompt_is_cut(case, reference, name):
    seqs, want = reference
    eng = _llm(case[2]).engine
    for i in ("a", "c", "d"):
        got = C.run(eng, {i: seqs[i]}, [[(i, n)] for n in SCHEDULES[name](len(seqs[i]))])[i]
        assert C.error(got, want[i]) < EXACT, i


def test_batches_of_unequal_requests_match_each_alone(case, reference):
    seqs, want = reference
    eng = _llm(case[2], kv_tokens=320, max_seqs=3).engine  # less than the sum of the requests: pages and state rows are used again
    for _ in range(2):
        got = C.run(eng, seqs, mixed_steps(seqs))
        for i in seqs:
            assert C.error(got[i], want[i]) < EXACT, i
    assert eng.pages.free_count == eng.num_pages - 1


def lefts(c):
    return [L["mixer"]["left"] for L in c["layers"] if L["type"] == "parallel"]


MISTAKES = {
    "no distance bias": lambda c, w: [w[f"l{i}.mix.left.rel"].zero_() for i in (1, 3)],
    "distances one off": lambda c, w: [w.update({f"l{i}.mix.left.rel": w[f"l{i}.mix.left.rel"].roll(1, 0)}) for i in (1, 3)],
    "reach of the table": lambda c, w: [l.update(bias_max=l["bias_max"] * 2) for l in lefts(c)],
    "number per head left out": lambda c, w: w["l1.mix.left.pb"].zero_(),
    "no query temperature": lambda c, w: [l["q_temp"].update(coef=0.0) for l in lefts(c)],
    "temperature steps": lambda c, w: [l["q_temp"].update(every=l["q_temp"]["every"] + 5) for l in lefts(c)],
    "oldest tap left out": lambda c, w: [w["l1.mix.left.k.conv"][:, 0].zero_(), w["l0.mix.v.conv"][:, 0].zero_()],
    "projection bias left out": lambda c, w: w["l1.mix.left.v.b"].zero_(),
    "output bias left out": lambda c, w: w["l3.mix.left.o.b"].zero_(),
    "gate bias of the recurrence": lambda c, w: w["l1.mix.right.z.b"].zero_(),
    "decay bias": lambda c, w: w["l0.mix.dt_bias"].add_(1.0),
    "one pass fewer": lambda c, w: c["loop"].update(times=1),
    "embedding not joined": lambda c, w: w["loop.in"][:, 112:].zero_(),
    "residual multiplier": lambda c, w: c.update(residual_mult=0.65),
    "embedding scale": lambda c, w: c["embedding"].update(scale=0.75),
    "one expert fewer": lambda c, w: c["layers"][0]["mlp"]["router"].update(top=1),
    "shared gate": lambda c, w: w["l1.mlp.shared.sg"].zero_(),
}


@pytest.mark.parametrize("name", MISTAKES)
def test_planted_mistakes_show(case, reference, name):
    """The oracle with one mistake is far from the framework, so the same mistake in the framework would be seen."""
    cfg, w, path = case
    t = reference[0]["e"]
    got = C.run(_llm(path).engine, {"x": t}, [[("x", n)] for n in C.cut(90, [31, 2, 1])])["x"]
    assert C.error(got, reference[1]["e"]) < EXACT
    c, wm = copy.deepcopy(cfg), {n: v.clone() for n, v in w.items()}
    MISTAKES[name](c, wm)
    assert C.error(got, O.forward(c, wm, t)) > SHOWS


def test_lost_states_and_far_tokens_show(case, reference):
    """What the first tokens leave in keys and states reaches the last logits: changing or dropping them shows there."""
    cfg, w, _ = case
    t, want = reference[0]["a"], reference[1]["a"]
    changed = O.forward(cfg, w, [(t[0] + 1) % V] + t[1:])
    assert C.error(changed[-20:], want[-20:]) > 10 * EXACT


@pytest.mark.parametrize("cfg,rows", [
    (C.config([C.delta(None, 1, 1, 6, 8, 1), C.delta(C.moe(2, 1, 8, 16), 6, 2, 40, 12, 4)], width=96, loop=(0, 2, 3)), 16),
    (C.config([C.parallel(C.moe(3, 3, 16, 24), 1, 1, 8, 40, 1, 1.3, 9, 0.0, 1, 17), C.parallel(None, 5, 5, 12, 7, 5, 0.7, 30.5, 1.0, 3, 200)], vocab=77, width=101,
              eps=1e-3, loop=(1, 2, 1)), 6),
    (C.config([C.parallel(None, 8, 2, 20, 12, 8, 0.2, 2000, 0.1, 7, 33), C.delta(C.moe(9, 4, 12, 30), 4, 4, 16, 16, 8)], width=81, mult=1.0, scale=1.0, loop=None), 32),
])
def test_other_sizes(tmp_path, cfg, rows):
    w = C.weights(cfg, seed=11, rows=rows)
    t = C.tokens(60, cfg["vocab"], 7)
    got = C.run(_llm(C.save(tmp_path, cfg, w)).engine, {"x": t}, [[("x", n)] for n in C.cut(60, [23, 1, 2])])["x"]
    assert C.error(got, O.forward(cfg, w, t)) < EXACT


def test_bfloat16_stays_near_the_oracle(case, reference):
    seqs, want = reference
    got = C.run(_llm(case[2], dtype=torch.bfloat16).engine, {"e": seqs["e"]}, [[("e", n)] for n in C.cut(90, [50, 1, 2])])["e"]
    assert C.error(got, want["e"]) < 0.08


# ----------------------------------------------------------------------------------- entry points
def greedy(cfg, w, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(O.forward(cfg, w, t)[-1].argmax()))
    return t[len(prompt):]


def test_greedy_generation_through_the_scheduler(case):
    cfg, w, path = case
    prompts = [C.tokens(n, V, 20 + n) for n in (50, 3, 21)]
    want = [greedy(cfg, w, p, 8) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    llm = _llm(path, chunk=16, enable_prefix_caching=True)
    assert [o.token_ids for o in llm.generate(prompts, sp)] == want
    again = llm.generate(prompts, sp)                     # the longest prompt's pages and state come from the prefix cache
    assert [o.token_ids for o in again] == want and again[0].cached_tokens >= 32
    spec = _llm(path, spec_method="ngram", max_draft=3)
    rep = [C.tokens(6, V, 5) * 6]
    assert spec.generate(rep, sp)[0].token_ids == greedy(cfg, w, rep[0], 8)


def test_rejected_rows_leave_no_trace(case, reference):
    seqs = {i: reference[0][i] for i in ("b", "c")}
    got = verify_with_rejected_rows(_llm(case[2]).engine, seqs)
    for i in seqs:
        assert C.error(got[i], reference[1][i]) < EXACT, i


def test_preempted_requests_resume(case):
    cfg, w, path = case
    prompts = [C.tokens(40, V, 30 + i) for i in range(4)]
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    llm = _llm(path, kv_tokens=144)                       # holds about three of the four
    assert [o.token_ids for o in llm.generate(prompts, sp)] == [greedy(cfg, w, p, 6) for p in prompts]


def test_command_line_generates_and_scores(case, capsys):
    from blaze_b200 import cli
    cfg, w, path = case
    t = C.tokens(9, V, 3)
    flags = ["--model", path, "--device", "cpu", "--max-model-len", "64", "--max-seqs", "2", "--kv-tokens", "128", "--kv-cache-dtype", "bf16",
             "--prompt-ids", ",".join(map(str, t))]
    assert cli.main(["generate", "--max-tokens", "4"] + flags) == 0
    assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["token_ids"]) == 4
    assert cli.main(["score"] + flags) == 0
    got = json.loads(capsys.readouterr().out.strip().splitlines()[-1])["logprobs"]
    lp = torch.log_softmax(O.forward(cfg, w, t), -1)
    assert np.allclose(got, [float(lp[i, t[i + 1]]) for i in range(8)], atol=0.2)
    assert cli.main(["inspect", "--model", path]) == 0


def test_random_weights_of_the_named_shape():
    llm = LLM(named_config("tiny-medodra"), device="cpu", kv_tokens=256, max_seqs=2, max_model_len=64)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.8, seed=1, max_tokens=5, ignore_eos=True))[0]
    assert len(out.token_ids) == 5 and llm.model.weight_bytes() > 0


def test_trace_replay_writes_the_wanted_logits(case, reference, tmp_path):
    _, _, path = case
    seqs, want = reference
    a, b = seqs["a"][:70], seqs["c"]
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": a[:30], "want": [29, 4]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": b, "want": []}, {"id": "p", "tokens": a[30:31], "want": []}], "end": ["q"]},
             {"step": 2, "entries": [{"id": "r", "tokens": b[:2], "want": [1]}, {"id": "p", "tokens": a[31:], "want": [0, 38]}], "end": ["p", "r"]}]
    r = subprocess.run([sys.executable, "bin/trace_run", "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128",
                        "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    rows = [np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, V) for n in (0, 2)]
    assert not (tmp_path / "1.f32").exists()
    assert C.error(torch.from_numpy(rows[0]), want["a"][[29, 4]]) < EXACT
    assert C.error(torch.from_numpy(rows[1]), torch.stack([want["c"][1], want["a"][31], want["a"][69]])) < EXACT
