"""The Rapisun design on the oracle op set: every mechanism and the whole model against the independent restatement in
``oracle_rapisun.py``, through the package's loader, cache, engine, scheduler and command line."""
import copy
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import oracle_rapisun as O
import rapisun_case as C
from blaze_b200.config import GatedLinearSpec, LatentAttnSpec, ModelConfig, MoeSpec, PolyNormSpec, RotarySpec, named_config
from blaze_b200.llm import LLM
from blaze_b200.models import model_class
from blaze_b200.ops import ref
from blaze_b200.ops.ref_ops import RefOps
from blaze_b200.sampler import SamplingParams
from test_niletar_cpu import verify_with_rejected_rows
from test_sevevik_cpu import ROOT, SCHEDULES, mixed_steps

EXACT = 1e-4            # fp32 rounding through these random models; a wrong key, state or constant gives 1e-2 and more
SHOWS = 1e-2


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
    return cfg, w, C.save(tmp_path_factory.mktemp("rapisun"), cfg, w)


def rand(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ----------------------------------------------------------------------------------- configuration and loading
def test_configuration_is_read_layer_by_layer():
    cfg = ModelConfig.from_json(C.config())
    assert cfg.architecture == "Rapisun" and model_class(cfg).__name__ == "Rapisun" and cfg.input_conv == 4 and cfg.rms_norm_eps == 1e-5
    assert cfg.layer_specs[0].attn == LatentAttnSpec(4, 24, 8, 40, 36, 48, 0.3, RotarySpec(8, 500.0, False), True, 20)
    assert cfg.layer_specs[0].mlp == PolyNormSpec(88) and cfg.layer_specs[1].rec == GatedLinearSpec(3, 20, 28)
    assert cfg.layer_specs[1].mlp == MoeSpec(6, 2, 40, 56) and cfg.layer_specs[4].mlp == MoeSpec(6, 3, 40, 0)
    assert cfg.layer_specs[3].attn.kv_from == 2 and cfg.layer_specs[3].mlp is None
    assert [cfg.layer_type(i) for i in (0, 1)] == ["latent_attention", "gated_linear"]
    assert ModelConfig.from_json(C.config([C.latent(window=None)])).layer_specs[0].attn.window == 0


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), lambda c: c["layers"][3]["mixer"].update(kv_from=4),
    lambda c: c["layers"][3]["mixer"].update(kv_from=1), lambda c: c["layers"][5]["mixer"].update(kv_from=3),
    lambda c: c["layers"][3]["mixer"].update(kv_rank=32), lambda c: c["layers"][3]["mixer"]["rot"].update(base=9.0),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7), lambda c: c["layers"][0]["mlp"].update(kind="glu"),
    lambda c: c["layers"][1]["mixer"].update(heads=0), lambda c: c["canon"].update(taps=-1), lambda c: c.update(layers=[])])
def test_configurations_that_make_no_model_are_refused(change):
    c = copy.deepcopy(C.config())
    change(c)
    with pytest.raises(ValueError):
        ModelConfig.from_json(c)


def test_tensors_of_the_wrong_shape_are_refused(tmp_path, case):
    cfg, w, _ = case
    for name in ("l0.mix.dkv", "l1.mix.lower", "l1.mlp.e5.up", "l3.mix.uk", "l0.mlp.act"):
        with pytest.raises(ValueError, match="asks for"):
            _llm(C.save(tmp_path, cfg, dict(w, **{name: w[name][:-1]})))


def test_pages_and_states_follow_each_layers_sizes(case):
    llm = _llm(case[2])
    kv = llm.engine.kv
    assert kv.k[0].shape[1:] == (1, 16, 48) and kv.v[0].shape[1:] == (1, 16, 8) and kv.k[2].shape[1:] == (1, 16, 64) and sorted(kv.k) == [0, 2, 3, 5]
    assert kv.k[3] is kv.k[2] and kv.v[5] is kv.v[0]                  # a layer that reads another's latents keeps none
    assert kv.rec_state[1].shape[1:] == (3, 20, 28) and kv.rec_state[1].dtype == torch.float32 and not kv.conv_state
    assert all(kv.input_state[i].shape[1:] == (3, 144) and kv.input_state[i].dtype == torch.float32 for i in range(6))
    assert kv.state_layers == list(range(6))
    per_page = 16 * 4 * (48 + 8 + 64 + 16) * kv.num_pages
    assert kv.nbytes() == per_page + kv.state_rows * 4 * (3 * 20 * 28 + 2 * 32 * 16 + 6 * 3 * 144)
    assert llm.model.weight_bytes() > sum(t.numel() * 4 for n, t in case[1].items() if n.endswith((".o", ".up", ".down", ".uq", ".uk", ".uv")))


def test_what_the_design_does_not_have_is_refused(case):
    with pytest.raises(ValueError, match="bf16 or fp32"):
        _llm(case[2], kv_cache_dtype="fp8")
    with pytest.raises(ValueError, match="dense"):
        LLM("tiny-rapisun", device="cpu", weight_format="nvfp4")
    with pytest.raises(ValueError, match="drafters"):
        _llm(case[2], spec_method="mtp")


# ----------------------------------------------------------------------------------- mechanisms alone
def test_norms():
    x, y, w = rand(5, 24), rand(5, 24, seed=1) + 3, rand(24, seed=2)
    got, h = RefOps().branch_norm(x, y.bfloat16(), w, 1e-2)
    assert torch.allclose(got.double(), x.double() + O.layer_norm(y.bfloat16().double(), w.double(), 1e-2), atol=1e-5) and h.dtype == torch.bfloat16
    rows = torch.tensor([3, 0])
    assert torch.allclose(RefOps().norm_rows(x, rows, w, 1e-2, torch.float32, centre=True).double(), O.layer_norm(x[rows].double(), w.double(), 1e-2), atol=1e-6)
    o, g = rand(4, 21), rand(7, seed=3)
    assert torch.allclose(ref.group_norm(o, None, g, 3, 1e-2, False, False).double(), (O.rms(o.double().view(4, 3, 7), 1e-2) * g.double()).view(4, 21), atol=1e-5)


def test_input_convolution_keeps_its_history():
    for taps in (1, 2, 4, 7):
        x, w = rand(30, 12), rand(12, taps, seed=1)
        st, out = torch.zeros(taps - 1, 12), []
        for n in (1, 2, 9, 1, 17):
            y, st = ref.input_conv(x[sum(map(len, out)):][:n], st, w.t())
            out.append(y)
        assert st.shape == (taps - 1, 12) and torch.allclose(torch.cat(out).double(), O.input_conv(x.double(), w.double()), atol=1e-5)


def test_gated_linear_attention_in_portions():
    T, H, d, e = 40, 3, 12, 10
    q, f, v, lo, b = rand(T, H, d), rand(T, H, d, seed=1) * 3, rand(T, H, e, seed=2), torch.sigmoid(rand(H * d, seed=3)), rand(H * d, seed=4) + 1
    S, outs = torch.zeros(H, d, e), []
    for i, n in ((0, 1), (1, 2), (3, 20), (23, 17)):
        s = slice(i, i + n)
        o, S = ref.gated_linear(q[s], f[s], v[s], lo, b, S)
        outs.append(o)
    gate = O.forget_gate(f.double() + b.double().view(H, d), lo.double().view(H, d))
    for h in range(H):
        want = O.gated_linear(O.silu(q[:, h].double()), gate[:, h], v[:, h].double())
        assert torch.allclose(torch.cat(outs)[:, h].double(), want, atol=1e-5)


@pytest.mark.parametrize("rot", [{"dims": 16, "base": 500.0}, {"dims": 6, "base": 1e5}, {"dims": 2, "base": 10.0}])
def test_rotation_of_half_vectors(rot):
    from blaze_b200.config import _rotary
    x = rand(50, 3, 16)
    got = ref.rotate_heads(x, torch.arange(50), torch.tensor(_rotary(rot).frequencies(), dtype=torch.float64), False)
    assert torch.allclose(got.double(), O.rotate_half(x.double(), rot["dims"], rot["base"]), atol=1e-5)


def test_sink_and_window_edges():
    """One key stands out: it shows while it is inside the window, not one token later; the sink takes its share once."""
    n, d, win, sink = 60, 8, 17, torch.tensor([2.0])
    q, k, v = rand(n, d), rand(n, d, seed=1) * 0.1, rand(n, d, seed=2)
    k[20] = 4 * torch.ones(d)
    q[36] = q[37] = torch.ones(d)
    pages = lambda t: torch.cat([t, t.new_zeros(4, d)]).view(4, 1, 16, d)      # noqa: E731
    got = ref.paged_attention(q[:, None], pages(k), pages(v), torch.arange(4).view(1, 4), [0], [0, n], [n], 0.5, window=win, sink=sink)[:, 0]
    want = O.sink_window_attention(q.double(), k.double(), v.double(), 0.5, win, sink[0].double())
    assert torch.allclose(got.double(), want, atol=1e-5)
    assert (want[36] - v[20].double()).abs().max() < 0.01 and (want[37] - v[20].double()).abs().max() > 0.3
    other = O.sink_window_attention(q.double(), k.double(), v.double(), 0.5, win, torch.tensor(-100.0).double())
    assert (other - want).abs().max() > 0.05


def test_activations_and_routing():
    z, act = rand(6, 30) * 2, torch.tensor([0.7, -0.4, 1.3, 0.25])
    assert torch.allclose(ref.poly_norm(z, act, 1e-2).double(), O.poly_norm(z.double(), act.double(), 1e-2), atol=1e-5)
    assert torch.allclose(ref.relu2(z).double(), O.squared_relu(z.double()), atol=1e-6)
    w, ids = ref.router_topk(z, 5)
    best, weight = O.route(z.double(), 5)
    assert torch.equal(ids.long(), best) and torch.allclose(w.double(), weight, atol=1e-6) and torch.allclose(w.sum(1), torch.ones(6))


# ----------------------------------------------------------------------------------- the whole model
@pytest.fixture(scope="module")
def reference(case):
    cfg, w, _ = case
    seqs = {"a": C.tokens(150, 320, 1), "b": C.tokens(67, 320, 2), "c": C.tokens(33, 320, 3), "d": C.tokens(1, 320, 4), "e": C.tokens(90, 320, 5)}
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


def windows(c, k):
    return [L["mixer"]["mask"].update(size=L["mixer"]["mask"]["size"] + k) for L in c["layers"] if L["type"] == "latent_attention"]


MISTAKES = {
    "sink left out": lambda c, w: [w[f"l{i}.mix.sink"].fill_(-40) for i in (0, 2, 3, 5)],
    "windows one short": lambda c, w: windows(c, -1),
    "windows one long": lambda c, w: windows(c, 1),
    "rotation left out": lambda c, w: [c["layers"][i]["mixer"]["rot"].update(dims=0) for i in (0, 2, 3, 5)],
    "latents of its own": lambda c, w: w.update({"l5.mix.dkv": w["l0.mix.dkv"], "l5.mix.dkv.norm": w["l0.mix.dkv.norm"]}) or c["layers"][5]["mixer"].pop("kv_from"),
    "oldest tap left out": lambda c, w: [w[f"l{i}.canon1"][:, 0].zero_() for i in range(6)],
    "no lower bound": lambda c, w: w["l1.mix.lower"].zero_(),
    "gate bias left out": lambda c, w: w["l1.mix.f.b"].zero_(),
    "a constant for another": lambda c, w: w["l0.mlp.act"].copy_(w["l0.mlp.act"][[1, 0, 2, 3]]),
    "one expert fewer": lambda c, w: c["layers"][1]["mlp"]["router"].update(top=1),
    "no shared expert": lambda c, w: c["layers"][1]["mlp"].update(shared=None),
    "embedding norm left out": lambda c, w: w["embed.norm"].fill_(1.0),
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
    """What the first tokens leave in the states reaches the last logits: changing or dropping them shows there."""
    cfg, w, _ = case
    t, want = reference[0]["a"], reference[1]["a"]
    dropped = O.forward(cfg, w, t[60:])
    assert C.error(dropped[-40:], want[-40:]) > SHOWS
    changed = O.forward(cfg, w, [(t[0] + 1) % 320] + t[1:])
    assert C.error(changed[-20:], want[-20:]) > EXACT


@pytest.mark.parametrize("cfg", [
    C.config([C.hgrn2(None, 1, 3, 8), C.hgrn2(C.moe(2, 1, 8, 0), 6, 40, 12)], width=96, taps=1),
    C.config([C.latent(C.dense(40), None, None, 1, 8, 2, 8, 5, 7, 1.3, 100.0), C.latent(C.moe(3, 3, 16, 24), 0, 1, 2, 8, 2, 6, 9, 7, 0.7, 100.0)], vocab=77, width=100,
             eps=1e-3, taps=2),
    C.config([C.latent(None, None, 5, 6, 10, 6, 6, 20, 30), C.hgrn2(C.dense(33), 2, 16, 16), C.latent(C.moe(9, 4, 12, 30), 0, 64, 2, 10, 6, 50, 64, 30)], width=81, taps=9),
])
def test_other_sizes(tmp_path, cfg):
    w = C.weights(cfg, seed=11)
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
    prompts = [C.tokens(n, 320, 20 + n) for n in (50, 3, 21)]
    want = [greedy(cfg, w, p, 8) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    llm = _llm(path, chunk=16, enable_prefix_caching=True)
    assert [o.token_ids for o in llm.generate(prompts, sp)] == want
    again = llm.generate(prompts, sp)                     # the longest prompt's pages and state come from the prefix cache
    assert [o.token_ids for o in again] == want and again[0].cached_tokens >= 32
    spec = _llm(path, spec_method="ngram", max_draft=3)
    rep = [C.tokens(6, 320, 5) * 6]
    assert spec.generate(rep, sp)[0].token_ids == greedy(cfg, w, rep[0], 8)


def test_rejected_rows_leave_no_trace(case, reference):
    seqs = {i: reference[0][i] for i in ("b", "c")}
    got = verify_with_rejected_rows(_llm(case[2]).engine, seqs)
    for i in seqs:
        assert C.error(got[i], reference[1][i]) < EXACT, i


def test_preempted_requests_resume(case):
    cfg, w, path = case
    prompts = [C.tokens(40, 320, 30 + i) for i in range(4)]
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    llm = _llm(path, kv_tokens=144)                       # holds about three of the four
    assert [o.token_ids for o in llm.generate(prompts, sp)] == [greedy(cfg, w, p, 6) for p in prompts]


def test_command_line_generates_and_scores(case, capsys):
    from blaze_b200 import cli
    cfg, w, path = case
    t = C.tokens(9, 320, 3)
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
    llm = LLM(named_config("tiny-rapisun"), device="cpu", kv_tokens=256, max_seqs=2, max_model_len=64)
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
    rows = [np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, 320) for n in (0, 2)]
    assert not (tmp_path / "1.f32").exists()
    assert C.error(torch.from_numpy(rows[0]), want["a"][[29, 4]]) < EXACT
    assert C.error(torch.from_numpy(rows[1]), torch.stack([want["c"][1], want["a"][31], want["a"][69]])) < EXACT
