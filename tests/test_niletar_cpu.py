"""The Niletar design on the oracle op set: every mechanism and the whole model against the independent restatement in
``oracle_niletar.py``, through the package's loader, cache, engine, scheduler and command line."""
import copy
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import niletar_case as C
import oracle_niletar as O
from blaze_b200.config import ModelConfig, RotarySpec, named_config
from blaze_b200.llm import LLM
from blaze_b200.models import model_class
from blaze_b200.ops import ref
from blaze_b200.sampler import SamplingParams
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
    return cfg, w, C.save(tmp_path_factory.mktemp("niletar"), cfg, w)


# ----------------------------------------------------------------------------------- configuration and loading
def test_configuration_is_read_layer_by_layer():
    cfg = ModelConfig.from_json(C.config())
    assert cfg.architecture == "Niletar" and model_class(cfg).__name__ == "Niletar" and cfg.residual_alpha == 1.7
    a, r = cfg.layer_specs[0].attn, cfg.layer_specs[0].rec
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.out_scale, a.group) == (4, 2, 24, 40, 0.35, 0.7, 2)
    assert a.rot == RotarySpec(16, 2000.0, True, 6.0, 1.0, 4.0, 96.0) and cfg.layer_specs[3].attn.rot.original == 0
    assert (r.heads, r.kv_heads, r.dim, r.vdim, r.conv, r.out_scale) == (6, 3, 20, 28, 3, 0.45)
    m = cfg.layer_specs[1]
    assert m.attn is None and (m.rec.heads, m.rec.vdim, m.rec.state, m.rec.groups, m.rec.norm_groups, m.rec.conv) == (4, 24, 20, 2, 3, 4)
    assert cfg.layer_specs[2].weights_of == 1 and cfg.layer_specs[3].mlp is None
    assert [cfg.layer_type(i) for i in (0, 1)] == ["soft_attention+delta_rule", "state_space"]


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][0]["mixer"]["left"].update(heads=5),
    lambda c: c["layers"][0]["mixer"]["right"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"].update(norm_groups=5),
    lambda c: c["layers"][1]["mixer"].update(groups=3), lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26),
    lambda c: c["layers"][2].update(weights_of=2), lambda c: c["layers"][2]["mixer"].update(state=24),
    lambda c: c["layers"][0]["mlp"].update(kind="experts"), lambda c: c.update(layers=[])])
def test_configurations_that_make_no_model_are_refused(change):
    c = copy.deepcopy(C.config())
    change(c)
    with pytest.raises(ValueError):
        ModelConfig.from_json(c)


def test_tensors_of_the_wrong_shape_are_refused(tmp_path, case):
    cfg, w, _ = case
    for name in ("l0.mix.left.k", "l1.mix.conv.b", "l0.mix.right.g2"):
        with pytest.raises(ValueError, match="mix"):
            _llm(C.save(tmp_path, cfg, dict(w, **{name: w[name][:, :-1] if name.endswith("g2") else w[name][:-1]})))


def test_pages_and_states_follow_each_layers_sizes(case):
    llm = _llm(case[2])
    kv, m = llm.engine.kv, llm.model
    assert kv.k[0].shape[1:] == (2, 16, 24) and kv.v[0].shape[1:] == (2, 16, 40) and sorted(kv.k) == [0, 3, 4]
    assert kv.rec_state[0].shape[1:] == (6, 20, 28) and kv.conv_state[0].shape[1:] == (2 * 60 + 168, 2)
    assert kv.rec_state[1].shape[1:] == (4, 20, 24) and kv.conv_state[1].shape[1:] == (96 + 80, 3)
    assert kv.rec_state[1].dtype == torch.float32 and kv.state_layers == [0, 1, 2, 3, 4]
    assert m.layers[2] is m.layers[1] and kv.rec_state[2] is not kv.rec_state[1] and kv.k[4] is not kv.k[0]
    assert m.weight_bytes() > sum(t.numel() * 4 for n, t in case[1].items() if n.endswith((".o", ".in", ".down")))


def test_what_the_design_does_not_have_is_refused(case):
    with pytest.raises(ValueError, match="bf16 or fp32"):
        _llm(case[2], kv_cache_dtype="fp8")
    with pytest.raises(ValueError, match="dense"):
        LLM("tiny-niletar", device="cpu", weight_format="nvfp4")
    with pytest.raises(ValueError, match="drafters"):
        _llm(case[2], spec_method="mtp")


# ----------------------------------------------------------------------------------- mechanisms alone
def rand(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


@pytest.mark.parametrize("rot", [{"dims": 16, "base": 500.0}, {"dims": 20, "base": 1e4, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}},
                                 {"dims": 8, "base": 300.0, "scaling": {"factor": 2.5, "low": 0.5, "high": 6.0, "original": 40}}])
def test_rotation_and_its_frequencies(rot):
    from blaze_b200.config import _rotary
    r = _rotary(rot)
    assert np.allclose(r.frequencies(), O.rotary_frequencies(rot), rtol=1e-12)
    if "scaling" in rot:                 # all three branches occur: kept, blended, slowed down by the whole factor
        ratio = np.array(r.frequencies()) / np.array(_rotary({k: v for k, v in rot.items() if k != "scaling"}).frequencies())
        f = 1 / rot["scaling"]["factor"]
        assert ratio.min() == pytest.approx(f) and ratio.max() == 1 and ((ratio > f * 1.001) & (ratio < 0.999)).any()
    x = rand(50, 3, 24)
    got = ref.rotate_heads(x, torch.arange(50), torch.tensor(r.frequencies(), dtype=torch.float64), True)
    assert torch.allclose(got.double(), O.rotate(x.double(), rot), atol=1e-5)
    half = ref.rotate_heads(x, torch.arange(50), torch.tensor(r.frequencies(), dtype=torch.float64), False)
    n = rot["dims"] // 2
    mixed = torch.cat([torch.stack([x[..., :n], x[..., n:2 * n]], -1).flatten(-2), x[..., 2 * n:]], -1)
    turned = O.rotate(mixed.double(), rot)
    assert torch.allclose(half[..., :n].double(), turned[..., 0:2 * n:2], atol=1e-5) and torch.allclose(half[..., n:2 * n].double(), turned[..., 1:2 * n:2], atol=1e-5)


def test_short_convolution_keeps_its_history():
    for taps in (1, 2, 3, 4, 7):
        x, w, b = rand(30, 12), rand(12, taps, seed=1), rand(12, seed=2)
        want = O.silu(O.short_conv(x.double(), w.double(), b.double()))
        st, out = torch.zeros(12, taps - 1), []
        for n in (1, 2, 9, 1, 17):
            y, st = ref.gdn_conv(x[sum(map(len, out)):][:n], st, w, b, round_sum=False)
            out.append(y)
        assert torch.allclose(torch.cat(out).double(), want, atol=1e-5)


def test_recurrences_in_portions():
    T, H, G, d, e = 40, 6, 2, 12, 10
    q, k, v, a, b = rand(T, G, d), rand(T, G, d, seed=1), rand(T, H, e, seed=2), rand(T, H, d, seed=3), rand(T, H, seed=4)
    A, bias = torch.rand(H) * 3 + 0.1, rand(H * d, seed=5) - 2
    S, outs = torch.zeros(H, d, e), []
    for i, n in ((0, 1), (1, 2), (3, 20), (23, 17)):
        s = slice(i, i + n)
        o, S = ref.delta_rule(q[s], k[s], v[s], a[s], b[s], A, bias, S)
        outs.append(o)
    got = torch.cat(outs).double()
    g = torch.exp(-A.double()[:, None] * O.softplus(a.double() + bias.double().view(H, d)))
    for h in range(H):
        want = O.delta_rule(O.unit(q[:, h // 3].double()) / d ** 0.5, O.unit(k[:, h // 3].double()), v[:, h].double(), g[:, h], O.sigmoid(b[:, h].double()))
        assert torch.allclose(got[:, h], want, atol=1e-5)
    N = 14
    x, B, Cm, dt, D = rand(T, H, e), rand(T, G, N, seed=6), rand(T, G, N, seed=7), rand(T, H, seed=8), rand(H, seed=9)
    S, outs, db = torch.zeros(H, N, e), [], rand(H, seed=10)
    for i, n in ((0, 3), (3, 1), (4, 36)):
        s = slice(i, i + n)
        o, S = ref.state_space(x[s], B[s], Cm[s], dt[s], A, db, D, S)
        outs.append(o)
    got, step = torch.cat(outs).double(), O.softplus(dt.double() + db.double())
    for h in range(H):
        want = O.state_space(x[:, h].double(), B[:, h // 3].double(), Cm[:, h // 3].double(), step[:, h], torch.exp(-A[h].double() * step[:, h]), float(D[h]))
        assert torch.allclose(got[:, h], want, atol=1e-4)


def test_gated_norms_and_the_residual():
    o, z, w = rand(5, 24), rand(5, 24, seed=1), rand(24, seed=2)
    want = O.rms((o * O.silu(z)).double().view(5, 3, 8), 1e-3).view(5, 24) * w.double()
    assert torch.allclose(ref.group_norm(o, z, w, 3, 1e-3, False, True).double(), want, atol=1e-5)
    want = 0.3 * (O.rms(o.double().view(5, 4, 6), 1e-3) * w[:6].double()).view(5, 24) * O.sigmoid(z.double())
    assert torch.allclose(ref.group_norm(o, z, w[:6], 4, 1e-3, True, False, 0.3).double(), want, atol=1e-5)
    from blaze_b200.ops.ref_ops import RefOps
    x, h = RefOps().residual_norm(o, 2.2, z.bfloat16(), 1 + w, 1e-3)
    assert torch.allclose(x.double(), O.centred_norm(2.2 * o.double() + z.bfloat16().double(), w.double(), 1e-3), atol=1e-5) and h.dtype == torch.bfloat16


def test_sink_takes_its_share_of_the_softmax():
    q, k, v, sink = rand(20, 2, 8), rand(2, 2, 16, 8, seed=1), rand(2, 2, 16, 6, seed=2), torch.tensor([3.0, -1.0])
    table = torch.tensor([[1, 0]], dtype=torch.int32)
    got = ref.paged_attention(q, k, v, table, [0], [0, 20], [20], 0.4, sink=sink)
    flat = lambda t, h: torch.cat([t[1, h], t[0, h]])[:20].double()      # noqa: E731
    for h in range(2):
        args = (q[:, h].double(), flat(k, h), flat(v, h), 0.4)
        assert torch.allclose(got[:, h].double(), O.sink_attention(*args, sink[h].double()), atol=1e-5)
        assert (got[:, h].double() - O.sink_attention(*args, torch.tensor(-100.0).double())).abs().max() > 0.05


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


MISTAKES = {
    "sink left out": lambda c, w: [w[f"l{i}.mix.left.sink"].fill_(-40) for i in (0, 3)],
    "bias left out": lambda c, w: w["l0.mix.left.v.b"].zero_(),
    "rotation one dimension short": lambda c, w: [L["mixer"]["left"]["rot"].update(dims=L["mixer"]["left"]["rot"]["dims"] - 2) for L in c["layers"] if L["type"] == "parallel"],
    "no frequency scaling": lambda c, w: [c["layers"][i]["mixer"]["left"]["rot"].pop("scaling", None) for i in (0, 4)],
    "left and right scales swapped": lambda c, w: [L["mixer"].update(left_scale=L["mixer"]["right_scale"], right_scale=L["mixer"]["left_scale"]) for L in c["layers"] if L["type"] == "parallel"],
    "one norm group": lambda c, w: [c["layers"][i]["mixer"].update(norm_groups=1) for i in (1, 2)],
    "skip term left out": lambda c, w: w["l1.mix.D"].zero_(),
    "oldest tap left out": lambda c, w: w["l1.mix.conv"][:, 0].zero_(),
    "alpha of one": lambda c, w: c.update(postln_alpha=1.0),
    "a shared layer left out": lambda c, w: c["layers"].pop(2) and [w.update({n.replace("l3.", "l2."): v for n, v in w.items() if n.startswith("l3.")})],
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
    """What the first tokens leave in the states and pages reaches the last logits: changing or dropping them shows there."""
    cfg, w, _ = case
    t, want = reference[0]["a"], reference[1]["a"]
    dropped = O.forward(cfg, w, t[60:])
    assert C.error(dropped[-40:], want[-40:]) > SHOWS
    changed = O.forward(cfg, w, [(t[0] + 1) % 320] + t[1:])
    assert C.error(changed[-20:], want[-20:]) > 10 * EXACT


@pytest.mark.parametrize("cfg", [
    C.config([C.mamba(heads=1, vdim=8, state=3, groups=1, norm_groups=1, conv=1), C.mamba(heads=6, vdim=12, state=40, groups=6, norm_groups=9, conv=2)], width=96),
    C.config([C.parallel(left={"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.3}, rot={"dims": 8, "base": 100.0},
                         right={"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 40, "conv": 5}, left_scale=1.0, right_scale=1.0)], alpha=1.0, vocab=77, width=100, eps=1e-3),
    C.config([C.parallel(left={"heads": 6, "kv_heads": 6, "dim": 10, "vdim": 6}, rot={"dims": 2, "base": 10.0},
                         right={"heads": 8, "kv_heads": 2, "dim": 40, "vdim": 4, "conv": 4}), C.mamba(), C.parallel(weights_of=0, left={"heads": 6, "kv_heads": 6, "dim": 10, "vdim": 6},
                         rot={"dims": 2, "base": 10.0}, right={"heads": 8, "kv_heads": 2, "dim": 40, "vdim": 4, "conv": 4}), C.mamba(weights_of=1)], width=80),
])
def test_other_sizes(tmp_path, cfg):
    w = C.weights(cfg, seed=11, ranks=(17, 3))
    t = C.tokens(60, cfg["vocab"], 7)
    got = C.run(_llm(C.save(tmp_path, cfg, w)).engine, {"x": t}, [[("x", n)] for n in C.cut(60, [23, 1, 2])])["x"]
    assert C.error(got, O.forward(cfg, w, t)) < EXACT


def test_bfloat16_stays_near_the_oracle(case, reference):
    seqs, want = reference
    got = C.run(_llm(case[2], dtype=torch.bfloat16).engine, {"e": seqs["e"]}, [[("e", n)] for n in C.cut(90, [50, 1, 2])])["e"]
    assert C.error(got, want["e"]) < 0.05


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


def verify_with_rejected_rows(eng, seqs):
    """Steps whose last rows are wrong guesses: their state is deferred, the right rows are replayed and the rest is dropped.
    Returns the logits of all right rows."""
    live, out = {i: eng.open_from() for i in seqs}, {i: [] for i in seqs}
    k = 0
    while live:
        items, keep = [], {}
        for i in list(live):
            n0 = live[i].length
            right = seqs[i][n0:n0 + (2 + (k + len(i)) % 3 if n0 else 20)]
            wrong = [(t + 7) % 300 for t in right[:k % 3]]
            items.append((live[i], right + wrong, len(right) + len(wrong)))
            keep[i] = (n0, len(right), len(wrong))
        got = eng.forward(eng.plan(items, defer_state=True), "logits").float().cpu()
        eng.commit_state([(live[i], keep[i][1]) for i in live])
        r = 0
        for i in list(live):
            n0, a, b = keep[i]
            out[i].append(got[r:r + a])
            r += a + b
            eng.truncate(live[i], n0 + a)
            if n0 + a == len(seqs[i]):
                eng.close(live.pop(i))
        k += 1
    return {i: torch.cat(o) for i, o in out.items()}


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
    assert np.allclose(got, [float(lp[i, t[i + 1]]) for i in range(8)], atol=0.15)
    assert cli.main(["inspect", "--model", path]) == 0


def test_random_weights_of_the_named_shape():
    llm = LLM(named_config("tiny-niletar"), device="cpu", kv_tokens=256, max_seqs=2, max_model_len=64)
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
