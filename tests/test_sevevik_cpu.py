"""The Sevevik design on the oracle op set: every mechanism and the whole model against the independent restatement in
``oracle_sevevik.py``, through the package's loader, cache, engine, scheduler and command line."""
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import oracle_sevevik as O
import sevevik_case as C
from blaze_b200.config import ModelConfig, named_config
from blaze_b200.llm import LLM
from blaze_b200.models import model_class
from blaze_b200.sampler import SamplingParams

EXACT = 2e-4            # fp32 rounding through these sharp random models; a wrong key or window gives 2e-2 and more


def _llm(path, dtype=torch.float32, **kw):
    kw = {"kv_tokens": 1024, "max_seqs": 4, "max_model_len": 512, "enable_prefix_caching": False, **kw}
    return LLM(path, device="cpu", dtype=dtype, **kw)


@pytest.fixture(scope="module")
def case(tmp_path_factory):
    cfg = C.config()
    w = C.weights(cfg, seed=3)
    path = C.save(tmp_path_factory.mktemp("sevevik"), cfg, w)
    return cfg, w, path


# ----------------------------------------------------------------------------------- configuration and loading
def test_configuration_is_read_layer_by_layer():
    cfg = ModelConfig.from_json(C.config())
    assert cfg.architecture == "Sevevik" and model_class(cfg).__name__ == "Sevevik"
    a, b = cfg.layer_specs[0].attn, cfg.layer_specs[1].attn
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.group) == (4, 2, 24, 40, 20, 2)
    assert (b.heads, b.kv_heads, b.window) == (3, 1, 33) and cfg.layer_specs[1].mlp is None
    assert cfg.layer_specs[2].weights_of == 0 and cfg.streams == 3 and cfg.embed_scale == 3.0 and cfg.residual_mult == 0.6
    assert model_class(named_config("tiny")).__name__ == "Model"


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="recurrent"), lambda c: c["layers"][0]["mixer"].update(heads=5),
                                    lambda c: c["layers"][2].update(weights_of=2), lambda c: c["layers"][2]["mixer"].update(diff=0.1),
                                    lambda c: c["layers"][0]["mlp"].update(kind="experts"), lambda c: c.update(layers=[])])
def test_configurations_that_make_no_model_are_refused(change):
    c = C.config(json.loads(json.dumps(C.config()["layers"])))
    change(c)
    with pytest.raises(ValueError):
        ModelConfig.from_json(c)


def test_a_tensor_of_the_wrong_shape_is_refused(tmp_path, case):
    cfg, w, _ = case
    bad = dict(w, **{"l0.mix.k": w["l0.mix.k"][:-1]})
    with pytest.raises(ValueError, match="l0.mix.k"):
        _llm(C.save(tmp_path, cfg, bad))


def test_pages_follow_each_layers_sizes(case):
    llm = _llm(case[2])
    kv = llm.engine.kv
    assert kv.k[0].shape[1:] == (4, 16, 24) and kv.v[0].shape[1:] == (2, 16, 40)
    assert kv.k[1].shape[1:] == (2, 16, 16) and kv.v[3].shape[1:] == (2, 16, 16)
    m = llm.model
    assert m.layers[2] is m.layers[0] and 2 in kv.k and kv.k[2] is not kv.k[0]     # shared tensors, a cache of its own


def test_fp8_pages_and_quantised_weights_are_refused(case):
    with pytest.raises(ValueError, match="bf16 or fp32"):
        _llm(case[2], kv_cache_dtype="fp8")
    with pytest.raises(ValueError, match="dense"):
        LLM("tiny-sevevik", device="cpu", weight_format="nvfp4")
    with pytest.raises(ValueError, match="drafters"):
        _llm(case[2], spec_method="mtp")


# ----------------------------------------------------------------------------------- mechanisms alone
def test_clamped_glu_reaches_both_clamps():
    from blaze_b200.ops import ref
    g = torch.tensor([[-9.0, -1.0, 0.3, 2.0, 9.0]])
    u = torch.tensor([[-9.0, 1.0, -0.3, 0.9, 9.0]])
    got = ref.clamped_glu(torch.cat([g, u], 1), 1.25)
    want = O.clamped_glu(g.double(), u.double(), 1.25)
    assert torch.allclose(got.double(), want, atol=1e-6)
    assert not torch.allclose(want[0, 4], O.clamped_glu(g.double(), u.double(), 20.0)[0, 4])


def test_streams_are_rewritten_from_the_old_ones():
    from blaze_b200.ops import ref
    gen = torch.Generator().manual_seed(1)
    x, y = torch.randn(5, 3, 8, generator=gen), torch.randn(5, 8, generator=gen)
    mix, out = torch.randn(3, 3, generator=gen), torch.randn(3, generator=gen)
    got = ref.streams_write(x, mix, out * 0.7, y)
    want = O.write_streams(x.transpose(0, 1).double(), mix.double(), out.double(), y.double(), 0.7).transpose(0, 1)
    assert torch.allclose(got.double(), want, atol=1e-5)


def test_map_weight_is_a_difference_of_exponentials():
    from blaze_b200.models.qwen3 import DiffAttn
    v = [torch.randn(24, generator=torch.Generator().manual_seed(i)) * 0.5 for i in range(4)]
    assert abs(DiffAttn.map_weight(*v, 0.45) - O.mix_weight(*[x.double() for x in v], 0.45)) < 1e-9


# ----------------------------------------------------------------------------------- the whole model
@pytest.fixture(scope="module")
def reference(case):
    cfg, w, _ = case
    seqs = {"a": C.tokens(150, 320, 1), "b": C.tokens(67, 320, 2), "c": C.tokens(33, 320, 3), "d": C.tokens(1, 320, 4), "e": C.tokens(90, 320, 5)}
    return seqs, {i: O.forward(cfg, w, t) for i, t in seqs.items()}


SCHEDULES = {
    "whole": lambda n: [n], "pairs": lambda n: C.cut(n, [2]), "mixed": lambda n: C.cut(n, [37, 2, 3, 17, 1, 64]),
    "page": lambda n: C.cut(n, [16]), "decode": lambda n: [min(n, 40)] + [1] * max(n - 40, 0), "all one": lambda n: [1] * n,
}


@pytest.mark.parametrize("name", SCHEDULES)
def test_logits_do_not_depend_on_how_a_prompt_is_cut(case, reference, name):
    seqs, want = reference
    eng = _llm(case[2]).engine
    for i, t in seqs.items():
        got = C.run(eng, {i: t}, [[(i, n)] for n in SCHEDULES[name](len(t))])[i]
        assert C.error(got, want[i]) < EXACT, i


def mixed_steps(seqs):
    """Portions of some beside single tokens of others; requests come and go so that rows and pages are used again."""
    left = {i: len(t) for i, t in seqs.items()}
    size = {"a": [29, 1, 1, 40, 2], "b": [1, 33, 2], "c": [2, 5, 1], "d": [1], "e": [64, 1]}
    steps, k, live = [], 0, []
    while any(left.values()):
        live = [i for i in live if left[i]] + [i for i in seqs if left[i] and i not in live]
        live = live[:3]
        step = []
        for j, i in enumerate(live):
            if (k + j) % 5 == 4 and len(live) > 1:
                continue                                   # this one sits a step out
            n = min(size[i][k % len(size[i])], left[i])
            step.append((i, n))
            left[i] -= n
        steps.append(step)
        k += 1
    return steps


def test_batches_of_unequal_requests_match_each_alone(case, reference):
    seqs, want = reference
    eng = _llm(case[2], kv_tokens=320).engine              # less than the sum of the requests: pages are used again
    for _ in range(2):
        got = C.run(eng, seqs, mixed_steps(seqs))
        for i in seqs:
            assert C.error(got[i], want[i]) < EXACT, i
    assert eng.pages.free_count == eng.num_pages - 1


def test_planted_window_edges_show(case):
    """The oracle with a window one longer or shorter is far from the framework, so a window off by one would be seen."""
    cfg, w, path = case
    t = C.tokens(80, 320, 9)
    got = C.run(_llm(path).engine, {"x": t}, [[("x", n)] for n in C.cut(80, [31, 2, 1])])["x"]
    assert C.error(got, O.forward(cfg, w, t)) < EXACT
    for off in (-1, 1):
        c = json.loads(json.dumps(cfg))
        for L in c["layers"]:
            L["mixer"]["mask"]["size"] += off
        assert C.error(got, O.forward(c, w, t)) > 0.02
    # nor may the layer on another's tensors be left out
    c = dict(cfg, layers=[cfg["layers"][i] for i in (0, 1, 3)])
    w3 = {**w, **{n.replace("l3.", "l2."): v for n, v in w.items() if n.startswith("l3.")}}
    assert C.error(got, O.forward(c, w3, t)) > 0.02


@pytest.mark.parametrize("cfg", [
    C.config([C.layer(heads=1, kv_heads=1, dim=8, vdim=8, window=1), C.layer(heads=6, kv_heads=2, dim=20, vdim=12, window=300)], streams=1, mult=1.0),
    C.config([C.layer(heads=2, kv_heads=1, window=16, ff=80, limit=7.0)], streams=5, width=100, vocab=77, eps=1e-3, embed=1.0),
    C.config([C.layer(window=None), C.layer(weights_of=0, window=None), C.layer(weights_of=0, window=None)], streams=2),
])
def test_other_sizes(tmp_path, cfg):
    w = C.weights(cfg, seed=11)
    path = C.save(tmp_path, cfg, w)
    t = C.tokens(60, cfg["vocab"], 7)
    got = C.run(_llm(path).engine, {"x": t}, [[("x", n)] for n in C.cut(60, [23, 1, 2])])["x"]
    assert C.error(got, O.forward(cfg, w, t)) < EXACT


def test_bfloat16_stays_near_the_oracle(tmp_path):
    cfg = C.config()
    w = C.weights(cfg, seed=5, sharp=1.0)
    t = C.tokens(100, 320, 8)
    got = C.run(_llm(C.save(tmp_path, cfg, w), dtype=torch.bfloat16).engine, {"a": t}, [[("a", n)] for n in C.cut(100, [50, 1, 2])])["a"]
    assert C.error(got, O.forward(cfg, w, t)) < 0.06


# ----------------------------------------------------------------------------------- entry points
def greedy(cfg, w, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(O.forward(cfg, w, t)[-1].argmax()))
    return t[len(prompt):]


def test_greedy_generation_through_the_scheduler(case):
    cfg, w, path = case
    prompts = [C.tokens(n, 320, 20 + n) for n in (50, 3, 21)]
    want = [greedy(cfg, w, p, 12) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    llm = _llm(path, chunk=16, enable_prefix_caching=True)
    assert [o.token_ids for o in llm.generate(prompts, sp)] == want
    again = llm.generate(prompts, sp)                     # the longest prompt's pages come from the prefix cache
    assert [o.token_ids for o in again] == want and again[0].cached_tokens >= 32
    spec = _llm(path, spec_method="ngram", max_draft=3, draft_tree_width=2)       # chains only: the design verifies no trees
    rep = [C.tokens(6, 320, 5) * 6]
    assert spec.generate(rep, sp)[0].token_ids == greedy(cfg, w, rep[0], 12)


def test_preempted_requests_resume(case):
    cfg, w, path = case
    prompts = [C.tokens(40, 320, 30 + i) for i in range(4)]
    sp = SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True)
    llm = _llm(path, kv_tokens=160)                       # holds about three of the four
    assert [o.token_ids for o in llm.generate(prompts, sp)] == [greedy(cfg, w, p, 10) for p in prompts]


def test_command_line_generates_and_scores(case, capsys):
    from blaze_b200 import cli
    cfg, w, path = case
    t = C.tokens(9, 320, 3)
    flags = ["--model", path, "--device", "cpu", "--max-model-len", "64", "--max-seqs", "2", "--kv-tokens", "128", "--kv-cache-dtype", "bf16",
             "--prompt-ids", ",".join(map(str, t))]
    assert cli.main(["generate", "--max-tokens", "4"] + flags) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert len(out["token_ids"]) == 4
    assert cli.main(["score"] + flags) == 0
    got = json.loads(capsys.readouterr().out.strip().splitlines()[-1])["logprobs"]
    lp = torch.log_softmax(O.forward(cfg, w, t), -1)
    assert np.allclose(got, [float(lp[i, t[i + 1]]) for i in range(8)], atol=0.15)
    assert cli.main(["inspect", "--model", path]) == 0


def test_random_weights_of_the_named_shape():
    llm = LLM("tiny-sevevik", device="cpu", kv_tokens=256, max_seqs=2, max_model_len=64)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))[0]
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
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    rows = [np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, 320) for n in (0, 2)]
    assert not (tmp_path / "1.f32").exists()
    assert C.error(torch.from_numpy(rows[0]), want["a"][[29, 4]]) < EXACT
    assert C.error(torch.from_numpy(rows[1]), torch.stack([want["c"][1], want["a"][31], want["a"][69]])) < EXACT


ROOT = __file__.rsplit("/tests/", 1)[0]
