"""The Sevevik design's kernels on a B200 against the independent restatement in ``oracle_sevevik.py``: each mechanism alone over
many sizes, then whole models in bf16 and fp32 through the engine and the scheduler."""
import pytest
import torch

import oracle_sevevik as O
import sevevik_case as C

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def ops():
    from blaze_b200.ops import get_ops
    return get_ops(DEV)


def rel(got, want):
    return float((got.double().cpu() - want.double().cpu()).abs().max() / want.double().abs().max().cpu())


# ----------------------------------------------------------------------------------- streams, norms, products
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S,W,T", [(1, 64, 3), (2, 100, 5), (3, 257, 4), (4, 512, 37), (6, 96, 2), (12, 48, 3), (4, 4096, 2)])
def test_streams(ops, S, W, T, dtype):
    from blaze_b200.models.sevevik import StaticStreams
    g = torch.Generator().manual_seed(S * W)
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    table, tok = r(40, W).to(dtype), torch.randint(0, 40, (T,), generator=g)
    a, b = [(r(S), r(S, S), r(S)) for _ in range(2)]
    wa, wb = [StaticStreams(*x, 0.6, DEV, dtype) for x in (a, b)]
    na, nb = r(W), r(W)
    y1, y2 = r(T, W).to(dtype), r(T, W).to(dtype)
    xs = (table[tok].double() * 1.7)[None].repeat(S, 1, 1)
    tol = 1e-5 if dtype == torch.float32 else 8e-3
    src = ops.streams_begin(table.to(DEV), tok.to(DEV, torch.int32), 1.7, S)
    src, h = ops.streams_step(src, None, None, wa, na.to(DEV), 1e-5)
    assert rel(h, O.rms(O.read_streams(xs, a[0].double()), 1e-5, na.double())) < tol
    src, h = ops.streams_step(src, y1.to(DEV), wa, wb, nb.to(DEV), 1e-5)
    xs = O.write_streams(xs, a[1].double(), a[2].double(), y1.double(), 0.6)
    assert rel(h, O.rms(O.read_streams(xs, b[0].double()), 1e-5, nb.double())) < tol
    assert rel(src, xs.transpose(0, 1)) < 1e-5                  # the streams themselves are fp32 in either type
    src, h = ops.streams_step(src, y2.to(DEV), wb, wa, na.to(DEV), 1e-5)
    xs = O.write_streams(xs, b[1].double(), b[2].double(), y2.double(), 0.6)
    assert rel(h, O.rms(O.read_streams(xs, a[0].double()), 1e-5, na.double())) < tol
    total = ops.streams_sum(src, y1.to(DEV), wa)
    xs = O.write_streams(xs, a[1].double(), a[2].double(), y1.double(), 0.6)
    assert rel(total, xs.sum(0)) < 1e-5
    rows = torch.tensor([T - 1, 0, 0], device=DEV)
    assert rel(ops.norm_rows(total, rows, nb.to(DEV), 1e-5, dtype), O.rms(xs.sum(0), 1e-5, nb.double())[[T - 1, 0, 0]]) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,I,K", [(1, 96, 64), (5, 40, 100), (70, 512, 256), (300, 1024, 512), (3, 33, 24), (1, 16384, 2048), (200, 1024, 8192)])
def test_clamped_glu(ops, T, I, K, dtype):
    from blaze_b200.linear import Linear
    g = torch.Generator().manual_seed(I)
    w = (torch.randn(2 * I, K, generator=g) * 2.0 * K ** -0.5).to(dtype)
    x = torch.randn(T, K, generator=g).to(dtype)
    lin = Linear.from_dense(w.to(DEV), dtype=dtype)
    got = ops.linear_glu(lin, x.to(DEV), 1.3)
    y = x.double() @ w.double().T
    assert got.shape == (T, I) and rel(got, O.clamped_glu(y[:, :I], y[:, I:], 1.3)) < ((1e-5 if K < 4096 else 5e-5) if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("M,N,K", [(1, 7, 5), (65, 130, 33), (200, 64, 96)])
def test_products_in_true_32_bit(ops, M, N, K):
    from blaze_b200.linear import Linear
    g = torch.Generator().manual_seed(N)
    x, w = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g)
    lin = Linear.from_dense(w.to(DEV), dtype=torch.float32)
    want = x.double() @ w.double().T
    assert rel(ops.linear(lin, x.to(DEV)), want) < 2e-6
    assert torch.equal(ops.linear_argmax(lin, x.to(DEV)).cpu(), ops.linear(lin, x.to(DEV)).argmax(1).cpu())
    odd = Linear.from_dense(w.to(DEV), dtype=torch.bfloat16)              # a row length that the TMA kernels do not take
    if K % 16:
        assert rel(ops.linear(odd, x.to(DEV).bfloat16(), out_dtype=torch.float32), x.bfloat16().double() @ w.bfloat16().double().T) < 1e-5


# ----------------------------------------------------------------------------------- attention alone
class _Layer:
    def __init__(self, spec, lam):
        self.spec, self.lam = spec, lam


class _Paged:
    """One attention layer over paged keys and values, fed rows of q | k | v."""

    def __init__(self, ops, spec, dtype, pages=400, seqs=8, eps=1e-5):
        from blaze_b200.config import LayerSpec, ModelConfig
        from blaze_b200.engine import PageAllocator
        from blaze_b200.kv import KVCache
        self.ops, self.spec, self.eps = ops, spec, eps
        cfg = ModelConfig.of_layers([LayerSpec(spec)], architecture="Sevevik")
        self.kv = KVCache(cfg, pages, seqs, 256, "fp32" if dtype == torch.float32 else "bf16", DEV, "tiles")
        self.alloc, self.len, self.pages = PageAllocator(pages), {}, {}
        self.layer = _Layer(spec, 0.55)

    def step(self, entries):
        """entries: (slot, rows [n, width]) -> the outputs, one tensor per entry."""
        from blaze_b200.batch import SeqChunk, build_batch
        chunks = []
        for slot, rows in entries:
            n0, n = self.len.get(slot, 0), rows.shape[0]
            have = self.pages.setdefault(slot, [])
            need = (n0 + n + 15) // 16 - len(have)
            if need > 0:
                new = self.alloc.alloc(need)
                self.kv.set_pages(slot, new, len(have))
                have.extend(new)
            chunks.append(SeqChunk(slot, [0] * n, n0))
            self.len[slot] = n0 + n
        batch = build_batch(chunks, self.kv.block_table_host, DEV)
        out = self.ops.diff_attention(torch.cat([r for _, r in entries]).to(DEV), self.layer, batch, self.kv, 0, self.eps).cpu()
        assert self.ops.take_status() == 0
        return torch.split(out, [r.shape[0] for _, r in entries])

    def free(self, slot):
        self.alloc.release(self.pages.pop(slot))
        del self.len[slot]


def rows_of(spec, n, seed, dtype, plant=()):
    """Random q | k | v rows.  ``plant``: (query, key, map) places whose score is made to stand out, in every head."""
    H, G, d, e = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(n, H, 2, d, generator=g), torch.randn(n, G, 2, d, generator=g), torch.randn(n, G, e, generator=g)
    for i, j, m in plant:
        if 0 <= i < n and 0 <= j < n:
            u = torch.randn(d, generator=g)
            u = u / u.norm() * (30.0 / spec.scale) ** 0.5           # a score of about 30 among scores of order 1
            q[i, :, m], k[j, :, m] = u, u
    return torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], 1).to(dtype)


def attend(spec, rows, lam, eps):
    """The oracle's output for whole sequences of such rows (the output projection left out)."""
    H, G, d, e = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    n = rows.shape[0]
    q, k, v = torch.split(rows.double(), [H * 2 * d, G * 2 * d, G * e], 1)
    q, k, v = q.reshape(n, H, 2, d), k.reshape(n, G, 2, d), v.reshape(n, G, e)
    w = spec.window or None
    out = []
    for h in range(H):
        a = [O.window_attention(q[:, h, m], k[:, h // (H // G), m], v[:, h // (H // G)], spec.scale, w) for m in (0, 1)]
        out.append(O.rms(a[0] - lam * a[1], eps) * (1 - spec.diff))
    return torch.cat(out, 1)


def spec(heads, kv_heads, dim, vdim, window, scale=None, diff=0.3):
    from blaze_b200.config import DiffAttnSpec
    return DiffAttnSpec(heads, kv_heads, dim, vdim, scale or dim ** -0.5, diff, window)


SPECS = [(5, 5, 32, 64, 100), (4, 1, 16, 16, 24), (6, 2, 48, 80, 50), (8, 2, 64, 128, 200), (8, 1, 128, 128, 129), (4, 2, 40, 24, 33),
         (2, 2, 20, 36, 0), (3, 1, 64, 32, 1), (5, 1, 24, 120, 2), (2, 1, 144, 136, 40), (16, 1, 32, 32, 0), (40, 1, 16, 48, 90)]
PORTIONS = {"whole": [10 ** 6], "pairs and more": [2, 37, 3, 130, 1], "decode": [150, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1]}


@pytest.mark.parametrize("portions", PORTIONS)
@pytest.mark.parametrize("case", SPECS)
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_attention_windows_and_far_keys(ops, case, portions, dtype):
    s = spec(*case)
    n = 216
    w = s.window or n
    edges = [p for p in (15, 16, 63, 64, 127, 128, 150, 151, 155, 159, 160, 161, 167, 168, 200, 215)]
    # keys just inside and just outside the window, on either map, and far ones at page borders
    plant = [(i, i - w + 1 - (k % 2), k // 2 % 2) for k, i in enumerate(edges)] + [(i, (i - min(w, i) + 16) // 16 * 16, 1) for i in (100, 140, 190)]
    rows = rows_of(s, n, 7 + sum(case), dtype, plant)
    at = _Paged(ops, s, dtype)
    out, pos = [], 0
    for c in C.cut(n, PORTIONS[portions]):
        out.append(at.step([(0, rows[pos:pos + c])])[0])
        pos += c
    want = attend(s, rows, 0.55, 1e-5)
    got = torch.cat(out)
    err = (got.double() - want).abs().amax(1) / want.abs().max()
    limit = 2e-2 if dtype == torch.bfloat16 else 2e-4
    assert err.max() < limit, (int(err.argmax()), float(err.max()))
    assert err.mean() < limit / 5


@pytest.mark.parametrize("case", [(8, 2, 64, 128, 70), (3, 3, 32, 64, 0), (6, 2, 40, 24, 33)])
def test_attention_batches_of_unequal_sequences(ops, case):
    """Long portions, short portions and single rows in one step; a freed sequence's pages serve the next one."""
    s = spec(*case)
    lens = {0: 300, 1: 41, 2: 160, 3: 7, 4: 1, 5: 90}
    rows = {b: rows_of(s, n, 50 + b, torch.bfloat16, [(n - 1, max(n - (s.window or n), 0), b % 2)]) for b, n in lens.items()}
    want = {b: attend(s, r, 0.55, 1e-5) for b, r in rows.items()}
    at = _Paged(ops, s, torch.bfloat16, pages=50)
    got, pos = {b: [] for b in lens}, {b: 0 for b in lens}
    sizes = {0: [120, 1, 1, 50, 2, 3, 100], 1: [5, 1, 33, 1], 2: [1, 129, 1], 3: [2], 4: [1], 5: [64, 1]}
    k = 0
    while any(pos[b] < lens[b] for b in lens):
        step = []
        for b in lens:
            if pos[b] < lens[b] and not (b in (2, 5) and k < 3):             # two join later, in pages of those that have ended
                c = min(sizes[b][k % len(sizes[b])], lens[b] - pos[b])
                step.append((b, rows[b][pos[b]:pos[b] + c]))
        for (b, r), o in zip(step, at.step(step)):
            got[b].append(o)
            pos[b] += r.shape[0]
            if pos[b] == lens[b]:
                at.free(b)
        k += 1
    for b in lens:
        g = torch.cat(got[b]).double()
        assert (g - want[b]).abs().max() / want[b].abs().max() < 2e-2, b


def test_long_context_is_split_over_blocks(ops):
    s = spec(8, 2, 64, 96, 0)
    n = 1500
    rows = rows_of(s, n, 3, torch.bfloat16, [(n - 1, 5, 0), (n - 2, 700, 1), (n - 3, 0, 0)])
    at = _Paged(ops, s, torch.bfloat16)
    at.step([(0, rows[:n - 4])])
    got = torch.cat([at.step([(0, rows[i:i + 1])])[0] for i in range(n - 4, n)])
    H, G, d, e = 8, 2, 64, 96
    q, k, v = torch.split(rows.double(), [H * 2 * d, G * 2 * d, G * e], 1)
    for r in range(4):
        i = n - 4 + r
        want = []
        for h in range(H):
            a = []
            for m in (0, 1):
                sc = k.reshape(n, G, 2, d)[:i + 1, h // 4, m] @ q.reshape(n, H, 2, d)[i, h, m] * s.scale
                a.append(torch.softmax(sc, 0) @ v.reshape(n, G, e)[:i + 1, h // 4])
            want.append(O.rms(a[0] - 0.55 * a[1], 1e-5) * 0.7)
        want = torch.cat(want)
        assert (got[r].double() - want).abs().max() / want.abs().max() < 2e-2, r


# ----------------------------------------------------------------------------------- whole models
CONFIGS = {
    "mixed layers": C.config(),
    "wider": C.config([C.layer(heads=8, kv_heads=2, dim=64, vdim=128, window=70, ff=512, limit=3.0, scale=0.125),
                       C.layer(heads=4, kv_heads=4, dim=32, vdim=48, window=40, ff=512, limit=3.0),
                       C.layer(weights_of=1, heads=4, kv_heads=4, dim=32, vdim=48, window=40, ff=512, limit=3.0)], width=512, vocab=1000, streams=4),
    "ragged": C.config([C.layer(heads=3, kv_heads=3, dim=12, vdim=20, window=17, ff=72), C.layer(heads=2, kv_heads=1, dim=8, vdim=28, window=None, ff=None)],
                       width=100, vocab=77, streams=1, mult=1.0),
}


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_model_in_every_schedule(tmp_path, name, dtype):
    from blaze_b200.llm import LLM
    from test_sevevik_cpu import SCHEDULES, mixed_steps
    cfg = CONFIGS[name]
    w = C.weights(cfg, seed=2, sharp=1.0)
    V = cfg["vocab"]
    seqs = {"a": C.tokens(150, V, 1), "b": C.tokens(67, V, 2), "c": C.tokens(33, V, 3), "d": C.tokens(1, V, 4), "e": C.tokens(90, V, 5)}
    want = {i: O.forward(cfg, w, t) for i, t in seqs.items()}
    llm = LLM(C.save(tmp_path, cfg, w), device=DEV, dtype=dtype, kv_tokens=336, max_seqs=4, max_model_len=512, enable_prefix_caching=False)
    assert llm.model.ops.is_cuda and llm.engine.kv.layout == "tiles"
    limit = 1e-4 if dtype == torch.float32 else 0.06
    for sched, f in SCHEDULES.items():
        got = C.run(llm.engine, {"a": seqs["a"]}, [[("a", n)] for n in f(150)])["a"]
        assert C.error(got, want["a"]) < limit, sched
    for _ in range(2):
        got = C.run(llm.engine, seqs, mixed_steps(seqs))
        for i in seqs:
            assert C.error(got[i], want[i]) < limit, i


@pytest.mark.parametrize("graphs", [True, False])
def test_generation_follows_the_logits(tmp_path, graphs):
    """Greedy generation through the scheduler (captured decode steps, prefix cache, speculation): every chosen token is the best
    one of the oracle's logits for that context, up to bf16 rounding."""
    from blaze_b200.llm import LLM
    from blaze_b200.sampler import SamplingParams
    cfg = CONFIGS["wider"]
    w = C.weights(cfg, seed=6, sharp=1.0)
    path = C.save(tmp_path, cfg, w)
    prompts = [C.tokens(n, 1000, 40 + n) for n in (90, 5, 33, 64)]
    sp = SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True)
    for kw in ({}, {"spec_method": "ngram", "max_draft": 3}):
        llm = LLM(path, device=DEV, kv_tokens=2048, max_seqs=4, max_model_len=256, chunk=64, use_graphs=graphs, **kw)
        for outs in (llm.generate(prompts, sp), llm.generate(prompts, sp)):
            for p, o in zip(prompts, outs):
                t = p + o.token_ids
                lg = O.forward(cfg, w, t[:-1], dtype=torch.float32)[len(p) - 1:]
                chosen = lg[torch.arange(len(o.token_ids)), torch.tensor(o.token_ids)]
                assert len(o.token_ids) == 40 and float((lg.max(1).values - chosen).max()) < 0.1 * float(lg.std())
        assert bool(llm.engine._graphs) == graphs


def test_32_bit_generation_is_the_oracles(tmp_path):
    from blaze_b200.llm import LLM
    from blaze_b200.sampler import SamplingParams
    cfg = CONFIGS["mixed layers"]
    w = C.weights(cfg, seed=9, sharp=1.0)
    prompts = [C.tokens(n, 320, 60 + n) for n in (40, 7)]
    llm = LLM(C.save(tmp_path, cfg, w), device=DEV, dtype=torch.float32, kv_tokens=512, max_seqs=2, max_model_len=128)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        t = list(p)
        for _ in range(24):
            t.append(int(O.forward(cfg, w, t)[-1].argmax()))
        assert o.token_ids == t[len(p):]


def test_other_models_refuse_32_bit_kernels():
    from blaze_b200.llm import LLM
    with pytest.raises(ValueError, match="do not run in"):
        LLM("tiny", device=DEV, dtype=torch.float32, kv_tokens=256, max_seqs=2, max_model_len=64)
