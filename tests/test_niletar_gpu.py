"""The Niletar design's kernels on a B200 against the independent restatement in ``oracle_niletar.py``: each mechanism alone over
many sizes, then whole models in bf16 and fp32 through the engine and the scheduler."""
import pytest
import torch

import niletar_case as C
import oracle_niletar as O
from test_sevevik_cpu import SCHEDULES, mixed_steps

pytestmark = pytest.mark.gpu
DEV = "cuda"
TYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def ops():
    from blaze_b200.ops import get_ops
    return get_ops(DEV)


def rel(got, want):
    return float((got.double().cpu() - want.double().cpu()).abs().max() / want.double().abs().max().cpu())


class Sequences:
    """State rows, pages and batches of one mixer fed by hand: ``step`` runs portions of several sequences."""

    def __init__(self, spec, dtype, pages=420, seqs=8):
        from blaze_b200.config import ModelConfig
        from blaze_b200.engine import PageAllocator
        from blaze_b200.kv import KVCache
        cfg = ModelConfig.of_layers([spec], architecture="Niletar")
        self.kv = KVCache(cfg, pages, seqs, 256, "fp32" if dtype == torch.float32 else "bf16", DEV, "tiles")
        for t in list(self.kv.rec_state.values()) + list(self.kv.conv_state.values()):
            t.fill_(3.0)                       # what an earlier sequence may have left: a fresh one must not see it
        self.alloc, self.len, self.pages = PageAllocator(pages), {}, {}

    def batch(self, entries, defer=()):
        """entries: (slot, rows)"""
        from blaze_b200.batch import SeqChunk, build_batch
        chunks = []
        for slot, n in entries:
            n0 = self.len.get(slot, 0)
            have = self.pages.setdefault(slot, [])
            need = (n0 + n + 15) // 16 - len(have)
            if need > 0:
                new = self.alloc.alloc(need)
                self.kv.set_pages(slot, new, len(have))
                have.extend(new)
            chunks.append(SeqChunk(slot, [0] * n, n0, defer_state=slot in defer))
            if slot not in defer:
                self.len[slot] = n0 + n
        return build_batch(chunks, self.kv.block_table_host, DEV)

    def free(self, slot):
        self.alloc.release(self.pages.pop(slot))
        del self.len[slot]


def schedule(lens, sizes, late=()):
    """Steps of (sequence, count); the late ones join after three steps."""
    pos, k = {b: 0 for b in lens}, 0
    while any(pos[b] < lens[b] for b in lens):
        step = []
        for b in lens:
            if pos[b] < lens[b] and not (b in late and k < 3):
                n = min(sizes[b][k % len(sizes[b])], lens[b] - pos[b])
                step.append((b, pos[b], n))
                pos[b] += n
        if step:
            yield step
        k += 1


LENS = {0: 300, 1: 41, 2: 160, 3: 7, 4: 1, 5: 90}
SIZES = {0: [120, 1, 1, 50, 2, 3, 100], 1: [5, 1, 33, 1], 2: [1, 129, 1], 3: [2], 4: [1], 5: [64, 1]}


# ----------------------------------------------------------------------------------- residual, norms, products
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("T,W", [(1, 64), (5, 100), (3, 257), (37, 512), (2, 4096), (300, 2048)])
def test_residual_norm(ops, T, W, dtype):
    g = torch.Generator().manual_seed(W)
    x, y1, y2, w = [torch.randn(*s, generator=g) for s in ((T, W), (T, W), (T, W), (W,))]
    x, y1, y2 = x.to(dtype), y1.to(dtype), y2.to(dtype)
    want = O.centred_norm(1.7 * x.double() + y1.double(), w.double(), 1e-5)
    r, h = ops.residual_norm(x.to(DEV), 1.7, y1.to(DEV), (1 + w).to(DEV), 1e-5)
    assert r.dtype == torch.float32 and h.dtype == dtype and rel(r, want) < 1e-6 and rel(h, want) < (1e-6 if dtype == torch.float32 else 8e-3)
    r, h = ops.residual_norm(r, 1.7, y2.to(DEV), (1 + w).to(DEV), 1e-5)
    assert rel(r, O.centred_norm(1.7 * want + y2.double(), w.double(), 1e-5)) < 2e-6


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("T,I,K", [(1, 96, 64), (5, 40, 100), (70, 512, 256), (3, 33, 24), (200, 1024, 512)])
def test_gated_feed_forward(ops, T, I, K, dtype):
    from blaze_b200.linear import Linear
    g = torch.Generator().manual_seed(I)
    w, x = (torch.randn(2 * I, K, generator=g) * 2.0 * K ** -0.5).to(dtype), torch.randn(T, K, generator=g).to(dtype)
    y = x.double() @ w.double().T
    got = ops.linear_swiglu(Linear.from_dense(w.to(DEV), dtype=dtype), x.to(DEV))
    assert got.shape == (T, I) and rel(got, O.silu(y[:, :I]) * y[:, I:]) < (1e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("dtype", TYPES)
def test_products_with_biases_and_of_some_columns(ops, dtype):
    from blaze_b200.linear import Linear
    g = torch.Generator().manual_seed(1)
    for M, N, K, off, wide in ((3, 72, 48, 16, 200), (300, 264, 96, 8, 120), (2, 1000, 512, 64, 640), (130, 40, 20, 3, 31)):
        x, w, b = [torch.randn(*s, generator=g).to(dtype) for s in ((M, wide), (N, K), (N,))]
        lin = Linear.from_dense(w.to(DEV), dtype=dtype)
        lin.bias = b.to(DEV)
        want = x[:, off:off + K].double() @ w.double().T + b.double()
        assert rel(ops.linear(lin, x.to(DEV)[:, off:off + K], out_dtype=torch.float32), want) < (1e-5 if dtype == torch.float32 else 2e-3)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("T,groups,n,period,first", [(3, 4, 24, 96, True), (5, 7, 20, 20, False), (2, 1, 4096, 4096, True), (9, 3, 33, 33, False),
                                                     (40, 16, 128, 128, False), (1, 2, 1000, 2000, True), (300, 8, 256, 2048, True), (2, 3, 5000, 15000, True)])
def test_group_norm(ops, T, groups, n, period, first, dtype):
    from blaze_b200.ops.cuda_ops import VP, _ptr
    g = torch.Generator().manual_seed(n)
    C_ = groups * n
    o, z, w = torch.randn(T, C_, generator=g), torch.randn(T, C_ + 24, generator=g).to(dtype), torch.randn(period, generator=g)
    for off in (8, 3):
        od, wd, zz, out = o.to(DEV), w.to(DEV), z.to(DEV), torch.zeros(T, C_ + 16, dtype=dtype, device=DEV)
        sig = not first
        ops._check(ops.lib.blz_group_norm(_ptr(od), VP(zz.data_ptr() + off * zz.element_size()), zz.stride(0), _ptr(wd),
                                          VP(out.data_ptr() + 8 * out.element_size()), out.stride(0), T, groups, n, period, 1e-4, 0.6, int(sig), int(first),
                                          int(dtype == torch.float32), ops._stream()), "group_norm")
        zd = z[:, off:off + C_].double()
        gate = O.sigmoid(zd) if sig else O.silu(zd)
        x = o.double() * gate if first else o.double()
        x = O.rms(x.view(T, groups, n), 1e-4).view(T, C_) * w.double().repeat(C_ // period)
        want = 0.6 * (x if first else x * gate)
        assert rel(out[:, 8:8 + C_], want) < (2e-6 if dtype == torch.float32 else 8e-3)
        assert float(out[:, :8].abs().max()) == 0 and float(out[:, 8 + C_:].abs().max()) == 0


# ----------------------------------------------------------------------------------- convolution and recurrences
def mixer_of(kind, spec, dtype, seed=0):
    """A mixer's recurrent part with random constants (no projections)."""
    from blaze_b200.models.qwen3 import Mixer, Recurrence
    g = torch.Generator().manual_seed(seed)
    R = Recurrence(spec, kind, 1)
    R.conv_w = torch.randn(spec.conv_dim, spec.conv, generator=g).to(DEV, dtype)
    R.conv_b = torch.randn(spec.conv_dim, generator=g).to(DEV) if kind == "ssm" else None
    n = spec.heads * (spec.dim if kind == "delta" else 1)
    R.A = (torch.rand(spec.heads, generator=g) * 3 + 0.05).to(DEV)
    R.dt_bias, R.D = (torch.randn(n, generator=g) - 2.5).to(DEV), torch.randn(spec.heads, generator=g).to(DEV)
    M = Mixer()
    M.rec = R
    return M


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("taps,channels", [(1, 40), (2, 33), (3, 300), (4, 128), (6, 65), (8, 16)])
def test_short_convolution(ops, taps, channels, dtype):
    from blaze_b200.config import LayerSpec, StateSpaceSpec
    spec = StateSpaceSpec(heads=1, vdim=channels - 2, state=1, groups=1, norm_groups=1, conv=taps)
    M = mixer_of("ssm", spec, dtype)
    M.cols = {"conv": 3}
    S = Sequences(LayerSpec(rec=spec), dtype)
    g = torch.Generator().manual_seed(channels)
    x = {b: torch.randn(n, channels + 5, generator=g).to(dtype) for b, n in LENS.items()}
    want = {b: O.silu(O.short_conv(x[b][:, 3:3 + channels].double(), M.rec.conv_w.double().cpu(), M.rec.conv_b.double().cpu())) for b in x}
    got = {b: [] for b in LENS}
    for step in schedule(LENS, SIZES, late=(2, 5)):
        batch = S.batch([(b, n) for b, _, n in step])
        out = ops.short_conv(torch.cat([x[b][p:p + n] for b, p, n in step]).to(DEV), M, batch, S.kv, 0).cpu()
        for (b, _, _), o in zip(step, out.split([n for _, _, n in step])):
            got[b].append(o)
    for b in LENS:
        assert rel(torch.cat(got[b]), want[b]) < (3e-6 if dtype == torch.float32 else 8e-3), b


DELTAS = [(2, 2, 20, 28), (6, 3, 32, 16), (4, 1, 64, 64), (3, 3, 128, 128), (8, 2, 96, 40), (2, 1, 160, 24), (1, 1, 300, 9), (4, 2, 8, 200)]
SPACES = [(4, 24, 20, 2), (6, 32, 64, 3), (4, 64, 128, 1), (8, 48, 16, 8), (2, 130, 96, 1), (3, 20, 200, 3), (2, 7, 400, 1)]


def run_recurrence(ops, kind, spec, dtype, lens, sizes, late=()):
    """(outputs, what the oracle gives) of every sequence; q, k, v or x, B, C come after the convolution here."""
    from blaze_b200.config import LayerSpec
    M = mixer_of(kind, spec, dtype)
    M.cols = {"beta": 5, "dt": 5}
    S = Sequences(LayerSpec(rec=spec), dtype)
    g = torch.Generator().manual_seed(spec.state)
    H, e, N = spec.heads, spec.vdim, spec.state
    y = {b: torch.randn(n, spec.conv_dim, generator=g).to(dtype) for b, n in lens.items()}
    proj = {b: (torch.randn(n, H + 9, generator=g) * 1.5).to(dtype) for b, n in lens.items()}
    low = {b: torch.randn(n, H * N + 4, generator=g).to(dtype) for b, n in lens.items()}
    got = {b: [] for b in lens}
    for k, step in enumerate(schedule(lens, sizes, late)):
        cat = lambda d: torch.cat([d[b][p:p + n] for b, p, n in step]).to(DEV)        # noqa: E731
        T = sum(n for _, _, n in step)
        out = torch.full((T, H * e), float("nan"), device=DEV)
        ents = [(b, n) for b, _, n in step]
        if k % 2:                            # the same rows once more with the state kept as it was
            before = {b: S.len.get(b, 0) for b, _ in ents}
            ops.recur(cat(y), cat(proj), cat(low), M, S.batch(ents, defer=[b for b, _ in ents]), S.kv, 0, None)
            assert all(S.len.get(b, 0) == n for b, n in before.items())
        ops.recur(cat(y), cat(proj), cat(low), M, S.batch(ents), S.kv, 0, out)
        for (b, p, n), o in zip(step, out.cpu().split([n for _, _, n in step])):
            got[b].append(o)
            if p + n == lens[b]:
                S.free(b)
    want = {}
    A, bias, D = M.rec.A.double().cpu(), M.rec.dt_bias.double().cpu(), M.rec.D.double().cpu()
    for b in lens:
        yd, pd, n = y[b].double(), proj[b].double()[:, 5:5 + H], lens[b]
        heads = []
        if kind == "delta":
            G = spec.kv_heads
            q, k, v = yd[:, :G * N].view(n, G, N), yd[:, G * N:2 * G * N].view(n, G, N), yd[:, 2 * G * N:].view(n, H, e)
            dec = torch.exp(-A[:, None] * O.softplus(low[b].double()[:, :H * N].view(n, H, N) + bias.view(H, N)))
            for h in range(H):
                heads.append(O.delta_rule(O.unit(q[:, h * G // H]) * N ** -0.5, O.unit(k[:, h * G // H]), v[:, h], dec[:, h], O.sigmoid(pd[:, h])))
        else:
            G, inner = spec.groups, H * e
            x, B, Cm = yd[:, :inner].view(n, H, e), yd[:, inner:inner + G * N].view(n, G, N), yd[:, inner + G * N:].view(n, G, N)
            dt = O.softplus(pd + bias)
            for h in range(H):
                heads.append(O.state_space(x[:, h], B[:, h * G // H], Cm[:, h * G // H], dt[:, h], torch.exp(-A[h] * dt[:, h]), D[h]))
        want[b] = torch.cat(heads, 1)
    return {b: torch.cat(got[b]) for b in lens}, want


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("sizes", DELTAS)
def test_delta_rule(ops, sizes, dtype):
    from blaze_b200.config import DeltaSpec
    got, want = run_recurrence(ops, "delta", DeltaSpec(*sizes, conv=2), dtype, LENS, SIZES, late=(2, 5))
    for b in LENS:
        assert rel(got[b], want[b]) < 1e-5, b            # fp32 inside for either type: inputs are exact


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("sizes", SPACES)
def test_state_space(ops, sizes, dtype):
    from blaze_b200.config import StateSpaceSpec
    H, e, N, G = sizes
    got, want = run_recurrence(ops, "ssm", StateSpaceSpec(H, e, N, G, 1, 2), dtype, LENS, SIZES, late=(2, 5))
    for b in LENS:
        assert rel(got[b], want[b]) < 1e-5, b


@pytest.mark.parametrize("kind", ["delta", "ssm"])
def test_recurrences_with_many_sequences(ops, kind):
    """Enough sequences that every width of the kernels' column split is taken; long runs beside single tokens."""
    from blaze_b200.config import DeltaSpec, StateSpaceSpec
    spec = DeltaSpec(32, 8, 64, 64, 2) if kind == "delta" else StateSpaceSpec(32, 64, 64, 2, 1, 2)
    for count, n in ((1, 70), (4, 60), (8, 40)):
        lens = {b: n + 3 * b for b in range(count)}
        got, want = run_recurrence(ops, kind, spec, torch.bfloat16, lens, {b: [33, 1, 17] for b in lens})
        for b in lens:
            assert rel(got[b], want[b]) < 1e-5, (count, b)


# ----------------------------------------------------------------------------------- attention alone
ATTN = [(5, 5, 32, 64, 32), (4, 1, 16, 16, 8), (6, 2, 48, 80, 20), (8, 2, 64, 128, 64), (8, 1, 128, 128, 64), (4, 2, 40, 24, 0), (2, 2, 20, 36, 12),
        (3, 1, 64, 32, 2), (5, 1, 24, 120, 24), (2, 1, 144, 136, 96), (16, 1, 32, 32, 16), (40, 1, 16, 48, 16), (9, 3, 10, 6, 6)]
PORTIONS = {"whole": [10 ** 6], "pairs and more": [2, 37, 3, 130, 1], "decode": [190] + [1] * 30}


class AttnLayer:
    """An attention layer fed rows of q | k | v | gate; the kernels' outputs and the oracle's."""

    def __init__(self, ops, case, dtype, window=0):
        from blaze_b200.config import LayerSpec, RotarySpec, SoftAttnSpec
        from blaze_b200.models.qwen3 import Mixer, SoftAttn
        H, G, d, e, rd = case
        self.rot = {"dims": rd, "base": 300.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 120}} if rd else None
        r = RotarySpec(rd, 300.0, True, 4.0, 1.0, 4.0, 120.0) if rd else None
        self.a = SoftAttnSpec(H, G, d, e, 2.5 / d ** 0.5, r, True, True, True, True, window, 0.8)
        self.M = Mixer()
        self.sink = torch.randn(H, generator=torch.Generator().manual_seed(d)) * 2 + 1
        self.M.attn = SoftAttn(self.a, DEV, self.sink)
        at = [H * d, G * d, G * e, H * e]
        self.M.cols = dict(zip(("q", "k", "v", "gate"), [0, at[0], at[0] + at[1], sum(at[:3])]))
        self.width, self.ops, self.dtype, self.S = sum(at), ops, dtype, Sequences(LayerSpec(self.a), dtype)

    def step(self, entries):
        """entries: (slot, rows) -> outputs"""
        n = self.a.heads * self.a.vdim
        out = torch.full((sum(r.shape[0] for _, r in entries), n + 8), 7.0, dtype=self.dtype, device=DEV)
        self.ops.soft_attention(torch.cat([r for _, r in entries]).to(DEV), self.M, self.S.batch([(s, r.shape[0]) for s, r in entries]), self.S.kv, 0,
                                1e-5, out[:, :n])
        assert self.ops.take_status() == 0 and bool((out[:, n:] == 7).all())
        return torch.split(out[:, :n].cpu(), [r.shape[0] for _, r in entries])

    def rows(self, n, seed, plant=()):
        """Random rows; ``plant``: (query, key) places whose score is made to stand out, in every head."""
        a = self.a
        g = torch.Generator().manual_seed(seed)
        q, k = torch.randn(n, a.heads, a.dim, generator=g), torch.randn(n, a.kv_heads, a.dim, generator=g)
        for i, j in plant:
            u = torch.randn(a.dim, generator=g)
            if self.rot:                                  # undo the rotations, so that the rotated vectors agree
                q[i], k[j] = self.turn(u, -i), self.turn(u, -j)
            else:
                q[i], k[j] = u, u
        v, gate = torch.randn(n, a.kv_heads * a.vdim, generator=g), torch.randn(n, a.heads * a.vdim, generator=g)
        return torch.cat([q.reshape(n, -1), k.reshape(n, -1), v, gate], 1).to(self.dtype)

    def turn(self, u, p):
        y = u.clone()
        for i, f in enumerate(O.rotary_frequencies(self.rot)):
            c, s = torch.cos(torch.tensor(p * f)), torch.sin(torch.tensor(p * f))
            y[2 * i], y[2 * i + 1] = u[2 * i] * c - u[2 * i + 1] * s, u[2 * i + 1] * c + u[2 * i] * s
        return y

    def oracle(self, rows):
        a, n = self.a, rows.shape[0]
        q, k, v, gate = torch.split(rows.double(), [a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, a.heads * a.vdim], 1)
        q, k, v = q.reshape(n, a.heads, a.dim), k.reshape(n, a.kv_heads, a.dim), v.reshape(n, a.kv_heads, a.vdim)
        if self.rot:
            q, k = O.rotate(q, self.rot), O.rotate(k, self.rot)
        q, k = O.rms(q, 1e-5), O.rms(k, 1e-5)
        out = [O.sink_attention(q[:, h], k[:, h // a.group], v[:, h // a.group], a.scale, self.sink[h].double()) for h in range(a.heads)]
        return 0.8 * torch.cat(out, 1) * O.sigmoid(gate)


@pytest.mark.parametrize("portions", PORTIONS)
@pytest.mark.parametrize("case", ATTN)
@pytest.mark.parametrize("dtype", TYPES)
def test_attention_with_sink_and_gate(ops, case, portions, dtype):
    L, n = AttnLayer(ops, case, dtype), 220
    # far keys at page borders and at the first tokens, for rows at the edges of row blocks and portions
    plant = [(i, j) for i, j in ((15, 0), (16, 15), (17, 1), (63, 16), (64, 31), (127, 32), (128, 0), (129, 127), (150, 2), (190, 48), (191, 143), (205, 160), (219, 5))]
    rows, out, pos = L.rows(n, 7 + sum(case), plant), [], 0
    for c in C.cut(n, PORTIONS[portions]):
        out.append(L.step([(0, rows[pos:pos + c])])[0])
        pos += c
    want, got = L.oracle(rows), torch.cat(out)
    err = (got.double() - want).abs().amax(1) / want.abs().max()
    limit = 2e-2 if dtype == torch.bfloat16 else 1e-5
    assert err.max() < limit, (int(err.argmax()), float(err.max()))
    assert err.mean() < limit / 4


@pytest.mark.parametrize("case", [(8, 2, 64, 128, 32), (3, 3, 32, 64, 32), (6, 2, 40, 24, 8)])
def test_attention_batches_of_unequal_sequences(ops, case):
    """Long portions, short portions and single rows in one step; a freed sequence's pages serve the next one."""
    L = AttnLayer(ops, case, torch.bfloat16)
    rows = {b: L.rows(n, 50 + b, [(n - 1, n // 3)] if n > 3 else []) for b, n in LENS.items()}
    got = {b: [] for b in LENS}
    for step in schedule(LENS, SIZES, late=(2, 5)):
        for (b, p, n), o in zip(step, L.step([(b, rows[b][p:p + n]) for b, p, n in step])):
            got[b].append(o)
            if p + n == LENS[b]:
                L.S.free(b)
    for b in LENS:
        assert rel(torch.cat(got[b]), L.oracle(rows[b])) < 2e-2, b


def test_long_context_is_split_over_blocks(ops):
    L, n = AttnLayer(ops, (8, 2, 64, 96, 32), torch.bfloat16), 1500
    rows = L.rows(n, 3, [(n - 1, 5), (n - 2, 700), (n - 3, 0), (n - 4, n - 4)])
    L.step([(0, rows[:n - 4])])
    got = torch.cat([L.step([(0, rows[i:i + 1])])[0] for i in range(n - 4, n)])
    want = L.oracle(rows)[-4:]
    assert rel(got, want) < 2e-2


# ----------------------------------------------------------------------------------- whole models
def wide_parallel(**kw):
    return C.parallel(ff=512, left={"heads": 8, "kv_heads": 4, "dim": 64, "vdim": 64, "scale": 0.2}, right={"heads": 4, "kv_heads": 2, "dim": 64, "vdim": 128, "conv": 4},
                      rot={"dims": 64, "base": 1e5, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}}, **kw)


CONFIGS = {
    "mixed layers": C.config(),
    "wider": C.config([wide_parallel(), C.mamba(ff=512, heads=16, vdim=64, state=128, groups=2, norm_groups=4), wide_parallel(weights_of=0),
                       C.mamba(ff=512, heads=16, vdim=64, state=128, groups=2, norm_groups=4, weights_of=1)], width=512, vocab=1000),
    "ragged": C.config([C.mamba(ff=72, heads=5, vdim=9, state=7, groups=1, norm_groups=3, conv=3),
                        C.parallel(ff=None, left={"heads": 3, "kv_heads": 3, "dim": 12, "vdim": 20}, right={"heads": 3, "kv_heads": 1, "dim": 11, "vdim": 13, "conv": 2},
                                   rot={"dims": 6, "base": 50.0})], width=100, vocab=77, alpha=1.0),
}


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("dtype", TYPES)
def test_model_in_every_schedule(tmp_path, name, dtype):
    from blaze_b200.llm import LLM
    from test_niletar_cpu import verify_with_rejected_rows
    cfg = CONFIGS[name]
    w = C.weights(cfg, seed=2)
    V = cfg["vocab"]
    seqs = {"a": C.tokens(150, V, 1), "b": C.tokens(67, V, 2), "c": C.tokens(33, V, 3), "d": C.tokens(1, V, 4), "e": C.tokens(90, V, 5)}
    want = {i: O.forward(cfg, w, t) for i, t in seqs.items()}
    llm = LLM(C.save(tmp_path, cfg, w), device=DEV, dtype=dtype, kv_tokens=336, max_seqs=3, max_model_len=512, enable_prefix_caching=False)
    assert llm.model.ops.is_cuda and llm.engine.kv.layout == "tiles"
    limit = 1e-4 if dtype == torch.float32 else 0.06
    for sched, f in SCHEDULES.items():
        got = C.run(llm.engine, {"a": seqs["a"]}, [[("a", n)] for n in f(150)])["a"]
        assert C.error(got, want["a"]) < limit, sched
    for _ in range(2):
        got = C.run(llm.engine, seqs, mixed_steps(seqs))
        for i in seqs:
            assert C.error(got[i], want[i]) < limit, i
    got = verify_with_rejected_rows(llm.engine, {i: [t % 300 for t in seqs[i]] if V >= 300 else seqs[i] for i in ("b", "c")}) if V >= 300 else {}
    for i in got:
        assert C.error(got[i], O.forward(cfg, w, [t % 300 for t in seqs[i]])) < limit, i


@pytest.mark.parametrize("graphs", [True, False])
def test_generation_follows_the_logits(tmp_path, graphs):
    """Greedy generation through the scheduler (captured decode steps, prefix cache, speculation): every chosen token is the best
    one of the oracle's logits for that context, up to bf16 rounding."""
    from blaze_b200.llm import LLM
    from blaze_b200.sampler import SamplingParams
    cfg = CONFIGS["wider"]
    w = C.weights(cfg, seed=6)
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
    w = C.weights(cfg, seed=9)
    prompts = [C.tokens(n, 320, 60 + n) for n in (40, 7)]
    llm = LLM(C.save(tmp_path, cfg, w), device=DEV, dtype=torch.float32, kv_tokens=512, max_seqs=2, max_model_len=128)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        t = list(p)
        for _ in range(24):
            t.append(int(O.forward(cfg, w, t)[-1].argmax()))
        assert o.token_ids == t[len(p):]
