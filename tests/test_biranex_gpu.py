"""Biranex on the GPU against the plain implementation (tests/plain_biranex.py): every mechanism's kernels alone (the
delta rule in its three forms, the state-space recurrence in its two, the convolution without bias, the gated group
norm, the norm on the way into the stream, whole-row query/key norm with rotation and cache write), then whole models
through trace replay in every way of cutting, keys at the window's edge, and greedy generation through the entry
point."""
import copy

import numpy as np
import pytest
import torch

import plain_biranex as pb
import replay_util as ru
from biranex_util import BX_A, BX_B, BX_C, layer, other_ranks, par, sharpen, write_model

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


def rel(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max())


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def err_word():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


def cut_and_run(lens, cuts, slots, run):
    """Feeds the sequences in the given portions, all sequences of a step in one call; ``run(rows, q_start, slots)``
    with rows = [(sequence, first token, count)] returns the step's result; returns it per sequence."""
    got, at = [[] for _ in lens], [0] * len(lens)
    for step in range(max(len(c) for c in cuts)):
        rows, q_start = [], [0]
        for s, c in enumerate(cuts):
            if step < len(c):
                rows.append((s, at[s], c[step]))
                q_start.append(q_start[-1] + c[step])
                at[s] += c[step]
        y = run(rows, q_start, [slots[s] for s, _, _ in rows])
        for r, (s, _, _) in enumerate(rows):
            got[s].append(y[q_start[r]:q_start[r + 1]].float().cpu())
    assert at == list(lens)
    return [torch.cat(g) for g in got]


# ---------------------------------------------------------------------------
# the delta rule
# ---------------------------------------------------------------------------
def delta_data(H, kv, d, dv, lens, dtype, decay, seed):
    """Convolution results, step and beta pre-activations per sequence, and the plain outputs and end states."""
    g = torch.Generator().manual_seed(seed)
    dt_bias, a_log = torch.randn(H * d, generator=g) + decay, torch.randn(H, generator=g)
    share = [h // (H // kv) for h in range(H)]
    data, want = [], []
    for n in lens:
        c = torch.randn(n, 2 * kv * d + H * dv, generator=g).to(DT[dtype])
        step, b = torch.randn(n, H * d, generator=g) * 2, torch.randn(n, H, generator=g) * 2
        data.append((c, step, b))
        cd = c.double()
        q = pb.unit(cd[:, :kv * d].reshape(n, kv, d))[:, share] * d ** -0.5
        k = pb.unit(cd[:, kv * d:2 * kv * d].reshape(n, kv, d))[:, share]
        dec = torch.exp(-torch.exp(a_log.double())[None, :, None] *
                        pb.softplus(step.double() + dt_bias.double()).view(n, H, d))
        o = pb.delta_memory(q, k, cd[:, 2 * kv * d:].reshape(n, H, dv), dec, torch.sigmoid(b.double()))
        want.append(o.reshape(n, H * dv))
    return dt_bias.cuda(), a_log.cuda(), data, want


@pytest.mark.parametrize("dtype,form", [("float32", "walk"), ("bfloat16", "walk"), ("bfloat16", "chunks")])
@pytest.mark.parametrize("H,kv,d,dv,decay", [(4, 2, 20, 28, -3.0), (2, 2, 64, 128, -5.0), (3, 1, 128, 40, 0.0),
                                             (1, 1, 33, 17, 3.0), (2, 1, 256, 8, -2.0)])
def test_delta_rule_in_portions_equals_the_plain_recurrence(dtype, form, H, kv, d, dv, decay, monkeypatch):
    """Three sequences in portions of one token, two, sixteen, seventeen and many, beside each other and through state
    slots that were used before; slow decays (everything stays in the state), ordinary ones, and decays so strong
    that their products leave float32's range within a few tokens."""
    from rllm_b200.kernels import ops
    if form == "walk":
        monkeypatch.setenv("RLLM_CHANNEL_DELTA", "simt")
    lens = [90, 33, 150]
    dt_bias, a_log, data, want = delta_data(H, kv, d, dv, lens, dtype, decay, H * d + dv)
    state = torch.randn(5, H, d, dv, device="cuda")
    slots = [3, 0, 4]
    state[slots] = 0.0
    keep = state[[1, 2]].clone()

    def run(rows, q_start, use):
        c, step, b = (torch.cat([data[s][j][a:a + n] for s, a, n in rows]).cuda() for j in range(3))
        err = err_word()
        o = ops.channel_delta_scan(c, step, b, dt_bias, a_log, 1e-6, state, i32(q_start), i32(use), len(rows), H, kv, d, dv,
                                   err, max_q_len=max(n for _, _, n in rows))
        assert int(err.item()) == 0
        return o

    got = cut_and_run(lens, [[1, 2, 40, 17, 30], [33], [16, 100, 2, 31, 1]], slots, run)
    tol = 3e-6 if form == "walk" else 1e-4
    for s in range(3):
        assert torch.isfinite(got[s]).all() and rel(got[s], want[s]) <= tol, s
    assert torch.equal(state[[1, 2]], keep)


def test_delta_rule_in_several_calls_of_chunks(monkeypatch):
    """A workspace bound of a few chunks: the portion goes in several calls, the state through the slot."""
    from rllm_b200.kernels import ops
    H, kv, d, dv, lens = 2, 2, 64, 48, [200, 75]
    dt_bias, a_log, data, want = delta_data(H, kv, d, dv, lens, "bfloat16", -3.0, 4)
    monkeypatch.setattr(ops, "CHANNEL_DELTA_WORK_BYTES", 1 << 18)
    state, err = torch.zeros(2, H, d, dv, device="cuda"), err_word()
    c, step, b = (torch.cat([x[j] for x in data]).cuda() for j in range(3))
    before = ops.LAUNCHES[0]
    o = ops.channel_delta_scan(c, step, b, dt_bias, a_log, 1e-6, state, i32([0, 200, 275]), i32([1, 0]), 2, H, kv, d, dv,
                               err, max_q_len=200)
    assert ops.LAUNCHES[0] - before > 2 and int(err.item()) == 0
    assert rel(o[:200], want[0]) <= 1e-4 and rel(o[200:], want[1]) <= 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,kv,d,dv,taps,rank", [(2, 2, 20, 28, 3, 8), (2, 2, 64, 128, 4, 24), (4, 2, 100, 36, 2, 16),
                                                 (1, 1, 128, 256, 1, 128), (3, 3, 8, 4, 9, 40)])
def test_delta_rule_one_token_kernel(dtype, H, kv, d, dv, taps, rank):
    """The decoding kernel, from the first product's row to the output product's input, token by token for three
    sequences, against the plain functions (convolutions, unit vectors, low-rank products, recurrence, norm, gate)."""
    from rllm_b200.kernels import ops
    g = torch.Generator().manual_seed(d * H + taps)
    S, T, width, eps, ch = 3, 12, 40, 1e-5, 2 * kv * d + H * dv
    rnd = lambda *shape, m=1.0: (torch.randn(*shape, generator=g) * m).to(DT[dtype])
    w = {"b": rnd(H, width, m=0.3), "a2": rnd(H * d, rank, m=0.3), "g2": rnd(H * dv, rank, m=0.3), "conv": rnd(ch, taps, m=0.6)}
    f32 = {"dt_bias": torch.randn(H * d, generator=g) - 2, "a_log": torch.randn(H, generator=g),
           "norm": 1 + 0.1 * torch.randn(dv, generator=g)}
    at_a, at_g = ch + (-ch) % 8, ch + (-ch) % 8 + rank
    a, x = rnd(S, T, at_g + rank), rnd(S, T, width)
    wc = {k: v.cuda() for k, v in {**w, **f32}.items()}
    wc["norm"] = wc["norm"].repeat(H)
    state, tail = torch.zeros(S + 1, H, d, dv, device="cuda"), torch.zeros(S + 1, taps - 1, ch, device="cuda")
    slots, got = i32([2, 3, 0]), []
    tseq, q0 = i32([0, 1, 2]), i32([0, 1, 2, 3])
    for t in range(T):
        err, at = err_word(), a[:, t].cuda()
        c = None if kv == H else ops.causal_conv(at[:, :ch], wc["conv"], None, tail, q0, tseq, slots, S, False, err)
        y = ops.channel_delta_step(at, c, x[:, t].cuda(), wc, at_a, at_g, taps, 1e-6, eps, tail, state, slots, H, kv, d, dv,
                                   err)
        assert int(err.item()) == 0
        got.append(y.float().cpu())
    got = torch.stack(got, dim=1)
    share = [h // (H // kv) for h in range(H)]
    W = {k: v.double() for k, v in {**w, **f32}.items()}
    for s in range(S):
        row, n = a[s].double(), T
        act = pb.silu(pb.short_conv(row[:, :ch], W["conv"]))
        q = pb.unit(act[:, :kv * d].reshape(n, kv, d))[:, share] * d ** -0.5
        k = pb.unit(act[:, kv * d:2 * kv * d].reshape(n, kv, d))[:, share]
        step = pb.softplus(row[:, at_a:at_a + rank] @ W["a2"].t() + W["dt_bias"]).view(n, H, d)
        dec = torch.exp(-torch.exp(W["a_log"])[None, :, None] * step)
        o = pb.delta_memory(q, k, act[:, 2 * kv * d:].reshape(n, H, dv), dec, torch.sigmoid(x[s].double() @ W["b"].t()))
        gate = torch.sigmoid(row[:, at_g:at_g + rank] @ W["g2"].t()).view(n, H, dv)
        want = (pb.rms(o, eps) * W["norm"] * gate).reshape(n, -1)
        assert rel(got[s], want) <= (1e-5 if dtype == "float32" else 2e-2), s


# ---------------------------------------------------------------------------
# the state-space recurrence and its norm, the convolution
# ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,N,P,slow", [(6, 3, 10, 12, True), (2, 1, 64, 64, True), (4, 2, 128, 32, False), (3, 3, 33, 18, True),
                                          (1, 1, 1, 24, False), (2, 2, 200, 72, True), (2, 1, 96, 128, False)])
def test_state_space_in_portions_and_chunks_equals_the_plain_recurrence(dtype, H, G, N, P, slow):
    """Portions of one token, two, sizes around the chunk of 64 and long ones that run as chunks side by side (on the
    tensor cores in bfloat16, heads filled up to the built sizes), groups of heads with one B and C."""
    from rllm_b200.kernels import ops
    g = torch.Generator().manual_seed(H * N + P)
    lens = [430, 70, 258]
    dt_bias, a_log = torch.randn(H, generator=g) - 2, torch.randn(H, generator=g) - (3 if slow else -1)
    skip = torch.randn(H, generator=g)
    data, want = [], []
    for n in lens:
        c, dt = torch.randn(n, H * P + 2 * G * N, generator=g).to(DT[dtype]), torch.randn(n, H, generator=g) * 2
        data.append((c, dt))
        x, B, C = torch.split(c.double(), [H * P, G * N, G * N], dim=1)
        want.append(pb.state_space(x.reshape(n, H, P), B.reshape(n, G, N), C.reshape(n, G, N),
                                   pb.softplus(dt.double() + dt_bias.double()), torch.exp(a_log.double()),
                                   skip.double()).reshape(n, H * P))
    state = torch.randn(4, H, N, P, device="cuda")
    state[[2, 0, 3]] = 0.0

    def run(rows, q_start, use):
        c, dt = (torch.cat([data[s][j][a:a + n] for s, a, n in rows]).cuda() for j in range(2))
        err = err_word()
        y = ops.ssd_scan(c, dt, dt_bias.cuda(), a_log.cuda(), skip.cuda(), state, i32(q_start), i32(use), len(rows), H, G, N, P,
                         err, max_q_len=max(n for _, _, n in rows))
        assert int(err.item()) == 0
        return y

    got = cut_and_run(lens, [[1, 2, 300, 127], [64, 5, 1], [258]], [2, 0, 3], run)
    for s in range(3):
        assert rel(got[s], want[s]) <= (5e-6 if dtype == "float32" else 1e-4), s


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps", [1, 2, 5, 8, 9])
def test_short_convolution_without_a_bias_in_portions(dtype, taps):
    from rllm_b200.kernels import ops
    g = torch.Generator().manual_seed(taps)
    E, lens = 70, [40, 13]
    x = [torch.randn(n, E + 6, generator=g).to(DT[dtype]) for n in lens]
    w = torch.randn(E, taps, generator=g).to(DT[dtype])
    tail = torch.randn(3, taps - 1, E, device="cuda")
    tail[[2, 1]] = 0.0

    def run(rows, q_start, use):
        part = torch.cat([x[s][a:a + n] for s, a, n in rows]).cuda()
        seq = i32([r for r, (_, _, n) in enumerate(rows) for _ in range(n)])
        err = err_word()
        y = ops.causal_conv(part[:, 3:3 + E], w.cuda(), None, tail, i32(q_start), seq, i32(use), len(rows),
                            any(n > 1 for _, _, n in rows), err)
        assert int(err.item()) == 0
        return y

    got = cut_and_run(lens, [[1, 2, 3, 20, 14], [2, 1, 10]], [2, 1], run)
    for s in range(2):
        want = pb.silu(pb.short_conv(x[s][:, 3:3 + E].double(), w.double()))
        assert rel(got[s], want) <= (2e-6 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,groups", [(72, 4), (40, 40), (4608, 1), (6000, 2)])
def test_gated_group_norm(dtype, E, groups):
    """The gate comes ahead of the norm: a group whose gates are nearly closed is brought back to size by the norm."""
    from rllm_b200.kernels import ops
    g = torch.Generator().manual_seed(E)
    T, eps = 7, 1e-5
    y, w = torch.randn(T, E, generator=g) * 3, 1 + 0.1 * torch.randn(E, generator=g)
    z = torch.randn(T, E + 5, generator=g)
    z[2] -= 6.0
    z = z.to(DT[dtype])
    out = ops.silu_gated_group_rmsnorm(y.cuda(), z.cuda()[:, 2:2 + E], w.cuda(), eps, groups, DT[dtype])
    v = y.double() * pb.silu(z[:, 2:2 + E].double())
    want = pb.rms(v.view(T, groups, -1), eps).reshape(T, E) * w.double()
    assert rel(out, want) <= (3e-6 if dtype == "float32" else 1e-2)


# ---------------------------------------------------------------------------
# into the stream
# ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [37, 72, 2048, 5000])
@pytest.mark.parametrize("two", [False, True])
def test_norm_of_a_result_times_a_constant_into_the_stream(dtype, H, two):
    from rllm_b200.kernels import ops
    from rllm_b200.parts.base import WeightedSum
    g = torch.Generator().manual_seed(H)
    T, eps = 5, 1e-5
    x, w = torch.randn(T, H, generator=g) * 3, 1 + 0.2 * torch.randn(H, generator=g)
    a, b = ((torch.randn(T, H, generator=g) * m).to(DT[dtype]) for m in (1.0, 4.0))
    y = a.double() if not two else 0.3 * a.double() - 1.7 * b.double()
    want = x.double() + 0.45 * pb.rms(y, eps) * w.double()
    xd = x.cuda()
    arg = a.cuda() if not two else WeightedSum((a.cuda(), b.cuda()), (0.3, -1.7))
    act = ops.postnorm_add(xd, arg, w.cuda(), eps, 0.45, DT[dtype])
    assert xd.dtype is torch.float32 and rel(xd, want) <= 1e-6
    assert act.dtype is DT[dtype] and rel(act, want) <= (1e-6 if dtype == "float32" else 5e-3)
    assert (act.data_ptr() == xd.data_ptr()) == (dtype == "float32")
    assert torch.equal(ops.activation_rows(xd, DT[dtype]), xd.to(DT[dtype]))
    if two:
        s = ops.scaled_sum2(a.cuda(), b.cuda(), 0.3, -1.7)
        assert rel(s, y) <= (1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nq,nkv,d,dv,rd,pad", [(6, 2, 24, 40, 10, False), (4, 4, 64, 64, 64, False), (4, 2, 32, 16, 16, True),
                                                (1, 1, 8, 12, 0, False)])
def test_whole_row_norm_rotation_and_cache_write(dtype, nq, nkv, d, dv, rd, pad):
    """Queries and keys over the root mean square of ALL their heads (heads of very different sizes), rotated, keys
    and values in the right page; columns behind the values are left alone."""
    from rllm_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    positions, tseq, page, eps = [0, 1, 9, 130, 4000, 7], [0, 0, 0, 1, 1, 1], 8, 1e-5
    T, W = len(positions), nq * d + nkv * (d + dv)
    rows = torch.randn(T, W + 3, generator=g)
    rows[:, :d] *= 20.0                                   # the first query head carries the row's size
    rows = rows.to(DT[dtype])
    wq, wk = 1 + 0.1 * torch.randn(nq * d, generator=g), 1 + 0.1 * torch.randn(nkv * d, generator=g)
    table = torch.cat([torch.tensor([[3, 1], [0, 2]], dtype=torch.int32), torch.full((2, 510), 4, dtype=torch.int32)], dim=1).cuda()
    dp = max(d, dv)
    kc = torch.zeros(6, nkv, page, dp if pad else d, dtype=DT[dtype], device="cuda")
    vc = torch.zeros(6, nkv, page, dp if pad else dv, dtype=DT[dtype], device="cuda")
    q_out = torch.empty(T, nq * dp, dtype=DT[dtype], device="cuda") if pad else None
    freqs = torch.tensor([90.0 ** (-2.0 * i / rd) / 2.0 for i in range(rd // 2)], dtype=F64, device="cuda") if rd else None
    qkv, err = rows.cuda(), err_word()
    ops.head_norm_kv_write(qkv, i32(positions), i32(tseq), wq.cuda(), wk.cuda(), eps, table, kc, vc, nq, nkv, d, dv, err,
                           q_out=q_out, inv_freq=freqs, rotary_dim=rd, row_norm=True)
    assert int(err.item()) == 0
    rd64, h = rows.double(), rd // 2
    q = (pb.rms(rd64[:, :nq * d], eps) * wq.double()).view(T, nq, d)
    k = (pb.rms(rd64[:, nq * d:(nq + nkv) * d], eps) * wk.double()).view(T, nkv, d)
    if rd:                                                # the kernel rotates halves
        a = torch.tensor(positions)[:, None, None].double() * freqs.cpu()
        for x in (q, k):
            lo, hi = x[..., :h].clone(), x[..., h:rd].clone()
            x[..., :h], x[..., h:rd] = lo * torch.cos(a) - hi * torch.sin(a), hi * torch.cos(a) + lo * torch.sin(a)
    tol = 3e-6 if dtype == "float32" else 1e-2
    got_q = (q_out.view(T, nq, dp)[..., :d] if pad else qkv[:, :nq * d].view(T, nq, d))
    assert rel(got_q, q) <= tol
    assert not pad or float(q_out.view(T, nq, dp)[..., d:].abs().sum()) == 0.0
    assert torch.equal(qkv[:, W:].cpu(), rows[:, W:])
    v = rd64[:, (nq + nkv) * d:W].view(T, nkv, dv)
    for t, (p, s) in enumerate(zip(positions, tseq)):
        at = (int(table[s, p // page]), slice(None), p % page)
        assert float((kc[at][:, :d].double().cpu() - k[t]).abs().max()) <= tol * float(k.abs().max())
        assert torch.equal(vc[at][:, :dv].double().cpu(), v[t])


# ---------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------
CFG = {"A": BX_A, "B": BX_B, "C": BX_C}


@pytest.fixture(scope="module")
def bx_dirs(tmp_path_factory):
    return {"A": write_model(str(tmp_path_factory.mktemp("bx_a")), BX_A, 51, other_ranks),
            "B": write_model(str(tmp_path_factory.mktemp("bx_b")), BX_B, 52, sharpen),
            "C": write_model(str(tmp_path_factory.mktemp("bx_c")), BX_C, 53, sharpen)}


def plain_rows(folder, dtype, reqs):
    cfg, w = pb.read_model_dir(folder, round_to=torch.bfloat16 if dtype == "bfloat16" else None)
    return {r: pb.forward(cfg, w, toks).numpy() for r, toks in reqs.items()}


def compare(got, want, reqs, dtype, what):
    """float32: every position's largest difference against the largest logit.  bfloat16: every sublayer's result is
    normalised on its way into the stream, so its relative rounding error reaches the logits whole; a position's
    error is taken as root mean square over the vocabulary against the logits' own."""
    errs = []
    for r, toks in reqs.items():
        have = np.stack([got[(r, p)] for p in range(len(toks))])
        assert np.isfinite(have).all()
        if dtype == "float32":
            err = np.abs(have - want[r]).max(axis=1) / np.abs(want[r]).max()
            assert err.max() <= 1e-4, (what, r, int(err.argmax()), float(err.max()))
        else:
            errs.append(np.sqrt(((have - want[r]) ** 2).mean(axis=1)) / np.sqrt((want[r] ** 2).mean()))
    if dtype == "bfloat16":
        e = np.concatenate(errs)
        assert np.median(e) <= 0.025 and (e > 0.06).mean() <= 0.02 and e.max() <= 0.1, (what, np.median(e), e.max())


def make_requests(vocab, lengths, seed):
    rng = np.random.default_rng(seed)
    return {f"r{i}": [int(t) for t in rng.integers(0, vocab, size=n)] for i, n in enumerate(lengths)}


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_layers_match_the_plain_residual_after_every_layer(bx_dirs, name):
    from rllm_b200.engine.loading import load_model
    from rllm_b200.engine.replay import TraceSession
    cfg, w = pb.read_model_dir(bx_dirs[name])
    toks = make_requests(CFG[name]["vocab"], [75], seed=2)["r0"]
    want = []
    pb.forward(cfg, w, toks, want)
    _, model = load_model(bx_dirs[name], dtype="float32")
    sess = TraceSession(model, 128, 16, 2)
    trace, orig = [], sess.runner.build_context

    def with_trace(entries):
        ctx, a, b = orig(entries)
        ctx.extras["residual_trace"] = trace
        return ctx, a, b

    sess.runner.build_context = with_trace
    sess.step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": []}], "end": ["a"]})
    assert len(trace) == len(want) == len(CFG[name]["layers"])
    for i, (g, x) in enumerate(zip(trace, want)):
        assert rel(g, x) <= 2e-5, i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page", [("A", 16), ("A", 4), ("B", 16), ("B", 8), ("C", 16)])
def test_every_way_of_cutting_gives_the_plain_logits(bx_dirs, name, page, dtype):
    """Whole prompts, token by token from the first token on, portions down to two tokens, and mixed batches of up to
    four live requests whose pages and state slots are given back and used again (the pool holds exactly the peak);
    every position's logits are compared."""
    V = CFG[name]["vocab"]
    reqs = make_requests(V, [61, 1, 2, 17, 150, 33, 5], seed=7)
    want = plain_rows(bx_dirs[name], dtype, reqs)
    for what, tb in (("whole", ru.trace_whole(reqs)), ("one by one", ru.trace_tail_decode(reqs, tail=1000)),
                     ("tail decoded", ru.trace_tail_decode(reqs, tail=45)),
                     ("portions", ru.trace_portions(reqs, seed=1)),
                     ("mixed", ru.trace_mixed(reqs, seed=2, live=4, tail=6)),
                     ("mixed b", ru.trace_mixed(reqs, seed=3, live=3, tail=30))):
        got = ru.run_trace(bx_dirs[name], dtype, tb, V, page_size=page, max_live=4)
        compare(got, want, reqs, dtype, f"{name}/{dtype}/page {page}/{what}")


@pytest.mark.parametrize("dtype,name", [("float32", "A"), ("bfloat16", "B")])
def test_long_prompts_run_as_chunks_side_by_side(bx_dirs, dtype, name):
    """Prompts long enough for the chunked scans, whole and behind a first portion that ends inside a chunk."""
    V = CFG[name]["vocab"]
    reqs = make_requests(V, [520, 300], seed=4)
    want = plain_rows(bx_dirs[name], dtype, reqs)
    tb = ru.TraceBuilder()
    a, b = reqs["r0"], reqs["r1"]
    tb.step([("r0", a[:37]), ("r1", b[:300])], end=["r1"])
    tb.step([("r0", a[37:518])])
    tb.step([("r0", a[518:519])])
    tb.step([("r0", a[519:])], end=["r0"])
    compare(ru.run_trace(bx_dirs[name], dtype, tb, V), want, reqs, dtype, "long prompts")


@pytest.mark.parametrize("dtype,name", [("float32", "A"), ("bfloat16", "B")])
def test_long_decoding_over_many_pages_beside_a_later_request(bx_dirs, dtype, name):
    """A prompt of 3 tokens, then 260 tokens one by one (pages of 8; the window passes over decoded tokens and pages
    behind it are given back), beside a second request that starts later."""
    V = CFG[name]["vocab"]
    reqs = make_requests(V, [263, 120], seed=9)
    want = plain_rows(bx_dirs[name], dtype, reqs)
    tb = ru.TraceBuilder()
    a, b = reqs["r0"], reqs["r1"]
    tb.step([("r0", a[:3])])
    for i in range(3, 263):
        entries = [("r0", a[i:i + 1])]
        j = i - 60
        if j == 0:
            entries.append(("r1", b[:25]))
        elif 0 < j < 96:
            entries.append(("r1", b[24 + j:25 + j]))
        tb.step(entries, end=(["r0"] if i == 262 else []) + (["r1"] if j == 95 else []))
    got = ru.run_trace(bx_dirs[name], dtype, tb, V, page_size=8)
    compare(got, want, reqs, dtype, "long decoding")


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim", [("float32", 4, 2, 32, 32), ("bfloat16", 4, 2, 64, 64),
                                                     ("bfloat16", 2, 2, 24, 40), ("bfloat16", 4, 1, 16, 64)])
@pytest.mark.parametrize("window,page", [(37, 16), (64, 16), (5, 8)])
def test_a_key_just_inside_the_window_shows_and_one_just_outside_does_not(tmp_path, dtype, heads, kv, dim, vdim, window, page):
    """One token of the sequence is the only key that the last query matches: it is put at the window's last place and
    one place behind it, in prompts, behind portions and with the last tokens decoded.  Attention alone
    (the other branch's scale is 0), the rotation slowed so far that it does not move the score, the sink low."""
    cfg = {"architecture": "Biranex", "vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "residual_mult": 1.0,
           "layers": [layer(par((heads, kv, dim, vdim, 1.0, window, 10.0, 8, 1e6), 1.0, (2, 8, 8, 1, 2, 1), 0.0))]}
    hot = 5

    def edit(w):
        q, k = w["l0.mix.left.q"], w["l0.mix.left.k"]
        w["embed"].mul_(0.05)
        w["embed"][hot] = 0.0
        w["embed"][hot, 0] = 1.0                       # the key
        w["embed"][hot + 1] = 0.0
        w["embed"][hot + 1, 1] = 1.0                   # the query that matches it
        u = torch.randn(dim, generator=torch.Generator().manual_seed(1))
        k[:, 0] = u.repeat(kv)
        q[:, 1] = u.repeat(heads)
        w["l0.mix.left.q.norm"].fill_(1.0)
        w["l0.mix.left.k.norm"].fill_(1.0)
        w["l0.mix.left.sink"].fill_(-2.0)
    folder = write_model(str(tmp_path), cfg, 8, edit)
    pcfg, pw = pb.read_model_dir(folder, round_to=torch.bfloat16 if dtype == "bfloat16" else None)
    rng = np.random.default_rng(3)
    last = {}
    for end in (window, 3 * page - 1, 3 * page, 130):  # the last token's place
        if end < window:
            continue
        for back in (window - 1, window):
            toks = [int(t) for t in rng.integers(8, 64, size=end + 1)]
            toks[end - back] = hot
            toks[end] = hot + 1
            if back == 0:
                continue
            want = pb.forward(pcfg, pw, toks).numpy()
            last[(end, back)] = want[-1]
            reqs = {"r": toks}
            for tb in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, tail=1), ru.trace_tail_decode(reqs, tail=window + 3),
                       ru.trace_portions(reqs, seed=end)):
                got = ru.run_trace(folder, dtype, tb, 64, page_size=page)
                row = got[("r", end)]
                err = np.sqrt(((row - want[-1]) ** 2).mean()) / np.sqrt((want[-1] ** 2).mean())
                assert err <= (1e-4 if dtype == "float32" else 0.03), (end, back, float(err))
        a, b = last[(end, window - 1)], last[(end, window)]
        assert np.sqrt(((a - b) ** 2).mean()) > 0.1 * np.sqrt((a ** 2).mean()), "the key would not show"


def test_the_sink_and_the_gate_change_the_result(tmp_path):
    """With the first layer's sinks high the attention gives next to nothing, with them low it does not; the engine
    follows the plain implementation in both."""
    cfg = copy.deepcopy(BX_B)
    cfg["layers"] = cfg["layers"][:1]
    reqs = make_requests(256, [70], seed=1)
    rows = []
    for i, value in enumerate((-30.0, 6.0)):
        def edit(w):
            sharpen(w)
            w["l0.mix.left.sink"].fill_(value)
        folder = write_model(str(tmp_path / str(i)), cfg, 8, edit)
        want = plain_rows(folder, "float32", reqs)
        for tb in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, tail=30)):
            compare(ru.run_trace(folder, "float32", tb, 256), want, reqs, "float32", value)
        rows.append(want["r0"])
    assert np.abs(rows[0] - rows[1]).max() > 0.05 * np.abs(rows[0]).max()


def test_the_runner_as_a_program_and_pools_no_larger_than_asked(bx_dirs):
    """bin/trace_run as a child process with a pool of exactly the peak of live tokens and its four slots."""
    V = BX_B["vocab"]
    reqs = make_requests(V, [40, 70, 9, 64, 3, 20], seed=13)
    want = plain_rows(bx_dirs["B"], "float32", reqs)
    tb = ru.trace_mixed(reqs, seed=5, live=4, tail=4)
    got = ru.run_trace(bx_dirs["B"], "float32", tb, V, page_size=16, subprocess_mode=True, max_live=None)
    compare(got, want, reqs, "float32", "child process")


def plain_greedy(cfg, w, prompt, n_new):
    seq, out = list(prompt), []
    for _ in range(n_new):
        t = int(torch.argmax(pb.forward(cfg, w, seq)[-1]))
        out.append(t)
        seq.append(t)
    return out


@pytest.mark.parametrize("dtype,name", [("float32", "A"), ("float32", "C"), ("bfloat16", "B")])
def test_greedy_generation_through_the_entry_point(bx_dirs, dtype, name):
    """Nine requests through LLM.generate with the scheduler cutting prompts into portions of at most 16 tokens beside
    decoding requests, CUDA graphs for the decode steps, more requests than sequences at a time.  float32: the plain
    implementation's tokens.  bfloat16: its choice at (nearly) all places where that is clear."""
    from rllm_b200 import LLM, SamplingParams
    V = CFG[name]["vocab"]
    rng = np.random.default_rng(17)
    prompts = [[int(t) for t in rng.integers(0, V, size=int(n))] for n in (5, 41, 1, 23, 60, 2, 9, 30, 14)]
    n_new = 12
    llm = LLM(bx_dirs[name], dtype="fp32" if dtype == "float32" else "bf16", block_size=8, num_gpu_blocks=96,
              max_num_seqs=4, max_num_batched_tokens=24, long_prefill_token_threshold=16, enable_prefix_caching=False)
    assert llm.engine.runner.capture_graphs
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n_new, ignore_eos=True))
    cfg, w = pb.read_model_dir(bx_dirs[name], round_to=torch.bfloat16 if dtype == "bfloat16" else None)
    clear = wrong = 0
    for p, o in zip(prompts, outs):
        got = o.outputs[0].token_ids
        assert len(got) == n_new
        if dtype == "float32":
            assert got == plain_greedy(cfg, w, p, n_new)
            continue
        rows = pb.forward(cfg, w, list(p) + got[:-1])[len(p) - 1:]
        for t, row in zip(got, rows):
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) > 4e-2 * float(row.abs().max()):
                clear += 1
                wrong += t != int(torch.argmax(row))
    assert dtype == "float32" or (clear >= 20 and wrong <= 0.05 * clear), (clear, wrong)
    assert any(g.graph is not None for g in llm.engine.runner.graphs.values())
    llm.engine.cache.check()
    assert llm.engine.cache.usage()["num_requests"] == 0
