"""Bikovik on the GPU against the plain implementation (tests/plain_bikovik.py): every mechanism's kernels alone, then
whole models through trace replay in every way of cutting, keys at the window's edges, and greedy generation through
the entry point."""
import math

import numpy as np
import pytest
import torch

import plain_bikovik as pb
import replay_util as ru

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


def rel(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max())


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def err_word():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


# ---------------------------------------------------------------------------
# the recurrences
# ---------------------------------------------------------------------------
def frequencies(base, dims):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64, device="cuda")


def recurrence_case(kind, H, d, dv, rd, lens, dtype, slow, seed):
    """Rows of projections per sequence, the kernel's arguments, and the plain results."""
    g = torch.Generator().manual_seed(seed)
    eps, base = 1e-5, 300.0
    width = H * (2 * d + dv * (2 if kind == "retention" else 1))
    rows = [torch.randn(n, width + 3, generator=g).to(DT[dtype]) for n in lens]
    if kind == "retention":
        decay = (1.0 - 2.0 ** -torch.linspace(3, 11, H)) if slow else torch.rand(H, generator=g)
        args = dict(decay=decay.float().cuda(), rotary_dim=rd, k_scale=d ** -0.5, gated=True,
                    inv_freq=frequencies(base, rd) if rd else None)
    else:
        bias = torch.randn(H * d, generator=g) * (2 if slow else 8) + (4 if slow else 0)
        lower = torch.rand(H * d, generator=g) * 0.95
        lower[::3] = 0.0
        norm = 1 + 0.2 * torch.randn(dv, generator=g)
        args = dict(f_bias=bias.cuda(), lower=lower.cuda(), norm=norm.cuda())
    want = []
    for a in rows:
        n, x = a.shape[0], a.double()
        q, k = x[:, :H * d].reshape(n, H, d), x[:, H * d:2 * H * d].reshape(n, H, d)
        v = x[:, 2 * H * d:2 * H * d + H * dv].reshape(n, H, dv)
        if kind == "retention":
            rot = {"base": base, "dims": rd} if rd else None
            keep = args["decay"].double().cpu()[None, :, None].expand(n, H, d)
            o = pb.linear_state(pb.rotated(q, rot), pb.rotated(k, rot) * d ** -0.5, v, keep)
            y = pb.rms(o, eps).reshape(n, -1) * pb.silu(x[:, width - H * dv:width])
        else:
            f = pb.forget_gate(k.reshape(n, -1) + bias.double(), lower.double()).view(n, H, d)
            y = (pb.rms(pb.linear_state(pb.silu(q), 1.0 - f, v, f), eps) * norm.double()).reshape(n, -1)
        want.append(y)
    return rows, args, want, eps


@pytest.mark.parametrize("kind", ["retention", "hgrn2"])
@pytest.mark.parametrize("dtype,form", [("float32", "walk"), ("bfloat16", "walk"), ("bfloat16", "chunks")])
@pytest.mark.parametrize("H,d,dv,rd,slow", [(3, 20, 28, 12, True), (2, 64, 128, 64, True), (2, 128, 64, 128, False),
                                            (1, 33, 17, 6, True), (4, 96, 36, 0, False), (2, 128, 128, 16, True),
                                            (1, 8, 4, 8, False), (2, 256, 256, 64, True), (1, 300, 100, 20, True)])
def test_recurrence_in_portions_equals_the_plain_one(kind, dtype, form, H, d, dv, rd, slow, monkeypatch):
    """Three sequences in portions of one token, two and many, around the chunk of 64 and the block of 16, beside each
    other and through state slots used before; slow decays (everything stays in the state) and decays of all strengths,
    some so strong that their products leave float32's range within a few tokens."""
    from rllm_b200.kernels import ops
    if form == "walk":
        monkeypatch.setenv("RLLM_LINEAR_STATE", "simt")
    elif d > 128 or dv > 128:
        pytest.skip("the chunks are built for heads up to 128")
    lens = [171, 33, 230]
    rows, args, want, eps = recurrence_case(kind, H, d, dv, rd, lens, dtype, slow, H * d + dv)
    state = torch.randn(5, H, d, dv, device="cuda")
    slots = [3, 0, 4]
    state[slots] = 0.0
    keep = state[[1, 2]].clone()
    cuts = [[1, 2, 64, 17, 87], [33], [128, 1, 70, 2, 29]]
    got, at = [[] for _ in lens], [0, 0, 0]
    for step in range(5):
        part = [(s, c[step]) for s, c in enumerate(cuts) if step < len(c)]
        part.sort(key=lambda x: x[1] != 1)                # single tokens come first, as in a step
        a = torch.cat([rows[s][at[s]:at[s] + n] for s, n in part]).cuda()
        pos = i32([at[s] + i for s, n in part for i in range(n)])
        q_start, err = np.cumsum([0] + [n for _, n in part]).tolist(), err_word()
        y = ops.linear_state_scan(a, state, i32(q_start), i32([slots[s] for s, _ in part]), len(part), eps, err, positions=pos,
                                  max_q_len=max(n for _, n in part), num_decode=sum(n == 1 for _, n in part), **args)
        assert int(err.item()) == 0 and y.dtype is DT[dtype]
        for r, (s, n) in enumerate(part):
            got[s].append(y[q_start[r]:q_start[r + 1]].float().cpu())
            at[s] += n
    assert at == lens
    tol = 2e-5 if dtype == "float32" else 6e-3
    for s in range(3):
        y = torch.cat(got[s])
        assert torch.isfinite(y).all() and rel(y, want[s]) <= tol, (s, rel(y, want[s]))
    assert torch.equal(state[[1, 2]], keep)


@pytest.mark.parametrize("kind", ["retention", "hgrn2"])
def test_both_forms_leave_the_same_state_and_calls_go_on_from_it(kind, monkeypatch):
    """The chunked form's states against the walk's (what is carried on is float32: no bfloat16 number in between), over
    several calls of a few chunks each."""
    from rllm_b200.kernels import ops
    H, d, dv, lens = 2, 96, 72, [500, 130]
    rows, args, _, eps = recurrence_case(kind, H, d, dv, 32, lens, "bfloat16", True, 9)
    a, pos = torch.cat(rows).cuda(), i32(list(range(500)) + list(range(130)))
    end = []
    for form in ("simt", "chunks"):
        monkeypatch.setenv("RLLM_LINEAR_STATE", form)
        monkeypatch.setattr(ops, "LINEAR_STATE_WORK_BYTES", 300_000)
        state, err, before = torch.zeros(2, H, d, dv, device="cuda"), err_word(), ops.LAUNCHES[0]
        ops.linear_state_scan(a, state, i32([0, 500, 630]), i32([1, 0]), 2, eps, err, positions=pos, max_q_len=500, **args)
        assert int(err.item()) == 0 and (ops.LAUNCHES[0] - before > 2) == (form == "chunks")
        end.append(state.double().cpu())
    assert rel(end[1], end[0]) <= 3e-5


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------
class Pages:
    """Key rows and values of several sequences in shuffled pages, filled by ``ops.talking_prep``."""

    def __init__(self, lens, page, dkp, vrow, dtype, seed):
        g = torch.Generator().manual_seed(seed)
        need = [-(-n // page) for n in lens]
        order = torch.randperm(sum(need) + 3, generator=g).tolist()
        self.page, self.table = page, torch.full((len(lens), max(need) + 1), -1, dtype=torch.int32)
        for s, n in enumerate(need):
            for b in range(n):
                self.table[s, b] = order.pop()
        # garbage where nothing was written: it must not be read
        self.k = torch.full((sum(need) + 3, 1, page, dkp), float("nan"), dtype=DT[dtype], device="cuda")
        self.v = torch.full((sum(need) + 3, 1, page, vrow), float("nan"), dtype=DT[dtype], device="cuda")


def attention_case(H, G, d, dv, rd, lens, dtype, seed, mixed):
    g = torch.Generator().manual_seed(seed)
    width = H * d + G * (d + dv)
    rows = [torch.randn(n, width + 5, generator=g).to(DT[dtype]) for n in lens]
    other = [torch.randn(n, G * dv + 2, generator=g).to(DT[dtype]) for n in lens]
    bias, other_bias = torch.randn(width, generator=g) * 0.5, torch.randn(G * dv, generator=g) * 0.5
    talk = torch.randn(H, H, generator=g) / H ** 0.5 + torch.eye(H)
    lam, base = 0.37, 500.0
    qkv = []
    for a, b in zip(rows, other):
        n, x = a.shape[0], a[:, :width].double() + bias.double()
        rot = {"base": base, "dims": rd} if rd else None
        q = pb.rotated(x[:, :H * d].reshape(n, H, d), rot)
        k = pb.rotated(x[:, H * d:(H + G) * d].reshape(n, G, d), rot)
        v = x[:, (H + G) * d:].reshape(n, G, dv)
        if mixed:
            v = (1 - lam) * v + lam * (b[:, :G * dv].double() + other_bias.double()).view(n, G, dv)
        qkv.append((q, k, v))
    return rows, other, bias, other_bias, talk, lam, frequencies(base, rd) if rd else None, qkv


SHAPES = [(6, 2, 24, 40, 10), (4, 4, 64, 64, 64), (16, 4, 64, 128, 32), (8, 1, 48, 16, 0), (3, 3, 20, 28, 20),
          (16, 4, 128, 128, 128), (12, 6, 80, 72, 16), (2, 2, 256, 200, 64), (40, 8, 64, 64, 64)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,rd", SHAPES)
@pytest.mark.parametrize("mixed", [False, True])
def test_mixed_queries_key_rows_and_values(dtype, H, G, d, dv, rd, mixed):
    """q'_h . row is the mixture of the heads' scores; the rows' and values' padding is zero; another layer's values
    join with their bias; positions far apart and every place of a page."""
    from rllm_b200.kernels import ops
    rows, other, bias, other_bias, talk, lam, inv, _ = attention_case(H, G, d, dv, rd, [9], dtype, H + d, mixed)
    positions, page = [0, 1, 7, 8, 9, 300, 4000, 33, 15], 8
    dkp, dvp = -(-G * d // 64) * 64, -(-dv // 8) * 8 + 8
    table = torch.full((1, 512), -1, dtype=torch.int32)
    for i, b in enumerate(sorted({p // page for p in positions})):
        table[0, b] = (i * 5 + 3) % 11
    kc = torch.full((11, 1, page, dkp), 7.0, dtype=DT[dtype], device="cuda")
    vc = torch.full((11, 1, page, G * dvp), 7.0, dtype=DT[dtype], device="cuda")
    err = err_word()
    kw = dict(v_other=other[0].cuda()[:, 1:1 + G * dv], other_bias=other_bias.cuda(), lam=torch.tensor([lam], device="cuda")) if mixed else {}
    q = ops.talking_prep(rows[0].cuda(), i32(positions), i32([0] * 9), bias.cuda(), talk.cuda(), inv, rd, table.cuda(), kc, vc,
                         H, G, d, dv, err, **kw)
    assert int(err.item()) == 0
    x = rows[0][:, :bias.numel()].double() + bias.double()
    turn = (lambda y: pb.rotate_halves(y, 500.0, rd, torch.tensor(positions))) if rd else (lambda y: y)
    qq, kk = turn(x[:, :H * d].reshape(9, H, d)), turn(x[:, H * d:(H + G) * d].reshape(9, G, d))
    vv = x[:, (H + G) * d:].reshape(9, G, dv)
    if mixed:
        vv = (1 - lam) * vv + lam * (other[0][:, 1:1 + G * dv].double() + other_bias.double()).view(9, G, dv)
    tol = 3e-6 if dtype == "float32" else 1e-2
    want_q = torch.zeros(9, H, dkp, dtype=F64)
    for h in range(H):
        for hh in range(H):
            at = hh // (H // G) * d
            want_q[:, h, at:at + d] += talk[h, hh].double() * qq[:, hh]
    assert rel(q.view(9, H, dkp), want_q) <= tol
    for t, p in enumerate(positions):
        at = (int(table[0, p // page]), 0, p % page)
        krow, vrow = kc[at].double().cpu(), vc[at].double().cpu().view(G, dvp)
        assert float((krow[:G * d] - kk[t].reshape(-1)).abs().max()) <= tol * float(kk.abs().max())
        assert float((vrow[:, :dv] - vv[t]).abs().max()) <= tol * float(vv.abs().max())
        assert float(krow[G * d:].abs().sum()) == 0.0 and float(vrow[:, dv:].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype,form", [("float32", "simt"), ("bfloat16", "simt"), ("bfloat16", "mma"), ("bfloat16", "tcgen05")])
@pytest.mark.parametrize("H,G,d,dv,rd", SHAPES)
@pytest.mark.parametrize("window,keep,page", [(None, 0, 16), (40, 4, 16), (7, 0, 4), (64, 70, 32), (300, 1, 16), (1, 9, 64)])
def test_attention_over_shared_key_rows(dtype, form, H, G, d, dv, rd, window, keep, page):
    """Prompt portions that end at the sequences' last tokens, whole ones, and single tokens, each kernel alone, against
    the plain mixture of scores under the window with kept first keys; pages elsewhere hold NaN."""
    from rllm_b200.kernels import ops
    lens, q_lens, scale = [190, 33, 417, 70], [190, 1, 90, 2], 1.0 / d ** 0.5
    dkp, dvp = -(-G * d // 64) * 64, 64 if dv <= 64 else (128 if dv <= 128 else dv)
    if form == "tcgen05" and not ops.shared_key_tcgen05_takes(DT[dtype], H, G, dkp, dvp, page) or \
            form == "mma" and not ops.shared_key_mma_takes(DT[dtype], H, dkp, G * dvp):
        pytest.skip("sizes of another kernel")
    rows, other, bias, other_bias, talk, lam, inv, qkv = attention_case(H, G, d, dv, rd, lens, dtype, d + dv, True)
    pg = Pages(lens, page, dkp, G * dvp, dtype, 5)
    table = pg.table.cuda()
    mixed = dict(other_bias=other_bias.cuda(), lam=torch.tensor([lam], device="cuda"))
    qs, err = [], err_word()
    for s, n in enumerate(lens):
        q = ops.talking_prep(rows[s].cuda(), i32(list(range(n))), i32([s] * n), bias.cuda(), talk.cuda(), inv, rd, table, pg.k,
                             pg.v, H, G, d, dv, err, v_other=other[s].cuda()[:, :G * dv], **mixed)
        qs.append(q[n - q_lens[s]:])
    q = torch.cat(qs).contiguous()
    q_start, T = np.cumsum([0] + q_lens).tolist(), sum(q_lens)
    out = torch.full((T, H * dv), float("nan"), dtype=DT[dtype], device="cuda")
    pos = i32([n - m + i for n, m in zip(lens, q_lens) for i in range(m)])
    seq = i32([s for s, m in enumerate(q_lens) for _ in range(m)])
    w = int(window or 0)
    if form == "simt":
        ops.attention_simt_kv(q, q.stride(0), out, pg.k, pg.v, table, pos, seq, H, G, w, scale, err, keep_first=keep if w else 0,
                              shared_keys=dv)
    elif form == "tcgen05":
        ops.shared_key_attention_tcgen05(q, out, pg.k, pg.v, table, i32(q_start), i32(lens), 0, 4, T, H, G, dv, w,
                                         keep if w else 0, scale, err)
    else:
        ops.shared_key_attention_mma(q, out, pg.k, pg.v, table, i32(q_start), i32(lens), 4, max(q_lens), H, G, dv, w,
                                     keep if w else 0, scale, err, max(lens))
    assert int(err.item()) == 0
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        qq, kk, vv = qkv[s]
        sc = pb.talking_scores(qq, kk, scale, talk.double()).masked_fill(~pb.visible(n, window, keep), -math.inf)
        p = torch.softmax(sc, dim=-1)
        want = torch.stack([p[h] @ vv[:, h // (H // G)] for h in range(H)], dim=1).reshape(n, -1)[n - m:]
        got = out[q_start[s]:q_start[s + 1]]
        assert torch.isfinite(got).all()
        assert rel(got, want) <= (1e-5 if dtype == "float32" else 4e-2), (s, rel(got, want))


@pytest.mark.parametrize("H,G,d,dv", [(16, 4, 128, 128), (6, 2, 24, 40), (32, 4, 64, 64)])
@pytest.mark.parametrize("window,keep", [(None, 0), (700, 4), (130, 200), (64, 64)])
def test_decoding_in_splits_equals_one_walk(H, G, d, dv, window, keep, monkeypatch):
    """Sequences of very different lengths, one query each: splits of every size the dispatch chooses (by the number of
    sequences) against the plain formula."""
    from rllm_b200.kernels import ops
    base, scale = [1500, 3, 64, 65, 800, 129], d ** -0.5
    dkp, dvp = -(-G * d // 64) * 64, 64 if dv <= 64 else 128
    g = torch.Generator().manual_seed(d)
    w = int(window or 0)
    for S in (1, 6, 24):
        lens = [base[i % 6] for i in range(S)]
        pg = Pages(lens, 16, dkp, G * dvp, "bfloat16", S)
        q = torch.randn(S, H, dkp, generator=g).bfloat16()
        q[:, :, G * d:] = 0
        data = []
        for s, n in enumerate(lens):
            k, v = torch.randn(n, dkp, generator=g).bfloat16(), torch.randn(n, G, dvp, generator=g).bfloat16()
            data.append((k, v))
            for b in range(-(-n // 16)):
                m = min(16, n - b * 16)
                pg.k[pg.table[s, b], 0, :m] = k[b * 16:b * 16 + m].cuda()
                pg.v[pg.table[s, b], 0, :m] = v[b * 16:b * 16 + m].reshape(m, -1).cuda()
        out, err = torch.empty(S, H * dv, dtype=torch.bfloat16, device="cuda"), err_word()
        ops.shared_key_attention_mma(q.reshape(S, -1).cuda(), out, pg.k, pg.v, pg.table.cuda(), i32(list(range(S + 1))), i32(lens),
                                     S, 1, H, G, dv, w, keep if w else 0, scale, err, max(lens))
        assert int(err.item()) == 0
        for s, n in enumerate(lens):
            seen = pb.visible(n, window, keep)[-1]
            p = torch.softmax(((q[s].double() @ data[s][0].double().t()) * scale).masked_fill(~seen, -math.inf), dim=-1)
            want = torch.stack([p[h] @ data[s][1][:, h // (H // G), :dv].double() for h in range(H)]).reshape(-1)
            assert rel(out[s], want) <= 2e-2, (S, s)
