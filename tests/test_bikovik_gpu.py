"""Bikovik on the GPU against the plain implementation (tests/plain_bikovik.py): every mechanism's kernels alone, then
whole models through trace replay in every way of cutting, keys at the window's edges, and greedy generation through
the entry point."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import plain_bikovik as pb
import replay_util as ru
from bikovik_util import BK_A, BK_B, BK_C, att, hgrn2, ret, sharpen, write_model

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


# ---------------------------------------------------------------------------
# norm, gate, cap
# ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [45, 72, 2048])
def test_dynamic_tanh_completes_the_stream_and_normalises_it(dtype, H):
    from rllm_b200.kernels import ops
    g = torch.Generator().manual_seed(H)
    x, delta = torch.randn(7, H, generator=g) * 3, (torch.randn(7, H, generator=g) * 2).to(DT[dtype])
    w = {"n": 1 + 0.2 * torch.randn(H, generator=g), "n.b": torch.randn(H, generator=g), "n.alpha": torch.tensor([0.8])}
    w64 = {k: v.double() for k, v in w.items()}
    rows = [5, 0, 5]
    for d in (None, delta):
        full = x.double() + (d.double() if d is not None else 0)
        for pick in (None, rows):
            xd = x.cuda()
            out = torch.empty(7 if pick is None else 3, H, dtype=DT[dtype], device="cuda")
            ops.dyt(xd, w["n.alpha"].cuda(), w["n"].cuda(), w["n.b"].cuda(), out, delta=None if d is None else d.cuda(),
                    rows=None if pick is None else i32(pick), writeback=d is not None and pick is None)
            want = pb.dynamic_tanh(w64, "n", full)
            assert rel(out, want if pick is None else want[pick]) <= (1e-6 if dtype == "float32" else 5e-3)
            assert rel(xd, full if d is not None and pick is None else x.double()) <= 1e-6


@pytest.mark.parametrize("M", [1, 3, 8, 16])
@pytest.mark.parametrize("N,K", [(72, 40), (128, 192), (2048, 512)])
def test_a_decode_product_adds_into_the_stream_and_makes_the_next_norm(M, N, K):
    """The residual epilogue with a dynamic tanh: the new stream, and its whole norm in bfloat16."""
    from rllm_b200.kernels import ops
    g = torch.Generator().manual_seed(N + M)
    x, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(N, K, generator=g) * 0.1).bfloat16()
    h = torch.randn(M, N, generator=g) * 2
    p = {"n": (1 + 0.2 * torch.randn(N, generator=g)), "n.b": torch.randn(N, generator=g), "n.alpha": torch.tensor([0.7])}
    for vec in (torch.float32, torch.bfloat16):
        pv = {k: (v if k == "n.alpha" else v.to(vec)) for k, v in p.items()}
        hd = h.cuda()
        _, scaled = ops.gemm_small_m_residual(x.cuda(), w.cuda(), hd, None,
                                              tanh_norm=(pv["n.alpha"].cuda(), pv["n"].cuda(), pv["n.b"].cuda()))
        want = h.double() + x.double() @ w.double().t()
        assert rel(hd, want) <= 1e-5
        assert rel(scaled, pb.dynamic_tanh({k: v.double() for k, v in pv.items()}, "n", want)) <= 5e-3


@pytest.mark.parametrize("rows", [1, 8, 16, 40, 300])
@pytest.mark.parametrize("dtype,mode", [("float32", ""), ("bfloat16", ""), ("bfloat16", "tcgen05"), ("bfloat16", "library")])
@pytest.mark.parametrize("limit", [0.4, 7.0])
def test_clamped_gate_in_every_form_of_the_product(rows, dtype, mode, limit, monkeypatch):
    """Gate pre-activations far above the limit, both signs of the other factor beyond it."""
    from rllm_b200.parts.registry import build_part
    from rllm_b200.parts.spec import PartSpec
    monkeypatch.setenv("RLLM_GEMM", mode)
    g = torch.Generator().manual_seed(rows)
    H, F = 64, 136
    w = {"m.gate": torch.randn(F, H, generator=g) * 0.6, "m.up": torch.randn(F, H, generator=g) * 0.6,
         "m.down": torch.randn(H, F, generator=g) * 0.2}
    w = {k: v.to(DT[dtype]) for k, v in w.items()}
    x = torch.randn(rows, H, generator=g).to(DT[dtype])
    part = build_part("feed_forward", PartSpec.of("gated_mlp", hidden_size=H, intermediate_size=F, limit=limit, slope=1.702,
                                                  up_shift=1.0, tensor_names={"gate": "gate", "up": "up", "down": "down"}), prefix="m.")
    part.load({k: v.cuda() for k, v in w.items()})
    want = pb.clamped_ff({k: v.double() for k, v in w.items()}, "m.", x.double(), limit)
    assert rel(part.forward(x.cuda()), want) <= (1e-5 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("shape", [(3, 97), (8, 32768), (1, 1)])
def test_logit_cap(shape):
    from rllm_b200.kernels import ops
    x = torch.randn(*shape, generator=torch.Generator().manual_seed(1)) * 40
    x[0, 0] = 1e8
    assert rel(ops.softcap_rows(x.cuda(), 20.0), pb.soft_cap(x.double(), 20.0)) <= 1e-6


# ---------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------
CFG = {"A": BK_A, "B": BK_B, "C": BK_C}


@pytest.fixture(scope="module")
def bk_dirs(tmp_path_factory):
    return {n: write_model(str(tmp_path_factory.mktemp("bk_" + n)), CFG[n], 61 + i, sharpen) for i, n in enumerate("ABC")}


def plain_rows(folder, dtype, reqs):
    cfg, w = pb.read_model_dir(folder, round_to=torch.bfloat16 if dtype == "bfloat16" else None)
    return {r: pb.forward(cfg, w, toks).numpy() for r, toks in reqs.items()}


def compare(got, want, reqs, dtype, what):
    """float32: every position's largest difference against the largest logit.  bfloat16: root mean square over the
    vocabulary against the logits' own."""
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
        assert np.median(e) <= 0.03 and (e > 0.08).mean() <= 0.02 and e.max() <= 0.2, (what, np.median(e), e.max())


def make_requests(vocab, lengths, seed):
    rng = np.random.default_rng(seed)
    return {f"r{i}": [int(t) for t in rng.integers(0, vocab, size=n)] for i, n in enumerate(lengths)}


@pytest.mark.parametrize("tokens", [75, 1])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_layers_match_the_plain_residual_after_every_layer(bk_dirs, name, tokens):
    """A prompt in one step, and its last token decoded; in bfloat16 the decode path with its fused norms runs too."""
    from rllm_b200.engine.loading import load_model
    from rllm_b200.engine.replay import TraceSession
    toks = make_requests(CFG[name]["vocab"], [75], seed=2)["r0"]
    for dtype in ("float32", "bfloat16"):
        cfg, w = pb.read_model_dir(bk_dirs[name], round_to=DT[dtype])
        want = []
        pb.forward(cfg, w, toks, want)
        _, model = load_model(bk_dirs[name], dtype=dtype)
        sess = TraceSession(model, 128, 16, 2)
        sess.runner.capture_graphs = False
        trace, orig = [], sess.runner.build_context

        def with_trace(entries):
            ctx, a, b = orig(entries)
            ctx.extras["residual_trace"] = trace
            return ctx, a, b

        if tokens == 1:
            sess.step({"step": 0, "entries": [{"id": "a", "tokens": toks[:-1], "want": []}], "end": []})
        sess.runner.build_context = with_trace
        sess.step({"step": 1, "entries": [{"id": "a", "tokens": toks[-tokens:], "want": []}], "end": ["a"]})
        assert len(trace) == len(want) == len(CFG[name]["layers"])
        for i, (g, x) in enumerate(zip(trace, want)):
            err = (g.double().cpu() - x[-tokens:]).pow(2).mean().sqrt() / x.pow(2).mean().sqrt()
            assert float(err) <= (2e-5 if dtype == "float32" else 4e-2), (dtype, i, float(err))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page", [("A", 16), ("A", 4), ("B", 16), ("B", 8), ("B", 64), ("C", 16)])
def test_every_way_of_cutting_gives_the_plain_logits(bk_dirs, name, page, dtype):
    """Whole prompts, token by token from the first token on, portions down to two tokens, and mixed batches of up to
    four live requests whose pages and state slots are given back and used again (the pool holds exactly the peak);
    every position's logits are compared."""
    V = CFG[name]["vocab"]
    reqs = make_requests(V, [61, 1, 2, 17, 150, 33, 5], seed=7)
    want = plain_rows(bk_dirs[name], dtype, reqs)
    for what, tb in (("whole", ru.trace_whole(reqs)), ("one by one", ru.trace_tail_decode(reqs, tail=1000)),
                     ("tail decoded", ru.trace_tail_decode(reqs, tail=45)),
                     ("portions", ru.trace_portions(reqs, seed=1)),
                     ("mixed", ru.trace_mixed(reqs, seed=2, live=4, tail=6)),
                     ("mixed b", ru.trace_mixed(reqs, seed=3, live=3, tail=30))):
        got = ru.run_trace(bk_dirs[name], dtype, tb, V, page_size=page, max_live=4)
        compare(got, want, reqs, dtype, f"{name}/{dtype}/page {page}/{what}")


@pytest.mark.parametrize("dtype,name", [("float32", "A"), ("bfloat16", "B"), ("bfloat16", "A")])
def test_long_prompts_behind_portions_that_end_anywhere(bk_dirs, dtype, name):
    """Prompts of several chunks, whole and behind a first portion that ends inside a chunk, beside a decoded token."""
    V = CFG[name]["vocab"]
    reqs = make_requests(V, [520, 300], seed=4)
    want = plain_rows(bk_dirs[name], dtype, reqs)
    tb = ru.TraceBuilder()
    a, b = reqs["r0"], reqs["r1"]
    tb.step([("r0", a[:37]), ("r1", b[:299])])
    tb.step([("r0", a[37:518]), ("r1", b[299:])], end=["r1"])
    tb.step([("r0", a[518:519])])
    tb.step([("r0", a[519:])], end=["r0"])
    compare(ru.run_trace(bk_dirs[name], dtype, tb, V), want, reqs, dtype, "long prompts")


@pytest.mark.parametrize("dtype,name", [("float32", "A"), ("bfloat16", "B")])
def test_long_decoding_over_many_pages_beside_a_later_request(bk_dirs, dtype, name):
    """A prompt of 3 tokens, then 260 tokens one by one (pages of 8; the windows pass over decoded tokens, pages behind
    them are given back, the kept ones stay), beside a second request that starts later."""
    V = CFG[name]["vocab"]
    reqs = make_requests(V, [263, 120], seed=9)
    want = plain_rows(bk_dirs[name], dtype, reqs)
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
    got = ru.run_trace(bk_dirs[name], dtype, tb, V, page_size=8)
    compare(got, want, reqs, dtype, "long decoding")


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim", [("float32", 4, 2, 32, 24), ("bfloat16", 4, 2, 64, 64),
                                                     ("bfloat16", 2, 2, 24, 40), ("bfloat16", 4, 4, 128, 128)])
@pytest.mark.parametrize("window,keep,page", [(37, 4, 16), (64, 17, 16), (5, 1, 8)])
def test_a_key_at_the_edges_of_the_window_and_of_the_kept_ones(tmp_path, dtype, heads, kv, dim, vdim, window, keep, page):
    """One token of the sequence is the only key that the last query matches: at the window's last place and one behind
    it, at the last kept place and one behind it; in prompts, behind portions and with the last tokens decoded.  The
    rotation's base is so large that it does not move the score."""
    cfg = {"architecture": "Bikovik", "vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
           "logit_softcap": 1000.0, "layers": [att(heads, kv, dim, vdim, 1.0, window, keep, 1e30, 4, False)]}
    hot = 5

    def edit(w):
        q, k = w["l0.mix.q"], w["l0.mix.k"]
        w["embed"].mul_(0.05)
        w["embed"][hot] = 0.0
        w["embed"][hot, 0] = 3.0                       # the key
        w["embed"][hot + 1] = 0.0
        w["embed"][hot + 1, 1] = 3.0                   # the query that matches it
        w["l0.norm1"].fill_(1.0)
        w["l0.norm1.b"].fill_(0.0)
        w["l0.norm1.alpha"].fill_(1.0)
        u = torch.randn(dim, generator=torch.Generator().manual_seed(1))
        u[:4] = 0.0                                    # nothing in the dimensions that rotate
        q.mul_(0.1)
        k.mul_(0.1)
        k[:, 0] = (u / u.norm() * 3.5).repeat(kv)
        q[:, 1] = (u / u.norm() * 3.5).repeat(heads)
        for n in ("q.b", "k.b"):
            w["l0.mix." + n].mul_(0.1)
        w["l0.mix.talk"].copy_(torch.eye(heads) + 0.05 * torch.randn(heads, heads, generator=torch.Generator().manual_seed(2)))
        w["l0.mix.v"].mul_(30.0)
        w["l0.mix.o"].mul_(10.0)
    folder = write_model(str(tmp_path), cfg, 8, edit)
    pcfg, pw = pb.read_model_dir(folder, round_to=torch.bfloat16 if dtype == "bfloat16" else None)
    rng = np.random.default_rng(3)
    for end in (window + keep, 3 * page - 1, 3 * page, 130):   # the last token's place
        if end < window + keep:
            continue
        last = {}
        for place in (end - window + 1, end - window, keep - 1, keep):
            toks = [int(t) for t in rng.integers(8, 64, size=end + 1)]
            toks[place], toks[end] = hot, hot + 1
            want = last[place] = pb.forward(pcfg, pw, toks).numpy()[-1]
            reqs = {"r": toks}
            for tb in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, tail=1), ru.trace_tail_decode(reqs, tail=window + 3),
                       ru.trace_portions(reqs, seed=end)):
                row = ru.run_trace(folder, dtype, tb, 64, page_size=page)[("r", end)]
                err = np.sqrt(((row - want) ** 2).mean()) / np.sqrt((want ** 2).mean())
                assert err <= (1e-4 if dtype == "float32" else 0.04), (end, place, float(err))
        for seen, hidden in ((end - window + 1, end - window), (keep - 1, keep)):
            a, b = last[seen], last[hidden]
            if hidden >= keep or hidden == keep:       # (behind the window, and no kept token)
                if end - hidden >= window:
                    assert np.sqrt(((a - b) ** 2).mean()) > 0.1 * np.sqrt((a ** 2).mean()), "the key would not show"


@pytest.mark.parametrize("what", ["talk", "value mix", "lower bound", "decay", "gate", "far key"])
def test_what_random_weights_might_hide_changes_the_result(bk_dirs, tmp_path, what):
    """Each of these changes the plain logits clearly, and the engine follows the change, in prompts and in decoding."""
    cfg = copy.deepcopy(BK_A)

    def edit(w):
        sharpen(w)
        if what == "talk":
            w["l1.mix.talk"].copy_(w["l1.mix.talk"].t().contiguous() * -1.0)
        elif what == "value mix":
            w["l4.mix.vmix"].fill_(3.0)
        elif what == "lower bound":
            w["l0.mix.lower"].fill_(0.97)
        elif what == "gate":
            w["l2.mix.g"].mul_(-1.0)
    if what == "decay":
        cfg["layers"][2]["mixer"]["decay"] = [0.5, 0.9999]
    elif what == "far key":
        cfg["layers"][1]["mixer"]["mask"]["keep_first"] = 0
    folder = write_model(str(tmp_path), cfg, 61, edit)
    reqs = make_requests(211, [70], seed=1)
    before, want = plain_rows(bk_dirs["A"], "float32", reqs)["r0"], plain_rows(folder, "float32", reqs)
    diff = np.sqrt(((want["r0"] - before)[30:] ** 2).mean()) / np.sqrt((before ** 2).mean())
    assert diff > 0.02, diff
    for tb in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, tail=30), ru.trace_portions(reqs, seed=3)):
        compare(ru.run_trace(folder, "float32", tb, 211), want, reqs, "float32", what)


def test_bfloat16_rounding_does_not_gather_in_the_states(tmp_path):
    """Slow decays over a long prompt, recurrences alone: a state that passed through bfloat16, or decays that lost their
    last digits, would drift; the error at the end is no larger than at the start."""
    cfg = {"architecture": "Bikovik", "vocab": 128, "width": 64, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
           "logit_softcap": 100.0, "layers": [hgrn2(2, 32, 48), ret(2, 32, 48, [0.999, 0.9999], 500.0, 32)]}

    def edit(w):
        sharpen(w)
        w["l0.mix.f.b"].fill_(8.0)
    folder = write_model(str(tmp_path), cfg, 5, edit)
    reqs = make_requests(128, [900], seed=1)
    want = plain_rows(folder, "bfloat16", reqs)["r0"]
    for tb in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, tail=300)):
        got = ru.run_trace(folder, "bfloat16", tb, 128)
        err = np.array([np.sqrt(((got[("r0", p)] - want[p]) ** 2).mean()) for p in range(900)]) / np.sqrt((want ** 2).mean())
        assert np.median(err[-100:]) <= 1.5 * np.median(err[100:200]) and err.max() <= 0.1, (np.median(err), err.max())


def test_fork_copies_pages_and_state(bk_dirs):
    """A request forked in the middle of a page goes on independently of its parent."""
    V = BK_A["vocab"]
    a = make_requests(V, [90, 90], seed=31)
    reqs = {"p": a["r0"], "c": a["r0"][:45] + a["r1"][45:]}
    want = plain_rows(bk_dirs["A"], "float32", reqs)
    tb = ru.TraceBuilder()
    tb.step([("p", reqs["p"][:45])])
    tb.step([("c", reqs["c"][45:70]), ("p", reqs["p"][45:46])], fork=[("p", "c")])
    for i in range(46, 90):
        tb.step([("p", reqs["p"][i:i + 1])] + ([("c", reqs["c"][24 + i:25 + i])] if i < 66 else []),
                end=(["c"] if i == 65 else []) + (["p"] if i == 89 else []))
    got = ru.run_trace(bk_dirs["A"], "float32", tb, V, max_tokens=256)
    for p in range(45):
        got[("c", p)] = got[("p", p)]
    compare(got, want, reqs, "float32", "fork")


def test_the_runner_as_a_program_and_pools_no_larger_than_asked(bk_dirs):
    """bin/trace_run as a child process with a pool of exactly the peak of live tokens and its four slots."""
    V = BK_B["vocab"]
    reqs = make_requests(V, [40, 70, 9, 64, 3, 20], seed=13)
    want = plain_rows(bk_dirs["B"], "float32", reqs)
    tb = ru.trace_mixed(reqs, seed=5, live=4, tail=4)
    got = ru.run_trace(bk_dirs["B"], "float32", tb, V, page_size=16, subprocess_mode=True, max_live=None)
    compare(got, want, reqs, "float32", "child process")


def plain_greedy(cfg, w, prompt, n_new):
    seq, out = list(prompt), []
    for _ in range(n_new):
        t = int(torch.argmax(pb.forward(cfg, w, seq)[-1]))
        out.append(t)
        seq.append(t)
    return out


@pytest.mark.parametrize("dtype,name", [("float32", "A"), ("float32", "C"), ("bfloat16", "B")])
def test_greedy_generation_through_the_entry_point(bk_dirs, dtype, name):
    """Nine requests through LLM.generate with the scheduler cutting prompts into portions of at most 16 tokens beside
    decoding requests, CUDA graphs for the decode steps, more requests than sequences at a time.  float32: the plain
    implementation's tokens.  bfloat16: its choice at (nearly) all places where that is clear."""
    from rllm_b200 import LLM, SamplingParams
    V = CFG[name]["vocab"]
    rng = np.random.default_rng(17)
    prompts = [[int(t) for t in rng.integers(0, V, size=int(n))] for n in (5, 41, 1, 23, 60, 2, 9, 30, 14)]
    n_new = 12
    llm = LLM(bk_dirs[name], dtype="fp32" if dtype == "float32" else "bf16", block_size=8, num_gpu_blocks=96,
              max_num_seqs=4, max_num_batched_tokens=24, long_prefill_token_threshold=16, enable_prefix_caching=False)
    assert llm.engine.runner.capture_graphs
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n_new, ignore_eos=True))
    cfg, w = pb.read_model_dir(bk_dirs[name], round_to=torch.bfloat16 if dtype == "bfloat16" else None)
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
            if float(top[0] - top[1]) > 6e-2 * float(row.abs().max()):
                clear += 1
                wrong += t != int(torch.argmax(row))
    assert dtype == "float32" or (clear >= 20 and wrong <= 0.05 * clear), (clear, wrong)
    assert any(g.graph is not None for g in llm.engine.runner.graphs.values())
    llm.engine.cache.check()
    assert llm.engine.cache.usage()["num_requests"] == 0


def test_generation_from_the_command_line(bk_dirs, capsys):
    """``rllm generate`` on token ids: the plain implementation's greedy tokens."""
    from rllm_b200.cli import main
    prompt = make_requests(BK_A["vocab"], [19], seed=8)["r0"]
    assert main(["generate", bk_dirs["A"], "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "6", "--temperature", "0",
                 "--dtype", "fp32", "--ignore-eos", "--num-gpu-blocks", "32", "--json"]) == 0
    got = json.loads([l for l in capsys.readouterr().out.splitlines() if l.startswith("{")][-1])["token_ids"]
    cfg, w = pb.read_model_dir(bk_dirs["A"])
    assert got == plain_greedy(cfg, w, prompt, 6)
