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
