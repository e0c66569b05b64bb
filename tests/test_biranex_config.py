"""Biranex on the host: configuration reader, model spec, tensor list, sizes that the file settles, cache layout and
the order of rotated pairs (no GPU)."""
import copy
import math

import pytest
import torch

import plain_biranex as pb
from biranex_util import BX_A, BX_B, BX_C, other_ranks, write_model
from rllm_b200.config.biranex_config import BiranexConfig
from rllm_b200.config.model_config import ConfigError
from rllm_b200.config.registry import resolve_architecture
from rllm_b200.models.decoder import DecoderModel
from rllm_b200.parts.registry import build_part
from rllm_b200.parts.rotary import rotary_frequencies
from rllm_b200.parts.spec import FreeDim, KVPagesNeed, PartSpec, StateNeed
from rllm_b200.weights.loader import FolderSource, WeightsMismatch, check_tensors, load_tensors


def build(cfg):
    arch = resolve_architecture(cfg)
    return DecoderModel(arch.build_spec(arch.parse_config(cfg)))


def test_every_layer_owns_pages_and_states_of_its_own_sizes():
    lay = build(BX_A).layout
    assert lay.groups[0] == StateNeed((4, 20, 28)) and lay.groups[1] == StateNeed((2, 2 * 2 * 20 + 4 * 28))
    assert lay.groups[2] == KVPagesNeed(2, 24, 11, v_dim=40)
    assert lay.groups[3] == StateNeed((6, 10, 12)) and lay.groups[4] == StateNeed((1, 72 + 2 * 3 * 10))
    assert KVPagesNeed(1, 20, 53) in lay.groups and StateNeed((8, 2 * 3 * 36 + 3 * 12)) in lay.groups
    assert lay.owners[2] == [(1, 0)] and lay.run_owner == [0, 1, 2, 3]
    # keys of 32 and values of 16: rows of one size, so that the tensor-core kernels take them
    c = build(BX_C).layout
    assert KVPagesNeed(2, 32, 19) in c.groups and c.owners[c.groups.index(KVPagesNeed(2, 32, 19))] == [(2, 0), (3, 0)]
    assert StateNeed((0, 1 * 24 + 2)) in c.groups                     # one tap keeps no inputs


def test_the_tensor_list_follows_the_configuration():
    names = {t.name: tuple(t.shape) for t in build(BX_A).tensor_specs()}
    assert names["embed"] == (211, 72) and names["final.norm"] == (72,)
    assert names["l0.norm1"] == (72,) and "l0.norm2" not in names and "l0.mlp.gate" not in names
    assert names["l0.mix.q"] == (40, 72) and names["l0.mix.k"] == (40, 72) and names["l0.mix.v"] == (112, 72)
    assert names["l0.mix.q.conv"] == (40, 3) and names["l0.mix.v.conv"] == (112, 3)
    assert names["l0.mix.b"] == (4, 72) and names["l0.mix.A_log"] == (4,) and names["l0.mix.dt_bias"] == (80,)
    assert names["l0.mix.norm"] == (28,) and names["l0.mix.o"] == (72, 112)
    assert names["l0.mix.a2"][0] == 80 and names["l0.mix.g2"][0] == 112 and names["l0.mix.a1"][1] == 72
    assert names["l1.mix.left.q"] == (144, 72) and names["l1.mix.left.v"] == (80, 72)
    assert names["l1.mix.left.q.norm"] == (144,) and names["l1.mix.left.k.norm"] == (48,)
    assert names["l1.mix.left.sink"] == (6,) and names["l1.mix.left.g"] == (6, 72)
    assert names["l1.mix.left.o"] == (72, 240)
    assert names["l1.mix.right.in"] == (72 + 72 + 60 + 6, 72) and names["l1.mix.right.conv"] == (132, 2)
    assert names["l1.mix.right.conv.b"] == (132,) and names["l1.mix.right.D"] == (6,)
    assert names["l1.mix.right.norm"] == (72,) and names["l1.mlp.up"] == (100, 72) and names["l1.norm2"] == (72,)
    assert "l3.norm2" not in names


def test_constants_reach_the_parts():
    model = build(BX_A)
    assert [b.multiplier for b in model.blocks] == [0.6] * 4
    p = model.blocks[1].mixer
    assert p.scales == (0.7, 0.9)
    left, right = p.branches
    assert left.qk_row and left.pairs and left.window == 11 and left.scale == 0.3 and left.gate == "head" and left.sinks
    assert left.position.freqs == [300.0 ** (-2.0 * i / 10) / 3.0 for i in range(5)] and left.qk_eps == 1e-5
    assert (right.groups, right.norm_groups, right.taps, right.eps) == (3, 4, 2, 1e-5)
    d = model.blocks[0].mixer
    assert (d.heads, d.kv, d.taps, d.unit_eps, d.eps) == (4, 2, 3, 1e-6, 1e-5)
    assert all(x.graph_safe for b in model.blocks for x in b.parts())
    c = BiranexConfig.from_json(BX_C)
    assert c.layers[0].mixer.left.rot_factor == 1.0 and c.layers[0].mixer.left.window == 1
    without = copy.deepcopy(BX_C)
    del without["layers"][0]["mixer"]["left"]["mask"], without["layers"][0]["mixer"]["left"]["rot"]
    c = BiranexConfig.from_json(without)
    assert c.layers[0].mixer.left.window is None and c.layers[0].mixer.left.rot_dims == 0
    assert build(without).blocks[0].mixer.branches[0].window is None


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0].__setitem__("type", "delta"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].__delitem__("vdim"), "vdim"),
    (lambda c: c["layers"][1]["mixer"]["left"].__setitem__("kv_heads", 4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 9), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 26), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].__setitem__("factor", 0), "factor"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][1]["mixer"]["right"].__setitem__("groups", 4), "groups"),
    (lambda c: c["layers"][1]["mixer"]["right"].__setitem__("norm_groups", 7), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].__delitem__("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda c: c.__delitem__("residual_mult"), "residual_mult"),
    (lambda c: c["norm"].__delitem__("eps"), "eps"),
])
def test_what_cannot_be_a_model_is_refused_with_the_reason(edit, what):
    cfg = copy.deepcopy(BX_A)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        BiranexConfig.from_json(cfg)
    assert what in str(e.value)


def test_ranks_come_from_the_file_and_must_agree_within_a_pair(tmp_path):
    folder = write_model(str(tmp_path), BX_A, 3, other_ranks)
    specs = build(BX_A).tensor_specs()
    src = FolderSource(folder)
    t = load_tensors(specs, src, torch.float32, torch.device("cpu"))
    assert t["l0.mix.a1"].shape == (5, 72) and t["l0.mix.a2"].shape == (80, 5)
    assert t["l2.mix.g1"].shape == (19, 72) and t["l2.mix.g2"].shape == (36, 19)
    src.close()

    def broken(w):
        other_ranks(w)
        w["l2.mix.g2"] = w["l2.mix.g2"][:, :7]
    folder = write_model(str(tmp_path / "b"), BX_A, 3, broken)
    src = FolderSource(folder)
    with pytest.raises(WeightsMismatch) as e:
        check_tensors(specs, src)
    assert [n for n, *_ in e.value.wrong_shape] == ["l2.mix.g2"] and e.value.wrong_shape[0][2] == (36, 19)
    src.close()
    d = FreeDim(24, "rank")
    assert d == 24 and d + 1 == 25 and d.key == "rank"


@pytest.mark.parametrize("d,dims", [(24, 10), (8, 8), (20, 2)])
def test_pairs_in_half_order_are_rotated_halves(d, dims):
    """A head put into ``half_order``, rotated half against half and put back is the head with its pairs rotated."""
    rot = {"base": 70.0, "dims": dims, "scaling": {"factor": 2.5}}
    part = build_part("position_encoding", PartSpec.of("rotary", head_dim=d, rotary_dim=dims, theta=70.0, interleaved=True,
                                                       scaling={"kind": "linear", "factor": 2.5}))
    assert part.freqs == rotary_frequencies(dims, 70.0, {"kind": "linear", "factor": 2.5}) and part.magnitude == 1.0
    x = torch.randn(6, 1, d, dtype=torch.float64)
    pos = torch.tensor([0, 1, 5, 77, 300, 4000])
    order = part.half_order()
    assert sorted(order) == list(range(d))
    y, h = x[..., order], dims // 2
    a = pos[:, None, None].double() * torch.tensor(part.freqs, dtype=torch.float64)
    c, s = torch.cos(a), torch.sin(a)
    z = y.clone()
    z[..., :h], z[..., h:dims] = y[..., :h] * c - y[..., h:dims] * s, y[..., h:dims] * c + y[..., :h] * s
    back = torch.empty_like(z)
    back[..., order] = z
    assert float((back - pb.rotate_pairs(x, rot, pos)).abs().max()) < 1e-12


def test_plain_small_functions():
    x = torch.tensor([-30.0, -1.0, 0.0, 2.0, 40.0], dtype=torch.float64)
    assert float((pb.softplus(x) - torch.tensor([math.log1p(math.exp(v)) for v in x.tolist()], dtype=torch.float64)).abs().max()) < 1e-12
    u = pb.short_conv(torch.tensor([[1.0], [2.0], [3.0]], dtype=torch.float64), torch.tensor([[10.0, 1.0]], dtype=torch.float64))
    assert u[:, 0].tolist() == [1.0, 12.0, 23.0]
    assert build(BX_B).spec.layers[1].ffn is not None
