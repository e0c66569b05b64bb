"""Bikovik on the host: configuration reader, model spec, tensor list, cache layout and constants (no GPU)."""
import copy
import math

import pytest
import torch

import plain_bikovik as pb
from bikovik_util import BK_A, BK_B, BK_C, sharpen, write_model
from rllm_b200.config.bikovik_config import BikovikConfig
from rllm_b200.config.model_config import ConfigError
from rllm_b200.config.registry import resolve_architecture
from rllm_b200.models.decoder import DecoderModel
from rllm_b200.parts.registry import build_part
from rllm_b200.parts.spec import KVPagesNeed, PartSpec, StateNeed
from rllm_b200.weights.loader import FolderSource, WeightsMismatch, check_tensors, load_tensors


def build(cfg):
    arch = resolve_architecture(cfg)
    return DecoderModel(arch.build_spec(arch.parse_config(cfg)))


def test_every_layer_owns_pages_or_a_state_of_its_own_sizes():
    lay = build(BK_A).layout
    assert lay.groups == [StateNeed((3, 20, 28)), KVPagesNeed(1, 64, 11, v_dim=128, keep_first=3), StateNeed((2, 24, 40)),
                          KVPagesNeed(1, 128, 53, v_dim=128), KVPagesNeed(1, 64, 30, v_dim=128, keep_first=2)]
    assert lay.run_owner == [0, 1, 2, 3, 4]
    b = build(BK_B).layout
    # a key row has all kv heads' keys, values have 64 or 128 places a head
    assert KVPagesNeed(1, 128, 64, v_dim=128, keep_first=5) in b.groups
    assert KVPagesNeed(1, 512, 150, v_dim=512, keep_first=20) in b.groups
    c = build(BK_C).layout
    assert KVPagesNeed(1, 64, None, v_dim=64) in c.groups and KVPagesNeed(1, 64, 2, v_dim=64, keep_first=7) in c.groups


def test_the_tensor_list_follows_the_configuration():
    model = build(BK_A)
    names = {t.name: tuple(t.shape) for t in model.tensor_specs()}
    assert names["embed"] == (211, 72) and names["head"] == (211, 72)
    for n in ("final.norm", "l0.norm1", "l0.norm2", "l4.norm1"):
        assert names[n] == (72,) and names[n + ".b"] == (72,) and names[n + ".alpha"] == ()
    assert names["l0.mix.q"] == names["l0.mix.f"] == (60, 72) and names["l0.mix.f.b"] == names["l0.mix.lower"] == (60,)
    assert names["l0.mix.v"] == (84, 72) and names["l0.mix.norm"] == (28,) and names["l0.mix.o"] == (72, 84)
    assert names["l1.mix.q"] == (120, 72) and names["l1.mix.q.b"] == (120,) and names["l1.mix.k.b"] == (40,)
    assert names["l1.mix.v.b"] == (24,) and names["l1.mix.talk"] == (6, 6) and names["l1.mix.o"] == (72, 72)
    assert names["l2.mix.g"] == (80, 72) and names["l2.mix.k"] == (48, 72) and "l2.mix.q.b" not in names
    assert "l2.mlp.gate" not in names and "l2.norm2" not in names
    # the first layer whose values are mixed in has a factor that nothing uses; the one without mixing none
    assert "l1.mix.vmix" not in names and "l3.mix.vmix" not in names and names["l4.mix.vmix"] == ()
    ignored = {n for p in model.parts() for n in p.ignored_tensors()}
    assert {"l1.mix.vmix", "l2.norm2", "l2.norm2.b", "l2.norm2.alpha"} <= ignored and "l0.norm2" not in ignored


def test_constants_reach_the_parts():
    model = build(BK_A)
    assert model.embedding.scale == 0.7 and model.head.softcap == 11.0 and model.head.tied_to is None
    a = model.blocks[1].mixer
    assert (a.window, a.keep_first, a.scale, a.value_mix, a.head_mix, a.out_bias) == (11, 3, 0.3, "source", True, False)
    assert a.position.freqs == [1.0 / (300.0 ** (2 * i / 10)) for i in range(5)]
    assert [b.mixer.value_mix for b in (model.blocks[3], model.blocks[4])] == [None, "mixed"]
    assert model.blocks[0].ffn.gate == (0.9, 1.702, 1.0) and model.blocks[2].ffn is None
    r = model.blocks[2].mixer
    assert r.decay == (0.9, 0.997) and r.position.rotary_dim == 16 and r.eps == 1e-5
    assert all(x.graph_safe for b in model.blocks for x in b.parts())
    c = build(BK_C)
    assert c.embedding.scale == 1.0 and c.blocks[4].mixer.window is None and c.blocks[1].mixer.position.fused_rotary() == (None, 0)
    without = copy.deepcopy(BK_A)
    del without["logit_softcap"], without["layers"][1]["mixer"]["mask"], without["layers"][1]["mixer"]["rot"]
    without["embedding"]["scale"] = 0.0
    m = build(without)
    assert m.head.softcap is None and m.blocks[1].mixer.window is None and m.embedding.scale == 0.0


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0].__setitem__("type", "gla"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].__delitem__("vdim"), "vdim"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 9), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 22), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("keep_first", -1), "keep_first"),
    (lambda c: c["layers"][4]["mixer"].__setitem__("vdim", 16), "v_mix"),
    (lambda c: c["layers"][2]["mixer"]["decay"].append(0.5), "decay"),
    (lambda c: c["layers"][2]["mixer"]["decay"].__setitem__(0, 1.5), "decay"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].__delitem__("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("limit", 0), "limit"),
    (lambda c: c.__setitem__("logit_softcap", -1), "softcap"),
    (lambda c: c.__delitem__("embedding"), "embedding"),
    (lambda c: c["norm"].__delitem__("eps"), "eps"),
])
def test_what_cannot_be_a_model_is_refused_with_the_reason(edit, what):
    cfg = copy.deepcopy(BK_A)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        BikovikConfig.from_json(cfg)
    assert what in str(e.value)


def test_a_file_may_carry_what_nothing_uses_and_must_carry_the_rest(tmp_path):
    def extra(w):
        sharpen(w)
        w["l1.mix.vmix"] = torch.tensor(0.3)
        for n in ("l2.norm2", "l2.norm2.b", "l2.norm2.alpha"):
            w[n] = w[n.replace("norm2", "norm1")].clone()
    folder = write_model(str(tmp_path), BK_A, 3, extra)
    model = build(BK_A)
    ignored = [n for p in model.parts() for n in p.ignored_tensors()]
    src = FolderSource(folder)
    t = load_tensors(model.tensor_specs(), src, torch.float32, torch.device("cpu"), ignored)
    assert t["l4.mix.vmix"].shape == () and "l1.mix.vmix" not in t
    src.close()
    folder = write_model(str(tmp_path / "b"), BK_A, 3, lambda w: (w.pop("l4.mix.vmix"), w.pop("l0.norm1.alpha")))
    src = FolderSource(folder)
    with pytest.raises(WeightsMismatch) as e:
        check_tensors(model.tensor_specs(), src, ignored)
    assert sorted(e.value.missing) == ["l0.norm1.alpha", "l4.mix.vmix"]
    src.close()


def _attention(**over):
    p = dict(hidden_size=16, num_heads=2, num_kv_heads=1, head_dim=8, bias="qkv", head_mix=True, tensor_prefix="m.",
             tensor_names={k: k for k in ("q", "k", "v", "o", "q_bias", "k_bias", "v_bias", "talk", "value_mix")})
    p.update(over)
    return build_part("mixer", PartSpec.of("attention", **p), prefix="m.")


def test_options_that_do_not_go_together_are_refused():
    assert _attention().cache_need() == KVPagesNeed(1, 64, None, v_dim=64)
    for over in (dict(softcap=5.0), dict(sinks="zero"), dict(bias=False), dict(value_mix="both"), dict(bias="out"),
                 dict(position=PartSpec.of("rotary", head_dim=8, theta=10.0, interleaved=True))):
        with pytest.raises(ValueError):
            _attention(**over)
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec.of("gated_mlp", hidden_size=4, intermediate_size=4, activation="gelu_tanh", limit=1.0,
                                               tensor_names={"gate": "g", "up": "u", "down": "d"}))


def test_plain_small_functions():
    seen = pb.visible(6, 2, 1)
    assert seen.int().tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0],
                                   [1, 0, 0, 1, 1, 0], [1, 0, 0, 0, 1, 1]]
    x = torch.randn(5, 1, 6, dtype=torch.float64)
    y = pb.rotate_halves(x, 10.0, 4, torch.arange(5))
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    assert abs(float(y[3, 0, 0]) - float(x[3, 0, 0] * math.cos(3) - x[3, 0, 2] * math.sin(3))) < 1e-12
    s = pb.talking_scores(torch.ones(1, 2, 3, dtype=torch.float64), torch.ones(1, 1, 3, dtype=torch.float64), 0.5,
                          torch.tensor([[1.0, 2.0], [0.0, -1.0]], dtype=torch.float64))
    assert s[:, 0, 0].tolist() == [4.5, -1.5]
    assert float(pb.soft_cap(torch.tensor(1e9), 3.0)) == 3.0
