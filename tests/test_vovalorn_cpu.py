"""Vovalorn without a device: the configuration reader, what the model description says, layers that run another layer's tensors,
the cache entries of keys that are values, and the plain implementation's mechanisms against closed forms."""
import copy
import math

import pytest
import torch

from plain import vovalorn_plain as P

from ithaca_b200.cache.cache import KVRequest, SequenceCache, plan_groups
from ithaca_b200.config import ConfigError, config_from_dict, describe, validate_schedule
from ithaca_b200.config.vovalorn import VovalornConfig
from ithaca_b200.engine.model import weight_manifest

ATT = {"heads": 6, "kv_heads": 3, "dim": 24, "vdim": 24, "scale": 0.2, "softcap": 30.0, "q_temp": {"coef": 0.2, "every": 50}}
GLA = {"heads": 3, "dim": 16, "vdim": 40, "tau": 8.0}
MOE = {"kind": "moe", "expert": {"ff": 24}, "shared": {"ff": 56}, "router": {"experts": 12, "top": 2, "scale": 1.5, "groups": {"count": 4, "keep": 2}}}
CFG = {
    "architecture": "Vovalorn", "vocab": 61, "width": 40, "norm": {"eps": 1e-6}, "residual_mult": 0.6,
    "layers": [
        {"type": "attention", "mixer": ATT, "mlp": MOE},
        {"type": "gla", "mixer": GLA, "mlp": None},
        {"type": "gla", "mixer": GLA, "mlp": None, "weights_of": 1},
        {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 8, "scale": 0.4},
         "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 3, "top": 3}}},
        {"type": "attention", "mixer": ATT, "mlp": MOE, "weights_of": 0},
        {"type": "gla", "mixer": GLA, "mlp": None, "weights_of": 2},
    ],
}


def test_the_description_names_parts_runs_and_tensors():
    arch, cfg = config_from_dict(CFG)
    assert isinstance(cfg, VovalornConfig) and arch.name == "Vovalorn"
    cfg = cfg.with_tensor_shapes({"l1.mix.a1": (5, 40)})
    spec = cfg.model_spec()
    validate_schedule(spec)
    assert [b.kind for b in spec.layers] == ["sandwich"] * 3 and [b.mixer.kind for b in spec.layers] == ["attention", "gla", "attention"]
    assert [e.layer for e in spec.schedule] == [0, 1, 1, 2, 0, 1] and [e.cache for e in spec.schedule] == list(range(6))
    assert len(describe(spec)) == 6 and all(b.params["residual_mult"] == 0.6 for b in spec.layers)
    man = weight_manifest(spec)
    assert {n: tuple(man[n].shape) for n in man if n.startswith("l0.mix")} == {"l0.mix.q": (144, 40), "l0.mix.k": (72, 40), "l0.mix.o": (40, 144)}
    assert {n: tuple(man[n].shape) for n in man if n.startswith("l1.")} == {
        "l1.mix.q": (48, 40), "l1.mix.k": (48, 40), "l1.mix.v": (120, 40), "l1.mix.g": (120, 40), "l1.mix.o": (40, 120), "l1.mix.norm": (40,),
        "l1.mix.a1": (5, 40), "l1.mix.a2": (48, 5), "l1.mix.a2.b": (48,),
        **{f"l1.{n}{s}": shape for n in ("norm1", "norm1b") for s, shape in (("", (40,)), (".b", (40,)), (".alpha", ()))}}
    assert not any(n.startswith(("l2.", "l4.", "l5.")) for n in man)
    assert tuple(man["l0.mlp.correction"].shape) == (12,) and tuple(man["l0.mlp.shared.down"].shape) == (40, 56) and "l3.mlp.shared.up" not in man
    assert {"embed", "embed.norm", "embed.norm.alpha", "final.norm.b", "head", "l0.norm2b.alpha", "l3.mlp.e2.gate"} <= set(man)
    att, moe = spec.layers[0].mixer, spec.layers[0].feed_forward
    assert att["values"] == "keys" and att["qk_norm"] == "unit" and att["q_temp"] == (0.2, 50) and att["softcap"] == 30.0
    assert att["distance_slopes"] == tuple(2.0 ** (-8 * (n + 1) / 6) for n in range(6))
    assert spec.layers[2].mixer["softcap"] is None and spec.layers[2].mixer["q_temp"] is None
    assert spec.layers[1].mixer["scale"] == 16 ** -0.5 and spec.layers[1].mixer["tau"] == 8.0
    assert (moe["n_groups"], moe["group_keep"], moe["group_score"], moe["weight_scale"], moe["shared"]) == (4, 2, "best_two", 1.5, 56)
    assert (spec.layers[2].feed_forward["n_groups"], spec.layers[2].feed_forward["weight_scale"]) == (0, 1.0)
    assert config_from_dict(cfg.to_dict())[1].model_spec() == spec


def test_a_layer_may_run_the_tensors_of_a_later_one():
    c = copy.deepcopy(CFG)
    c["layers"][1]["weights_of"] = 2
    del c["layers"][2]["weights_of"]
    c["layers"][5]["weights_of"] = 1
    spec = config_from_dict(c)[1].model_spec()
    assert [e.layer for e in spec.schedule] == [0, 1, 1, 2, 0, 1] and any(n.startswith("l2.mix") for n in weight_manifest(spec))
    assert not any(n.startswith("l1.") for n in weight_manifest(spec))


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][1].__setitem__("type", "mamba2"), "type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("vdim", 16), "vdim"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("softcap", 0), "softcap"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("q_temp", {"coef": 0.1}), "every"),
    (lambda c: c["layers"][3]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("tau", 0), "tau"),
    (lambda c: c["layers"][2].__setitem__("mixer", {**GLA, "tau": 9.0}), "mixer"),
    (lambda c: c["layers"][4].__setitem__("mlp", None), "mlp"),
    (lambda c: c["layers"][2].__setitem__("weights_of", 2), "weights_of"),
    (lambda c: c["layers"][2].__setitem__("weights_of", 9), "weights_of"),
    (lambda c: c["layers"][1].__setitem__("weights_of", 2), "weights_of"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 13), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("count", 5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("keep", 5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 7), "fewer experts"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "kind"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("vocab"), "vocab"),
])
def test_config_errors_name_the_key(change, word):
    c = copy.deepcopy(CFG)
    change(c)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(c)


# ------------------------------------------------------------------------------------------ the cache
def test_entries_whose_values_are_keys_hold_one_row_and_a_number():
    kv, _ = plan_groups({0: [KVRequest(2, 16, values_in_keys=True, key_scales=True)], 1: [KVRequest(2, 16, values_in_keys=True)],
                         2: [KVRequest(2, 16, values_in_keys=True, key_scales=True)], 3: [KVRequest(2, 16)]})
    assert [(g.v_head_dim, g.key_scales, g.cache_entries) for g in kv] == [(0, True, (0, 2)), (0, False, (1,)), (16, False, (3,))]
    c = SequenceCache({0: [KVRequest(2, 16, values_in_keys=True, key_scales=True)], 1: [KVRequest(2, 16)]}, max_tokens=128, max_slots=2,
                      kv_dtype=torch.float32, device="cpu")
    a, b = c.layer(0), c.layer(1)
    assert a.k_pages.shape == (2, 2, 64, 16) and a.v_pages is None and a.key_scales.shape == (2, 2, 64) and a.key_scales.dtype == torch.float32
    assert b.v_pages.shape == (2, 2, 64, 16) and b.key_scales is None
    assert c.bytes_per_token() == 2 * (16 * 4 + 4) + 2 * 32 * 4


# ------------------------------------------------------------------------------------------ the plain implementation
def test_plain_norm():
    t = {"n": torch.tensor([2.0, 1.0]), "n.b": torch.tensor([0.5, 0.0]), "n.alpha": torch.tensor(0.25)}
    y = P.dynamic_tanh(torch.tensor([[4.0, -2.0]], dtype=torch.float64), t, "n")
    assert torch.allclose(y, torch.tensor([[2 * math.tanh(1.0) + 0.5, -math.tanh(0.5)]], dtype=torch.float64))


def test_plain_linear_attention_is_a_weighted_sum():
    g = torch.Generator().manual_seed(0)
    T, H, K, V = 7, 2, 3, 5
    q, k, v = (torch.randn(s, generator=g, dtype=torch.float64) for s in ((T, H, K), (T, H, K), (T, H, V)))
    a = torch.rand(T, H, K, generator=g, dtype=torch.float64)
    o, S = P.gla(q, k, v, a)
    h, t = 1, 6
    want = sum((q[t, h] * k[j, h] * a[j + 1:t + 1, h].prod(0)).sum() * v[j, h] for j in range(t + 1))
    assert torch.allclose(o[t, h], want)
    o2, S2 = P.gla(q[4:], k[4:], v[4:], a[4:], P.gla(q[:4], k[:4], v[:4], a[:4])[1])
    assert torch.allclose(o2, o[4:]) and torch.allclose(S2, S)


def test_plain_decay_is_a_root_of_the_sigmoid():
    z = torch.tensor([-700.0, -3.0, 0.0, 2.0, 50.0], dtype=torch.float64)
    assert torch.allclose(P.channel_decay(z, 4.0)[1:], torch.sigmoid(z[1:]) ** 0.25) and math.isclose(float(P.channel_decay(z, 100.0)[0]), math.exp(-7.0))


def test_plain_attention_by_hand():
    """Three positions, two heads: temperature, cap in front of the bias, values in front of the norm."""
    m = {"heads": 2, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 3.0, "softcap": 2.0, "q_temp": {"coef": 0.5, "every": 2}}
    t = {"q": torch.eye(4, 2), "k": torch.eye(2), "o": torch.eye(4)}
    t["q"][2:] = torch.eye(2)
    h = torch.tensor([[3.0, 4.0], [1.0, 0.0], [0.0, 2.0]], dtype=torch.float64)
    out = P.attention_mixer(h, m, t, "", 0.0)
    unit = [x / x.pow(2).mean().sqrt() for x in h]
    temp = 1 + 0.5 * math.log(math.floor(3 / 2) + 1)
    for head, slope in enumerate((2.0 ** -4, 2.0 ** -8)):
        s = [2 * math.tanh(float(unit[2] @ unit[j]) * temp * 3 / 2) - slope * (2 - j) for j in range(3)]
        w = torch.softmax(torch.tensor(s, dtype=torch.float64), -1)
        assert torch.allclose(out[2, 2 * head:2 * head + 2], sum(w[j] * h[j] for j in range(3)))
    assert P.slopes(8)[0] == 0.5 and P.slopes(8)[7] == 2.0 ** -8 and math.isclose(P.slopes(6)[2], 2.0 ** -4)
    assert P.temperature(torch.tensor([0, 2, 3, 7]), 1.0, 4).tolist() == [1.0, 1.0, 1 + math.log(2), 1 + math.log(3)]


def test_plain_choice_of_experts():
    """Groups rank by their two best corrected scores; corrected scores may be negative; the weights know no correction."""
    s = torch.tensor([[0.9, 0.1, 0.6, 0.5, 0.3, 0.2]], dtype=torch.float64)
    r = {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}}
    zero = torch.zeros(6, dtype=torch.float64)
    assert P.choose(s, zero, r).tolist() == [[2, 3]]                        # 0.9 + 0.1 < 0.6 + 0.5
    assert P.choose(s, torch.tensor([0.0, 0.2, 0, 0, 0, 0]), r).tolist() == [[0, 1]]
    low = torch.full((6,), -5.0, dtype=torch.float64)
    assert sorted(P.choose(s, low, {**r, "top": 3, "groups": {"count": 3, "keep": 2}}).tolist()[0]) == [0, 2, 3]
    assert P.choose(s, zero, {"experts": 6, "top": 2}).tolist() == [[0, 2]]
    assert torch.allclose(P.weigh(s, torch.tensor([[2, 3]]), r), torch.tensor([[1.8, 1.5]], dtype=torch.float64) / 1.1)
    assert P.choose(s, zero, {**r, "top": 1, "groups": {"count": 6, "keep": 3}}).tolist() == [[0]]        # groups of one
