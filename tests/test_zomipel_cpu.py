"""Zomipel without a device: the configuration reader, what the model description says, the pages of kept first keys, and the
plain implementation's mechanisms against closed forms."""
import copy
import math

import pytest
import torch

from plain import zomipel_plain as P

from ithaca_b200.cache.cache import KVRequest, SequenceCache, plan_groups
from ithaca_b200.cache.pages import CacheError
from ithaca_b200.config import ConfigError, config_from_dict, describe, validate_schedule
from ithaca_b200.config.zomipel import ZomipelConfig
from ithaca_b200.engine.model import weight_manifest

CFG = {
    "architecture": "Zomipel", "vocab": 61, "width": 40, "norm": {"eps": 1e-6},
    "layers": [
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 3, "dim": 16, "vdim": 24, "scale": 0.2, "mask": {"size": 30, "keep_first": 5},
                                        "rot": {"dims": 8, "base": 300.0}},
         "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 56}}},
        {"type": "mamba2", "mixer": {"heads": 6, "vdim": 4, "state": 10, "groups": 2, "conv": 4, "norm_groups": 3}, "mlp": {"kind": "dense", "ff": 72}},
        {"type": "mamba2", "mixer": {"heads": 2, "vdim": 8, "state": 16, "groups": 1, "conv": 1, "norm_groups": 1}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.4},
         "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 3, "top": 3}}},
    ],
    "loop": {"start": 1, "stop": 3, "times": 3},
}


def test_the_description_names_parts_runs_and_tensors():
    arch, cfg = config_from_dict(CFG)
    assert isinstance(cfg, ZomipelConfig) and arch.name == "Zomipel"
    spec = cfg.model_spec()
    validate_schedule(spec)
    assert [b.kind for b in spec.layers] == ["parallel"] * 4 and [b.mixer.kind for b in spec.layers] == ["attention", "mamba2", "mamba2", "attention"]
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3] and [e.cache for e in spec.schedule] == list(range(8))
    assert [e.adds_input for e in spec.schedule] == [False, False, False, True, False, True, False, False]
    assert sum("input added first" in line for line in describe(spec)) == 2
    man = weight_manifest(spec)
    assert {n: tuple(man[n].shape) for n in man if n.startswith("l0.mix")} == {
        "l0.mix.q": (96, 40), "l0.mix.k": (48, 40), "l0.mix.v": (72, 40), "l0.mix.o": (40, 144),
        "l0.mix.q.b": (96,), "l0.mix.k.b": (48,), "l0.mix.v.b": (72,)}
    assert {n: tuple(man[n].shape) for n in man if n.startswith("l1.mix")} == {
        "l1.mix.in": (24 + 24 + 20 + 20 + 6, 40), "l1.mix.conv": (64, 4), "l1.mix.conv.b": (64,), "l1.mix.dt_bias": (6,),
        "l1.mix.A_log": (6,), "l1.mix.D": (6,), "l1.mix.norm": (24,), "l1.mix.o": (40, 24)}
    assert tuple(man["l0.mlp.shared.sg"].shape) == (1, 40) and tuple(man["l0.mlp.shared.down"].shape) == (40, 56)
    assert tuple(man["l0.mlp.router.b"].shape) == (5,) and tuple(man["l0.mlp.e4.gate"].shape) == (24, 40)
    assert set(n for n in man if n.startswith("l1.mlp")) == {"l1.mlp.up", "l1.mlp.down"}
    assert not any(n.startswith("l2.mlp") for n in man) and not any(n.startswith("l3.mlp.shared") for n in man)
    assert "head" not in man and {"embed", "final.norm", "l3.norm1"} <= set(man) and not any(n.endswith("norm2") for n in man)
    att = spec.layers[0].mixer
    assert att["window"] == 30 and att["keep_first"] == 5 and att["bias"] == "qkv" and spec.layers[0].position["rotary_dim"] == 8
    assert spec.layers[3].mixer["window"] is None and spec.layers[3].position is None
    assert spec.layers[0].norms["mixer"]["unit_offset"] and spec.layers[0].feed_forward["shared"] == 56
    assert config_from_dict(cfg.to_dict())[1].model_spec() == spec
    plain = copy.deepcopy(CFG)
    del plain["loop"]
    assert [e.layer for e in config_from_dict(plain)[1].model_spec().schedule] == [0, 1, 2, 3]


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][1].__setitem__("type", "mamba1"), "type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("groups", 4), "groups"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("norm_groups", 7), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("keep_first", -1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 6), "top"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "gated"), "kind"),
    (lambda c: c["loop"].__setitem__("stop", 5), "loop"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("vocab"), "vocab"),
])
def test_config_errors_name_the_key(change, word):
    c = copy.deepcopy(CFG)
    change(c)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(c)


# ------------------------------------------------------------------------------------------ pages of kept first keys
def _cache(window, keep, max_tokens=64 * 12):
    return SequenceCache({0: [KVRequest(1, 16, window, keep_first=keep)]}, max_tokens=max_tokens, max_slots=2, device=None)


def _pages(c, s):
    return [i for i, p in enumerate(c.table.tables[0][s]) if p >= 0]


@pytest.mark.parametrize("keep,kept", [(0, []), (1, [0]), (64, [0]), (65, [0, 1]), (130, [0, 1, 2])])
def test_pages_of_the_first_keys_are_never_released(keep, kept):
    c = _cache(70, keep)
    s = c.alloc_slot()
    for n in (300, 1, 63, 100):
        c.reserve([s], [n])
        c.commit([s], [n])
        first = (c.length(s) + 1 - 70) // 64                 # the page of the first key the next query's window reaches
        assert _pages(c, s) == sorted(set(kept) | set(range(first, -(-c.length(s) // 64))))
        c.table.check_consistent()
    assert c.table.pools[0].n_free == 12 - len(_pages(c, s))
    c.free_slot(s)
    assert c.table.pools[0].n_free == 12


def test_truncation_behind_a_window_with_kept_keys():
    c = _cache(70, 100)                                      # pages 0 and 1 stay
    s = c.alloc_slot()
    c.reserve([s], [190]), c.commit([s], [190])
    assert _pages(c, s) == [0, 1, 2]
    c.truncate(s, 3)                                         # nothing has been released: any prefix will do
    c.reserve([s], [397]), c.commit([s], [397])
    assert _pages(c, s) == [0, 1, 5, 6]                      # position 400 reaches back to 331
    with pytest.raises(CacheError, match="released"):
        c.truncate(s, 300)
    c.truncate(s, 390)                                       # reaches back to 321
    c.truncate(s, 0)
    assert _pages(c, s) == [] and c.table.pools[0].n_free == 12
    c.reserve([s], [65]), c.commit([s], [65])
    assert _pages(c, s) == [0, 1]
    c.table.check_consistent()


def test_layers_that_keep_other_first_keys_do_not_share_pages():
    kv, _ = plan_groups({0: [KVRequest(1, 16, 70, keep_first=5)], 1: [KVRequest(1, 16, 70)], 2: [KVRequest(1, 16, 70, keep_first=5)],
                         3: [KVRequest(1, 16, None, keep_first=5)], 4: [KVRequest(1, 16)]})
    assert [(g.window, g.keep_first, g.cache_entries) for g in kv] == [(70, 5, (0, 2)), (70, 0, (1,)), (None, 0, (3, 4))]


def test_seen_pages_covers_every_place_of_a_window():
    from ithaca_b200.csrc.attention_bf16 import seen_pages
    for window in (1, 2, 63, 64, 65, 66, 128, 200):
        for keep in (0, 1, 64, 65, 300):
            for n in range(1, 700, 7):
                pos = n - 1
                lo = max(0, pos + 1 - window)
                real = len(set(range(lo // 64, pos // 64 + 1)) | set(j // 64 for j in range(min(keep, lo))))
                assert real <= seen_pages(n, window, keep) <= -(-n // 64)
    assert seen_pages(1000, 0, 0) == 16


# ------------------------------------------------------------------------------------------ the plain implementation
def test_plain_visibility():
    v = P.visible(8, 3, 2)
    assert [[j for j in range(8) if v[i, j]] for i in (0, 1, 3, 7)] == [[0], [0, 1], [0, 1, 2, 3], [0, 1, 5, 6, 7]]
    assert P.visible(8, None, 2).sum() == 36 and torch.equal(P.visible(8, 3, 0).sum(1), torch.tensor([1, 2, 3, 3, 3, 3, 3, 3]))


def test_plain_state_space_recurrence_is_a_weighted_sum():
    g = torch.Generator().manual_seed(0)
    T, H, G, N, Pv = 7, 4, 2, 3, 5
    x, B, C = (torch.randn(s, generator=g, dtype=torch.float64) for s in ((T, H, Pv), (T, G, N), (T, G, N)))
    dt, A_log, D = torch.rand(T, H, generator=g, dtype=torch.float64), torch.randn(H, generator=g, dtype=torch.float64), torch.randn(H, generator=g, dtype=torch.float64)
    y, S = P.ssd(x, B, C, dt, A_log, D)
    h, t = 3, 6
    want = D[h] * x[t, h]
    for j in range(t + 1):
        decay = math.exp(-math.exp(float(A_log[h])) * float(dt[j + 1:t + 1, h].sum()))
        want = want + decay * float(dt[j, h]) * float(C[t, 1] @ B[j, 1]) * x[j, h]
    assert torch.allclose(y[t, h], want)
    y2, S2 = P.ssd(x[4:], B[4:], C[4:], dt[4:], A_log, D, P.ssd(x[:4], B[:4], C[:4], dt[:4], A_log, D)[1])
    assert torch.allclose(y2, y[4:]) and torch.allclose(S2, S)


def test_plain_gate_comes_before_the_norm_and_parts_are_apart():
    y, z = torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=torch.float64), torch.tensor([[1.0, -1.0, 0.5, 2.0]], dtype=torch.float64)
    w = torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=torch.float64)
    g = (y * z * torch.sigmoid(z))[0]
    out = P.gated_group_norm(y, z, w, 2, 0.0)[0]
    assert torch.allclose(out[:2], g[:2] / g[:2].pow(2).mean().sqrt() * w[:2]) and torch.allclose(out[2:], g[2:] / g[2:].pow(2).mean().sqrt() * w[2:])


def test_plain_router_weights_are_the_softmax_over_the_chosen():
    z, b = torch.tensor([[1.0, 2.0, 3.0, 0.0]], dtype=torch.float64), torch.tensor([0.0, -5.0, 0.0, 2.5], dtype=torch.float64)
    e, w = P.route(z, 2, torch.eye(4, dtype=torch.float64), b)
    assert e.tolist() == [[2, 3]] and torch.allclose(w, torch.softmax(torch.tensor([[3.0, 2.5]], dtype=torch.float64), -1))
