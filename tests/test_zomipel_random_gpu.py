"""Seeded random Zomipel configurations against the plain implementation: layer orders, loops, head counts, groups, state and
value sizes, taps, parts of the gated norm, windows, kept keys, experts and constants that no hand-written configuration of
the other tests has, among them sizes the tensor-core kernels take and sizes only the CUDA-core kernels take.  Every model runs
whole prompts, a prompt then decoded tokens, and an unequal batch decoded together with requests that end at different times,
in both types (the 16-bit run against the plain implementation with the library's choice of experts, as in
``test_zomipel_gpu.compare``)."""
import numpy as np
import pytest
import torch

from helpers import random_ids
from test_gunenex_gpu import _write
from test_zomipel_gpu import _att, _ff, _model, _moe, _ssd, compare, make_tensors

pytestmark = pytest.mark.gpu


def random_config(seed):
    r = np.random.default_rng(seed)
    pick = lambda xs: xs[int(r.integers(0, len(xs)))]
    layers = []
    for _ in range(int(r.integers(2, 6))):
        if r.random() < 0.5:
            dim = pick([32, 48, 64, 80, 128])
            kv = pick([1, 2, 3])
            rot = pick([None] + [(d, pick([1000.0, 10000.0, 250000.0])) for d in (8, 32, 48, 64, 128) if d <= dim])
            mask = pick([None, (pick([5, 33, 64, 65, 100, 129]), pick([0, 1, 4, 31, 64, 70, 128]))])
            m = _att(kv * pick([1, 2, 4]), kv, dim, pick([32, 96, dim, dim]), float(dim ** -0.5 * r.uniform(0.7, 1.5)), rot=rot, mask=mask)
        else:
            groups = pick([1, 2, 3])
            heads = groups * pick([1, 2, 4])
            vdim = pick([8, 16, 20, 32, 64, 72])
            m = _ssd(heads, vdim, pick([8, 12, 16, 32, 64, 96, 128]), groups, pick([1, 2, 3, 4, 5]), pick([g for g in (1, 2, 4, 8) if heads * vdim % g == 0 and heads * vdim >= 8 * g]))
        mlp = pick([None, _ff(pick([136, 200])), _moe(pick([48, 64, 104]), pick([2, 4, 7, 16]), pick([1, 2]), pick([None, 24, 136])),
                    _moe(pick([40, 96]), pick([3, 8]), 3, pick([None, 64]))])
        layers.append((m, mlp))
    lo = int(r.integers(0, len(layers)))
    loop = pick([None, (lo, int(r.integers(lo, len(layers) + 1)), pick([1, 2, 3]))])
    return _model(layers, int(r.integers(150, 700)), pick([96, 128, 160, 224]), eps=pick([1e-5, 1e-6]), loop=loop)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 4, 9, 17, 23, 31, 44, 58])
def test_random_configuration(tmp_path, seed, dtype):
    from ithaca_b200 import Engine
    cfg = random_config(seed)
    t = make_tensors(cfg, 900 + seed)
    eng = Engine(_write(tmp_path, cfg, t, "m"), dtype=dtype, max_tokens=1024)
    V = cfg["vocab"]
    reqs = {"a": random_ids(230, V, seed * 7 + 1), "b": random_ids(90, V, seed * 7 + 2), "c": random_ids(31, V, seed * 7 + 3)}
    compare(eng, cfg, t, reqs, [[("a", 230)], [("b", 90)], [("c", 31)]], dtype)
    compare(eng, cfg, t, {"a": reqs["a"]}, [[("a", 190)]] + [[("a", 1)] for _ in range(40)], dtype)
    compare(eng, cfg, t, reqs, [[("a", 170), ("b", 50), ("c", 1)]] + [[("a", 1), ("b", 1), ("c", 1)] for _ in range(30)]
            + [[("a", 1), ("b", 1)] for _ in range(10)] + [[("a", 1)] for _ in range(20)], dtype)
    assert eng.cache.table.n_slots_in_use() == 0
    del eng
    torch.cuda.empty_cache()
