"""Seeded random Vovalorn configurations against the plain implementation: layer orders, borrowed tensors, head counts, key and value
sizes, roots, ranks, caps, temperatures, experts, groups and constants that no hand-written configuration of the other tests has,
among them sizes the tensor-core kernels take and sizes only the CUDA-core kernels take.  Every model runs whole prompts, a
prompt then decoded tokens, and an unequal batch decoded together with requests that end at different times, in both types (the
16-bit run against the plain implementation with the library's choice of experts, as in ``test_vovalorn_gpu.compare``)."""
import numpy as np
import pytest
import torch

from helpers import random_ids
from test_gunenex_gpu import _write
from test_vovalorn_gpu import _att, _gla, _model, _moe, _stored, compare, make_tensors

pytestmark = pytest.mark.gpu


def random_config(seed):
    r = np.random.default_rng(seed)
    pick = lambda xs: xs[int(r.integers(0, len(xs)))]
    layers = []
    for i in range(int(r.integers(3, 8))):
        if i and r.random() < 0.3:
            layers.append(int(r.integers(0, i)))
            continue
        if r.random() < 0.5:
            dim, kv = pick([16, 32, 48, 64, 80, 96, 128, 20]), pick([1, 2, 3, 4])
            m = _att(kv * pick([1, 2, 4]), kv, dim, float(dim ** -0.5 * r.uniform(0.7, 1.5)), pick([None, 10.0, 30.0, 50.0]),
                     pick([None, (float(r.uniform(-0.2, 0.5)), pick([7, 32, 64, 100]))]))
        else:
            m = _gla(pick([1, 2, 3, 4]), pick([16, 32, 40, 48, 64, 96]), pick([16, 32, 48, 64, 72, 96]), pick([1.0, 4.0, 16.0]), pick([3, 8, 16, 17]))
        count = pick([1, 2, 4])
        E = count * pick([1, 2, 3, 4])
        keep = int(r.integers(1, count + 1))
        top = int(r.integers(1, min(4, keep * (E // count)) + 1))
        layers.append((m, pick([None, _moe(pick([40, 64, 96]), E, top, pick([(count, keep), (count, keep), None]), float(r.uniform(0.5, 2.5)),
                                           pick([None, 24, 104]))])))
    return _model(layers, int(r.integers(150, 700)), pick([96, 128, 160, 224]), eps=pick([1e-5, 1e-6]), mult=float(r.uniform(0.3, 1.2)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 4, 9, 17, 23, 31, 44, 58])
def test_random_configuration(tmp_path, seed, dtype):
    from ithaca_b200 import Engine
    cfg = random_config(seed)
    t = make_tensors(cfg, 900 + seed)
    eng = Engine(_write(tmp_path, _stored(cfg), t, "m"), dtype=dtype, max_tokens=1024)
    V = cfg["vocab"]
    reqs = {"a": random_ids(230, V, seed * 7 + 1), "b": random_ids(90, V, seed * 7 + 2), "c": random_ids(31, V, seed * 7 + 3)}
    compare(eng, cfg, t, reqs, [[("a", 230)], [("b", 90)], [("c", 31)]], dtype)
    compare(eng, cfg, t, {"a": reqs["a"]}, [[("a", 190)]] + [[("a", 1)] for _ in range(40)], dtype)
    compare(eng, cfg, t, reqs, [[("a", 170), ("b", 50), ("c", 1)]] + [[("a", 1), ("b", 1), ("c", 1)] for _ in range(30)]
            + [[("a", 1), ("b", 1)] for _ in range(10)] + [[("a", 1)] for _ in range(20)], dtype)
    assert eng.cache.table.n_slots_in_use() == 0
    del eng
    torch.cuda.empty_cache()
