"""The Vovalorn decoder and its mechanisms against the plain implementation (tests/plain/vovalorn_plain.py).

Small configurations with weights made here.  Per mechanism: the kernel against the plain function, also across several
steps where it carries a state, and one-layer models of each mixer and of the feed-forward.  Whole models: prompts against
token-by-token decoding, portions down to two tokens, batches of unequal requests against each alone, slots, pages and states
that are used again, long decoding, and greedy generation through the engine's own loop.  Where random weights would hide a
fault (a far key, a key at a page's edge, a state that was lost on the way), the weights are made so that one token decides the
result.
"""
import copy
import json
import os

import numpy as np
import pytest
import torch

from helpers import REL, random_ids, rel_err, run_schedule
from plain import vovalorn_plain as P
from test_gunenex_gpu import SLOTS, STEPS, TOTAL, RouterTap, _close, _ctx, _write, rows_hold, SCHEDULES

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _gla(heads, dim, vdim, tau=16.0, rank=16):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def _att(heads, kv, dim, scale, softcap=50.0, temp=(0.3, 40)):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def _moe(ff, experts, top, groups=None, scale=1.0, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups is not None:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _model(layers, vocab, width, eps=1e-5, mult=0.7):
    """``layers``: (mixer, feed-forward) or the number of the layer whose tensors to run."""
    out = []
    for l in layers:
        if isinstance(l, int):
            out.append({**out[l], "weights_of": l})
        else:
            out.append({"type": "gla" if "tau" in l[0] else "attention", "mixer": l[0], "mlp": l[1]})
    return {"architecture": "Vovalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": out}


# unlike layers: recurrent sizes the chunk kernels take and do not take, a rank that is no multiple of four, groups of which some
# are kept and none at all, a layer without feed-forward, a temperature that rises within a page, tensors run three times
CFG_A = _model([
    (_att(4, 2, 32, 0.2, 20.0, (0.4, 9)), _moe(24, 8, 2, (4, 2), 1.5, shared=40)),
    (_gla(3, 48, 64, 4.0, 7), _moe(40, 6, 3, None, 0.7)),
    (_gla(2, 24, 10, 16.0, 16), None),
    1,
    (_att(6, 3, 64, 0.1, 50.0, (0.2, 64)), _moe(16, 9, 2, (3, 1), 2.0, shared=24)),
    0, 1,
], 101, 64)
# one head, one expert, no temperature, no cap; a group of one expert each; every expert chosen; no groups, no shared expert
CFG_B = _model([
    (_att(1, 1, 64, 0.15, None, None), _moe(32, 1, 1, shared=16)),
    (_gla(1, 64, 32, 1.0, 4), _moe(16, 3, 3, (3, 3), 2.5)),
    (_att(5, 5, 16, 0.3, 5.0, None), _moe(16, 4, 2, (4, 2))),
    0,
], 67, 48, eps=1e-6, mult=1.0)
# heads of 128 in groups of four, wide values and a wide key (two channels' worth of threads a block), a strong decay
CFG_C = _model([
    (_gla(2, 128, 96, 2.0, 24), _moe(48, 16, 4, (4, 3), 2.0, shared=72)),
    (_att(8, 2, 128, 0.09, 30.0, (0.1, 100)), None),
    (_gla(1, 16, 160, 16.0, 5), _moe(56, 4, 1, (2, 1), 1.0, shared=8)),
    1, 2,
], 89, 64, mult=0.4)
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C}


def make_tensors(cfg, seed):
    """Weights by name with the shapes the library asks for; scales chosen so that activations are of order one."""
    from ithaca_b200.config import config_from_dict
    from ithaca_b200.engine.model import weight_manifest
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, req in weight_manifest(config_from_dict(cfg)[1].model_spec()).items():
        shape = tuple(req.shape)
        r = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = r
        elif last == "alpha":
            t = 0.7 + 0.1 * r
        elif last.startswith("norm"):
            t = 1.0 + 0.2 * r
        elif last == "correction":
            t = 0.5 * r - 0.6                                     # some corrected scores are negative
        elif name.endswith("a2.b"):
            t = r + 1.0
        elif len(shape) == 1:                                     # the norms' offsets
            t = 0.1 * r
        elif last == "router":
            t = r * (3.0 / shape[1] ** 0.5)
        else:
            t = r * (1.2 / shape[1] ** 0.5)
        out[name] = t.bfloat16()
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("vovalorn")
    out = {}
    for i, (n, c) in enumerate(CONFIGS.items()):
        t = make_tensors(c, 50 + i)
        out[n] = (_write(root, _stored(c), t, n), t)
    return out


def _stored(cfg):
    """The file as a folder holds it: the ranks are left to the tensors."""
    c = copy.deepcopy(cfg)
    for l in c["layers"]:
        l["mixer"].pop("rank", None)
    return c


def _plain(cfg, t, ids):
    return P.forward(cfg, t, ids).numpy()


def run_tapped(eng, cfg, reqs, schedule):
    """As ``run_schedule``, and beside the logits, for every request, the experts the library used in each routed run."""
    n = sum(1 for l in cfg["layers"] if l["mlp"] is not None)
    used = {r: [[None] * len(ids) for _ in range(n)] for r, ids in reqs.items()}
    slots, fed, got = {}, {}, {}
    with RouterTap() as tap:
        for step in schedule:
            for r, _ in step:
                if r not in slots:
                    slots[r], fed[r] = eng.alloc_slot(), 0
            tap.calls.clear()
            lg = eng.step([slots[r] for r, _ in step], [reqs[r][fed[r]:fed[r] + k] for r, k in step], "all").cpu().numpy()
            assert len(tap.calls) == n
            chosen = [c.cpu().tolist() for c in tap.calls]
            off = 0
            for r, k in step:
                got.setdefault(r, np.zeros((len(reqs[r]), lg.shape[1]), dtype=np.float32))[fed[r]:fed[r] + k] = lg[off:off + k]
                for j in range(n):
                    used[r][j][fed[r]:fed[r] + k] = chosen[j][off:off + k]
                off += k
                fed[r] += k
                if fed[r] == len(reqs[r]):
                    eng.free_slot(slots.pop(r))
    eng.check_status()
    return got, {r: [torch.tensor(u, dtype=torch.long) for u in us] for r, us in used.items()}


def compare(eng, cfg, t, reqs, schedule, dtype):
    """Runs the schedule and holds every request's logits against the plain implementation.  float32: as it is, every row within
    the tolerance.  bfloat16: two experts whose scores lie close change places under 16-bit operands, so that run is held
    against the plain implementation made to use the experts the library chose (which experts are the right ones is what the
    float32 run and the routing kernels' own test check)."""
    if dtype == "float32":
        got = run_schedule(eng, reqs, schedule)
        for r, ids in reqs.items():
            assert _close(got[r], _plain(cfg, t, ids)), (r, rel_err(got[r], _plain(cfg, t, ids)))
        return got
    got, used = run_tapped(eng, cfg, reqs, schedule)
    for r, ids in reqs.items():
        assert rows_hold(got[r], P.forward(cfg, t, ids, forced=used[r]).numpy()), r
    return got


# ------------------------------------------------------------------------------------------ the norm
def _norm(d, g, alpha):
    w, b = 1 + 0.3 * torch.randn(d, generator=g), 0.5 * torch.randn(d, generator=g)
    return (w.to(DEV), b.to(DEV), alpha), {"n": w.double(), "n.b": b.double(), "n.alpha": torch.tensor(alpha, dtype=torch.float64)}


@pytest.mark.parametrize("d", [4, 30, 64, 1031, 4096])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_dynamic_tanh_kernels(d, dtype):
    """In front of a sublayer (all rows and picked rows), behind the embedding, behind a sublayer with and without the next norm,
    and on experts' results that are not added up yet."""
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(d)
    n, pn = _norm(d, g, 0.8)
    n2, pn2 = _norm(d, g, -1.7)
    T, top = 7, 3
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    err = lambda a, b: rel_err(a.float().cpu().numpy(), b.numpy())
    x = torch.randn(T, d, generator=g) * torch.logspace(-3, 1.5, T)[:, None]
    assert err(ops.dynamic_tanh(x.to(DEV), n, dtype), P.dynamic_tanh(x.double(), pn, "n")) < tol
    rows = torch.tensor([5, 0, 5], dtype=torch.int32)
    assert err(ops.dynamic_tanh(x.to(DEV), n, dtype, rows_in=rows.to(DEV)), P.dynamic_tanh(x.double(), pn, "n")[rows.long()]) < tol
    table = torch.randn(11, d, generator=g).to(dtype)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    ids = torch.tensor([3, 10, 0, 3], dtype=torch.int32)
    assert err(ops.dynamic_tanh_embed(ids.to(DEV), table.to(DEV), n, 1.5, status), P.dynamic_tanh(table[ids.long()].double() * 1.5, pn, "n")) < 2e-6
    assert status.item() == 0
    ops.dynamic_tanh_embed(torch.tensor([3, 11], dtype=torch.int32, device=DEV), table.to(DEV), n, 1.0, status)
    assert status.item() == 1                                          # an id outside the table is reported, not followed
    res = torch.randn(T, d, generator=g)
    parts, w = torch.randn(T * top + 4, d, generator=g), torch.randn(T, top, generator=g)
    row_of = torch.randperm(T * top + 4, generator=g)[:T * top].to(torch.int32)
    ex, ew = torch.randn(T, d, generator=g), torch.randn(T, generator=g)
    summed = (parts[row_of.long()].view(T, top, d).double() * w.double()[:, :, None]).sum(1)
    dev = lambda v: v.to(DEV)
    for y, py in ((x.to(DEV), x.double()), (ops.ExpertSum(dev(parts), dev(w), dev(row_of), False, dev(ex), dev(ew)), summed + ex.double() * ew.double()[:, None]),
                  (ops.ExpertSum(dev(parts), dev(w), dev(row_of)), summed),
                  (ops.ExpertSum(dev(parts[:T * top].contiguous()), dev(w), None, True, dev(ex)), parts[:T * top].view(T, top, d).double().sum(1) + ex.double())):
        for nxt in (None, n2):
            r = res.to(DEV)
            copy_ = ops.dynamic_tanh_add(y, n, r, 0.6, nxt, dtype)
            want = res.double() + 0.6 * P.dynamic_tanh(py, pn, "n")
            assert err(r, want) < 2e-6 and (copy_ is None) == (nxt is None)
            if nxt is not None:
                assert copy_.dtype == dtype and err(copy_, P.dynamic_tanh(want, pn2, "n")) < max(tol, 1e-5)


# ------------------------------------------------------------------------------------------ the router
@pytest.mark.parametrize("E,top,groups,K,T", [(16, 4, (4, 3), 64, 70), (8, 2, (4, 1), 48, 5), (12, 3, (2, 1), 256, 9), (6, 2, (6, 3), 32, 40),
                                              (10, 10, (2, 2), 128, 3), (9, 2, None, 30, 65), (160, 6, (8, 3), 2052, 130), (64, 8, (1, 1), 64, 300)])
def test_choice_by_corrected_scores_within_the_best_groups(E, top, groups, K, T):
    """Choice and weights from the fused kernel and from ready-made logits; the correction makes scores negative and decides
    choices, and a group's two best count together."""
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(E + T)
    x, wr, c = torch.randn(T, K, generator=g), torch.randn(E, K, generator=g) * 2 / K ** 0.5, torch.randn(E, generator=g) * 0.6 - 1.0
    r = {"experts": E, "top": top, "scale": 2.5}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    z = x.double() @ wr.double().T
    s = P.sigmoid(z)
    e = P.choose(s, c.double(), r)
    w = P.weigh(s, e, r)
    kw = dict(n_groups=groups[0] if groups else 0, keep=groups[1] if groups else 0, renorm=True, score="sigmoid", correction=c.to(DEV),
              group_score="best_two", weight_eps=1e-20, weight_scale=2.5)
    got = ops.moe_router(x.to(DEV), wr.to(DEV), top, **kw)
    assert (got is None) == (K % 4 != 0)
    for chosen, weight in ([got] if got is not None else []) + [ops.moe_route(z.float().to(DEV), top, **kw)]:
        order, porder = chosen.cpu().long().sort(1), e.sort(1)
        assert torch.equal(order.values, porder.values)
        assert rel_err(weight.cpu().gather(1, order.indices).numpy(), w.gather(1, porder.indices).numpy()) < 1e-5
    if top < E:
        assert not torch.equal(P.choose(s, torch.zeros(E), r).sort(1).values, e.sort(1).values)
    if groups and groups[0] > 1 and E // groups[0] > 1 and groups[1] < groups[0]:
        best = ops.moe_route(z.float().to(DEV), top, **{**kw, "group_score": "best"})[0].cpu().long()
        assert not torch.equal(best.sort(1).values, e.sort(1).values)


# ------------------------------------------------------------------------------------------ the recurrence
@pytest.mark.parametrize("rank,C,T", [(1, 5, 3), (16, 192, 70), (7, 300, 130), (130, 64, 1), (64, 256, 65)])
def test_decays_from_a_low_rank_factor(rank, C, T):
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(rank)
    p, w, b = torch.randn(T, rank + 9, generator=g), torch.randn(C, rank, generator=g) * 3 / rank ** 0.5, torch.randn(C, generator=g) * 8
    z = p[:, 5:5 + rank].double() @ w.double().T + b.double()
    for tau in (16.0, 0.7):
        want = P.channel_decay(z, tau)
        args = (p.to(DEV), 5, w.t().contiguous().to(DEV), b.to(DEV), 1 / tau)
        assert float((ops.lowrank_decay(*args).cpu().double() - want).abs().max()) < 3e-6
        log2 = torch.log2(want.clamp_min(1e-300))
        assert float(((ops.lowrank_decay(*args, log2=True).cpu().double() - log2).abs() / (1 + log2.abs())).max()) < 1e-5
    assert float(want.min()) < 1e-4 and float(want.max()) > 0.99


def _gla_case(H, K, V, n, seed, strong):
    g = torch.Generator().manual_seed(seed)
    u = torch.randn(n, 2 * H * K + 2 * H * V + 4, generator=g)
    return u, -torch.rand(n, H * K, generator=g) ** 2 * strong          # log2 of the decays


def _gla_plain(u, log2, H, K, V, scale, state):
    n, u = u.shape[0], u[:, 4:].double()
    q, k, v = u[:, :H * K].view(n, H, K) * scale, u[:, H * K:2 * H * K].view(n, H, K), u[:, 2 * H * K:2 * H * K + H * V].view(n, H, V)
    return (*P.gla(q, k, v, torch.exp2(log2.double()).view(n, H, K), state), u[:, 2 * H * K + H * V:])


GLA_SIZES = [(4, 24, 40), (3, 80, 16), (1, 16, 32), (2, 64, 128), (2, 200, 8), (3, 48, 64), (1, 128, 256), (2, 112, 160), (2, 64, 96), (1, 300, 7)]


@pytest.mark.parametrize("strong", [0.3, 6.0, 40.0])
@pytest.mark.parametrize("H,K,V", GLA_SIZES)
def test_gated_linear_attention_kernels(H, K, V, strong):
    """Token by token and by chunks, across four steps of three sequences in scattered slots with leftovers in their states, from
    decays that hardly forget to ones that forget within a token (where a block's own columns are formed directly)."""
    from ithaca_b200.csrc import ops
    scale, eps = K ** -0.5, 1e-5
    nw = 1 + 0.3 * torch.randn(V, generator=torch.Generator().manual_seed(V))
    data = [_gla_case(H, K, V, n, 7 + b, strong) for b, n in enumerate(TOTAL)]
    states = [torch.randn(5, 2, H, V, K, device=DEV) for _ in range(2)]
    plain = [None] * 3
    takes = K % 16 == 0 and K <= 128 and V % 32 == 0
    for lo, hi in STEPS:
        ctx = _ctx(lo, hi, SLOTS)
        u = torch.cat([data[b][0][lo[b]:hi[b]] for b in range(3)]).to(DEV)
        log2 = torch.cat([data[b][1][lo[b]:hi[b]] for b in range(3)]).to(DEV)
        o = ops.row_decay("plain", u[:, 4:], 0, H * K, 2 * H * K, torch.exp2(log2), None, None, states[0], ctx, H, H, K, V, scale).cpu().double()
        mid = ops.gla_chunks(u[:, 4:], 0, H * K, 2 * H * K, 2 * H * K + H * V, log2, states[1], ctx, H, K, V, nw.to(DEV), eps, scale)
        assert (mid is not None) == takes
        at = 0
        for b in range(3):
            n = hi[b] - lo[b]
            want, S, gate = _gla_plain(data[b][0][lo[b]:hi[b]], data[b][1][lo[b]:hi[b]], H, K, V, scale, plain[b])
            plain[b] = S
            assert float((o[at:at + n].view(n, H, V) - want).abs().max() / want.abs().max()) < 5e-6
            want = (P.rms(want, eps) * nw.double()).reshape(n, H * V) * P.silu(gate)
            for st, tol in zip(states, (5e-6, 4e-5)):
                if st is states[0] or takes:
                    got = st[SLOTS[b], (hi[b] - 1) & 1].cpu().double().transpose(1, 2)
                    assert float((got - S).abs().max() / S.abs().max()) < tol
            if takes:
                assert rel_err(mid[at:at + n].float().cpu().numpy(), want.numpy()) < 6e-3
            at += n


@pytest.mark.parametrize("H,K,V,rank", [(4, 24, 40, 7), (3, 80, 16, 16), (1, 16, 32, 1), (2, 64, 128, 16), (2, 200, 8, 33), (2, 300, 24, 5), (16, 48, 64, 64), (1, 4, 300, 3),
                                        (2, 128, 256, 16)])
def test_the_decode_kernel_with_its_decay_norm_and_gate(H, K, V, rank):
    """Token by token from position 0 in slots with leftovers; running a step twice changes nothing (a captured graph does)."""
    from ithaca_b200.csrc import ops
    n, slots, scale, eps = 12, [2, 0], K ** -0.5, 1e-5
    g = torch.Generator().manual_seed(K)
    a_off = 4 + 2 * H * K + 2 * H * V
    rows = [torch.randn(n, a_off + rank + 2, generator=g) for _ in slots]
    a2, b2, nw = torch.randn(rank, H * K, generator=g) * rank ** -0.5, torch.randn(H * K, generator=g) * 3, 1 + 0.3 * torch.randn(V, generator=g)
    state = torch.randn(3, 2, H, V, K, device=DEV)
    want = []
    for b in range(2):
        log2 = torch.log2(P.channel_decay(rows[b][:, a_off:a_off + rank].double() @ a2.double() + b2.double(), 3.0))
        o, S, gate = _gla_plain(rows[b][:, :a_off], log2, H, K, V, scale, None)
        want.append(((P.rms(o, eps) * nw.double()).reshape(n, H * V) * P.silu(gate), S))
    for i in range(n):
        p = torch.stack([r[i] for r in rows]).to(DEV)
        for _ in range(2):
            y = ops.gla_decode(p, 4, 4 + H * K, 4 + 2 * H * K, 4 + 2 * H * K + H * V, a_off, a2.to(DEV), b2.to(DEV), 1 / 3.0, state, _ctx([i, i], [i + 1, i + 1], slots),
                               H, K, V, nw.to(DEV), eps, scale)
        for b in range(2):
            assert rel_err(y[b].float().cpu().numpy(), want[b][0][i].numpy()) < 6e-3, (i, b)
    for b in range(2):
        assert rel_err(state[slots[b], (n - 1) & 1].cpu().transpose(1, 2).numpy(), want[b][1].numpy()) < 1e-5


def test_the_decode_kernel_declines_odd_key_sizes():
    from ithaca_b200.csrc import ops
    z = lambda *s: torch.zeros(*s, device=DEV)
    assert ops.gla_decode(z(1, 24), 0, 6, 12, 16, 20, z(1, 6), z(6), 1.0, z(1, 2, 1, 4, 6), _ctx([0], [1], [0]), 1, 6, 4, z(4), 1e-6, 1.0) is None


@pytest.mark.parametrize("strong", [0.05, 1.0])
def test_long_prompts_in_chunks_against_token_by_token(strong):
    """Prompts of several chunks with a ragged end, three sequences, a portion behind each, many heads at once; the states of
    the two ways and what the read-outs come to."""
    from ithaca_b200.csrc import ops
    H, K, V = 16, 64, 128
    ends = [1000, 389, 64]
    data = [_gla_case(H, K, V, n, 3 + b, strong) for b, n in enumerate(ends)]
    nw = torch.ones(V, device=DEV)
    states = [torch.randn(3, 2, H, V, K, generator=torch.Generator().manual_seed(1)).to(DEV) for _ in range(2)]
    for lo, hi in (([0, 0, 0], [700, 256, 1]), ([700, 256, 1], ends)):
        ctx = _ctx(lo, hi, [1, 2, 0])
        u = torch.cat([data[b][0][lo[b]:hi[b]] for b in range(3)]).to(DEV)[:, 4:]
        log2 = torch.cat([data[b][1][lo[b]:hi[b]] for b in range(3)]).to(DEV)
        got = ops.gla_chunks(u, 0, H * K, 2 * H * K, 2 * H * K + H * V, log2, states[0], ctx, H, K, V, nw, 1e-6, K ** -0.5)
        o = ops.row_decay("plain", u, 0, H * K, 2 * H * K, torch.exp2(log2), None, None, states[1], ctx, H, H, K, V, K ** -0.5)
        want = ops.head_norm_gate(o, nw, 1e-6, u, 2 * H * K + H * V, H, torch.float32)
        assert rel_err(got.float().cpu().numpy(), want.cpu().numpy()) < 4e-3
        for b in range(3):
            a, w = (st[[1, 2, 0][b], (hi[b] - 1) & 1].cpu().numpy() for st in states)
            assert rel_err(a, w) < 4e-5


def test_the_token_loop_gives_the_same_bits_however_it_is_cut():
    from ithaca_b200.csrc import ops
    H, K, V, n = 3, 40, 24, 90
    u, log2 = (v.to(DEV) for v in _gla_case(H, K, V, n, 2, 0.5))
    dec = torch.exp2(log2)

    def run(cuts):
        state = torch.zeros(1, 2, H, V, K, device=DEV)
        ys = [ops.row_decay("plain", u[a:b], 4, 4 + H * K, 4 + 2 * H * K, dec[a:b].contiguous(), None, None, state, _ctx([a], [b], [0]), H, H, K, V, 0.3)
              for a, b in zip(cuts, cuts[1:])]
        return torch.cat(ys), state[0, (n - 1) & 1].clone()
    y, S = run([0, n])
    for cuts in ([0, 1, 3, 16, 17, 64, n], list(range(n + 1))):
        y2, S2 = run(cuts)
        assert torch.equal(y, y2) and torch.equal(S, S2)


# ------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,scales", [(6, 3, 32, True), (4, 1, 10, True), (3, 3, 64, False), (8, 2, 300, True), (2, 1, 6, False)])
def test_unit_norm_temperature_and_append(nh, nkv, hd, scales, dtype):
    """q normed per head and warmed up by its position; k either normed beside its values or stored as projected with a number
    beside it; both at every place of scrambled pages."""
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(hd)
    lens, new = [1, 130, 66], [1, 70, 3]
    T, pad = sum(new), 4
    p = torch.randn(T, pad + (nh + 2 * nkv) * hd, generator=g)
    p[2] *= 1e-3                                                       # eps matters
    tab = torch.tensor([[4, -1, -1], [0, 6, 2], [5, 1, -1]], dtype=torch.int32)
    seq = torch.tensor(np.repeat([0, 1, 2], new), dtype=torch.int32)
    pos = torch.tensor(np.concatenate([np.arange(l - n, l) for l, n in zip(lens, new)]), dtype=torch.int32)
    k = torch.zeros(7, nkv, 64, hd, dtype=dtype, device=DEV)
    v = None if scales else torch.zeros_like(k)
    ks = torch.zeros(7, nkv, 64, device=DEV) if scales else None
    q = torch.empty(T, nh * hd, dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.norm_rope_append(p.to(DEV)[:, pad:], 0, nh * hd, (nh + nkv) * hd, None, None, 1e-5, q, k, v, seq.to(DEV), pos.to(DEV), tab.to(DEV), None, 1.0,
                         nh, 0, 0, True, status, unit=True, q_temp=(0.4, 30), key_scales=ks)
    assert status.item() == 0
    x = p[:, pad:].double()
    pq, pk, pv = x[:, :nh * hd].view(T, nh, hd), x[:, nh * hd:(nh + nkv) * hd].view(T, nkv, hd), x[:, (nh + nkv) * hd:].view(T, nkv, hd)
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    want = P.rms(pq, 1e-5) * P.temperature(pos.long(), 0.4, 30)[:, None, None]
    assert rel_err(q.float().cpu().view(T, nh, hd).numpy(), want.numpy()) < tol
    page, place = tab[seq.long(), pos.long() // 64].long(), pos.long() % 64
    kept = k.float().cpu()[page, :, place]
    if scales:
        assert rel_err(kept.numpy(), pk.numpy()) < tol
        assert rel_err(ks.cpu()[page, :, place].numpy(), (pk.pow(2).mean(-1) + 1e-5).rsqrt().numpy()) < 2e-6
    else:
        assert rel_err(kept.numpy(), P.rms(pk, 1e-5).numpy()) < tol and rel_err(v.float().cpu()[page, :, place].numpy(), pv.numpy()) < tol


def _paged_case(nh, nkv, hd, lens, new, dtype, seed, scale, cap, one_row, loud=()):
    """Random rows of sequences in scrambled pages; the last ``new[b]`` positions of each are the step's queries.  ``one_row``: a
    row is key (times a number of its own) and value.  ``loud``: at these distances from the end keys that the last query likes."""
    from test_kernels_gpu import Paged
    g = torch.Generator().manual_seed(seed)
    qs = [torch.randn(l, nh, hd, generator=g).to(dtype) for l in lens]
    ks = [(torch.randn(l, nkv, hd, generator=g) * (1 + 3 * torch.rand(l, nkv, 1, generator=g))).to(dtype) for l in lens]
    for q, k, l in zip(qs, ks, lens):
        for d in loud:
            if l - 1 - d >= 0:
                k[l - 1 - d] = q[l - 1, ::nh // nkv] * 1.5
    vs = ks if one_row else [torch.randn(l, nkv, hd, generator=g).to(dtype) for l in lens]
    cs = [(k.double().pow(2).mean(-1) + 1e-6).rsqrt().float() if one_row else torch.ones(k.shape[:2]) for k in ks]
    pk, pv, pc = Paged(lens, nkv, hd, dtype, seed), Paged(lens, nkv, hd, dtype, seed), Paged(lens, nkv, 1, torch.float32, seed)
    pk.fill(ks, ks), pv.fill(vs, vs), pc.fill([c[..., None] for c in cs], [c[..., None] for c in cs])
    ref = torch.cat([P.attention_core(q[l - n:].double(), k.double() * c.double()[..., None], v.double(), scale, cap, l - n)
                     for q, k, v, c, l, n in zip(qs, ks, vs, cs, lens, new)]).reshape(sum(new), nh * hd)
    i32 = lambda a: torch.from_numpy(np.asarray(a).astype(np.int32)).to(DEV)
    return dict(q=torch.cat([q[l - n:] for q, l, n in zip(qs, lens, new)]).reshape(sum(new), nh * hd).to(DEV), k=pk.dev()[0],
                v=None if one_row else pv.dev()[0], c=pc.dev()[0][..., 0].contiguous() if one_row else None, tab=pk.dev()[2], ref=ref,
                seq=i32(np.repeat(np.arange(len(lens)), new)), pos=i32(np.concatenate([np.arange(l - n, l) for l, n in zip(lens, new)])),
                cu=i32(np.concatenate([[0], np.cumsum(new)])), lens=i32(lens), slopes=torch.tensor(P.slopes(nh), dtype=torch.float32, device=DEV))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd", [(4, 2, 16), (3, 1, 40), (8, 8, 10)])
@pytest.mark.parametrize("cap,one_row", [(0.0, True), (3.0, True), (20.0, False)])
def test_the_cuda_core_attention(dtype, nh, nkv, hd, cap, one_row):
    from ithaca_b200.csrc import ops
    lens, new = [1, 70, 300, 129, 64, 500], [1, 70, 170, 1, 64, 3]
    c = _paged_case(nh, nkv, hd, lens, new, dtype, 40, 0.7, cap, one_row)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    got = ops.attention_simt(c["q"], c["k"], c["v"], c["seq"], c["pos"], c["tab"], nh, 0.7, 0, status, softcap=cap, key_scales=c["c"], slopes=c["slopes"],
                             values_in_keys=hd if one_row else 0)
    assert status.item() == 0
    assert rel_err(got.float().cpu().numpy(), c["ref"].numpy()) < (3e-6 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("nh,nkv,hd,kind", [(4, 4, 16, "mma"), (6, 2, 48, "mma"), (8, 2, 64, "tc"), (8, 4, 128, "tc"), (6, 2, 128, "mma"), (20, 1, 64, "tc")])
@pytest.mark.parametrize("cap,one_row,slopes", [(0.0, True, True), (50.0, True, True), (1.5, True, True), (8.0, False, True), (30.0, True, False)])
def test_the_tensor_core_attention(nh, nkv, hd, kind, cap, one_row, slopes):
    """Prefill (both kernels) and decode with chunks of one to four pages; caps that scores hardly feel and caps they all run
    into; rows that are keys and values and rows that are keys alone; with and without a bias."""
    from ithaca_b200.csrc import attention_bf16 as A
    scale = 3.0 / hd ** 0.5
    lens, new = [1, 70, 300, 129, 64, 700], [1, 70, 67, 129, 5, 450]
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    if not slopes:
        ref_slopes, P_slopes = [0.0] * nh, P.slopes
        P.slopes = lambda n: ref_slopes
    try:
        c = _paged_case(nh, nkv, hd, lens, new, torch.bfloat16, 41, scale, cap, one_row)
        d = _paged_case(nh, nkv, hd, lens, [1] * len(lens), torch.bfloat16, 42, scale, cap, one_row)
    finally:
        if not slopes:
            P.slopes = P_slopes
    extra = dict(softcap=cap, key_scales=c["c"], slopes=c["slopes"] if slopes else None)
    got = A.prefill(c["q"], c["k"], c["v"], c["cu"], c["lens"], c["tab"], len(lens), max(new), nh, scale, 0, status, kind=kind, **extra)
    assert status.item() == 0
    assert rel_err(got.float().cpu().numpy(), c["ref"].numpy()) < 8e-3
    extra["key_scales"] = d["c"]
    for chunk in (1, 2, 4):
        got = A.decode(d["q"], d["k"], d["v"], d["lens"], d["tab"], len(lens), 1000, nh, scale, 0, status, chunk_pages=chunk, **extra)
        assert status.item() == 0
        assert rel_err(got.float().cpu().numpy(), d["ref"].numpy()) < 8e-3


@pytest.mark.parametrize("nh,nkv,hd,kind", [(8, 8, 32, "mma"), (8, 2, 64, "tc"), (16, 4, 128, "tc"), (40, 2, 64, "tc")])
@pytest.mark.parametrize("temp", [None, (0.5, 100), (-0.4, 50)])
def test_keys_the_bias_makes_negligible_are_not_visited(nh, nkv, hd, kind, temp):
    """A known bound on the scores lets steep heads stop early: the result is the one of visiting every key, also where the last
    query likes keys at the edge of what a head can reach."""
    from ithaca_b200.csrc import attention_bf16 as A
    scale = 8.0 / hd
    lens, new = [1, 900, 2100, 65], [1, 130, 2, 65]
    c = _paged_case(nh, nkv, hd, lens, new, torch.bfloat16, 44, scale, 20.0, True, loud=(0, 1, 64, 100, 200, 500, 1000, 2000))
    unit = c["q"].float().view(-1, nh, hd)                             # queries as the mixer makes them: of a known length
    warm = P.temperature(c["pos"].cpu().long(), *temp).float().to(DEV) if temp else torch.ones(len(c["pos"]), device=DEV)
    q = (unit / unit.pow(2).mean(-1, keepdim=True).sqrt() * warm[:, None, None]).bfloat16().reshape(c["q"].shape)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    reach = (scale * hd * 1.02,) + (temp or (0.0, 0))
    args = (q, c["k"], None, c["cu"], c["lens"], c["tab"], len(lens), max(new), nh, scale, 0, status)
    extra = dict(softcap=20.0, key_scales=c["c"], slopes=c["slopes"])
    all_, near = (A.prefill(*args, kind=kind, **extra, reach=r).float().cpu() for r in (None, reach))
    # (the tcgen05 kernel's weights are rounded to 16 bits against a reference that depends on the pages walked)
    assert rel_err(near.numpy(), all_.numpy()) < (3e-3 if kind == "tc" else 1e-4)
    last = torch.tensor(np.cumsum(new) - 1)
    args = (q[last.to(DEV)].contiguous(), c["k"], None, c["lens"], c["tab"], len(lens), 3000, nh, scale, 0, status)
    for chunk in (1, 4):
        all_, near = (A.decode(*args, chunk_pages=chunk, **extra, reach=r).float().cpu() for r in (None, reach))
        assert rel_err(near.numpy(), all_.numpy()) < 1e-4
    # pages further back than any head of the steepest group reaches are not even looked up
    if temp is None and nkv == nh:
        tab = c["tab"].clone()
        one = c["slopes"].clone()
        one[:] = 0.5
        tab[2, :20] = -1                                               # 2100 positions, slope 1/2: about 70 keys back
        A.decode(args[0], c["k"], None, c["lens"], tab, len(lens), 3000, nh, scale, 0, status, softcap=20.0, key_scales=c["c"], slopes=one, reach=reach)
        assert status.item() == 0
        A.decode(args[0], c["k"], None, c["lens"], tab, len(lens), 3000, nh, scale, 0, status, softcap=20.0, key_scales=c["c"], slopes=one)
        assert status.item() != 0


def test_modules_decline_what_they_were_not_compiled_for():
    from ithaca_b200.csrc import attention_bf16 as A
    assert A.module(64) is not A.module(64, True, True)
    with pytest.raises(Exception, match="slope"):
        A.decode(torch.zeros(1, 64, dtype=torch.bfloat16, device=DEV), torch.zeros(1, 1, 64, 64, dtype=torch.bfloat16, device=DEV), None,
                 torch.ones(1, dtype=torch.int32, device=DEV), torch.zeros(1, 1, dtype=torch.int32, device=DEV), 1, 64, 1, 1.0, 0, None,
                 slopes=torch.zeros(2, device=DEV))


# ------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,ff,E,top,groups,shared,T", [(64, 24, 8, 2, (4, 2), 40, 9), (48, 40, 1, 1, None, None, 3), (128, 96, 16, 4, (4, 3), 64, 300),
                                                        (72, 16, 3, 3, (3, 3), 200, 1), (256, 64, 12, 3, (2, 1), 72, 1500), (30, 7, 4, 2, (2, 2), 21, 20)])
def test_routed_feed_forward(dtype, d, ff, E, top, groups, shared, T):
    from ithaca_b200.config import config_from_dict
    from ithaca_b200.csrc import ops
    from ithaca_b200.parts import FEED_FORWARDS, Runtime
    fc = _moe(ff, E, top, groups, 1.7, shared)
    cfg = _model([(_gla(1, 16, 8), fc)], 13, d)
    t = make_tensors(cfg, 3)
    rt = Runtime(dtype, DEV)
    part = FEED_FORWARDS.get("moe")(config_from_dict(cfg)[1].model_spec().layers[0].feed_forward, t, rt)
    x = torch.randn(T, d, generator=torch.Generator().manual_seed(2)).bfloat16()
    res = torch.zeros(T, d, device=DEV)
    with RouterTap() as tap:
        part.forward(x.to(DEV).to(rt.act_dtype), None, res, accumulate=False)
        y = part.unsummed(x.to(DEV).to(rt.act_dtype), None)
    chosen = tap.calls[0].cpu().long()
    want = P.moe_ff(x.double(), fc, {k: v.double() for k, v in t.items()}, "l0.mlp.", chosen)
    assert rel_err(res.cpu().numpy(), want.numpy()) < (REL["float32"] if dtype == "float32" else 1.5e-2)
    again = ops.moe_combine(y.parts, y.weight, row_of=y.row_of, unweighted=y.unweighted, extra=y.extra, extra_weight=y.extra_weight)
    assert torch.equal(again, res)
    free = P.choose(P.sigmoid(x.double() @ t["l0.mlp.router"].double().T), t["l0.mlp.correction"], fc["router"])
    same = (chosen.sort(1).values == free.sort(1).values).all(1).double().mean()
    assert same == 1.0 if dtype == "float32" else same > 0.98


# ------------------------------------------------------------------------------------------ one-layer models
ONE_LAYER = {
    "recurrence": _model([(_gla(4, 32, 32, 8.0, 5), None)], 53, 48),
    "recurrence, no tensor-core sizes": _model([(_gla(3, 10, 6, 16.0, 3), None)], 53, 48),
    "recurrence, forgets within a token": _model([(_gla(2, 64, 64, 0.2, 16), None)], 53, 64, mult=1.3),
    "attention": _model([(_att(4, 2, 16, 0.25, 8.0, (0.3, 20)), None)], 53, 48),
    "attention, tcgen05 sizes": _model([(_att(4, 1, 64, 0.12, 50.0, (0.5, 64)), _moe(40, 4, 2, (2, 1), 1.2))], 53, 64),
    "attention, neither cap nor temperature": _model([(_att(3, 3, 8, 0.4, None, None), None)], 53, 48),
    "attention, cools down": _model([(_att(2, 2, 32, 0.2, 50.0, (-0.5, 16)), None)], 53, 48),
    "routed and shared": _model([(_gla(1, 16, 8), _moe(24, 8, 2, (4, 2), 2.0, shared=16))], 53, 48),
    "routed": _model([(_att(2, 1, 24, 0.3), _moe(24, 4, 4))], 53, 48),
    "the same tensors four times": _model([(_gla(2, 16, 32, 4.0, 9), _moe(24, 3, 1)), 0, 0, 0], 53, 48),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ONE_LAYER))
def test_one_layer_models(tmp_path, name, dtype):
    from ithaca_b200 import Engine
    cfg = ONE_LAYER[name]
    t = make_tensors(cfg, 11)
    eng = Engine(_write(tmp_path, _stored(cfg), t, "one"), dtype=dtype, max_tokens=1024)
    reqs = {"a": random_ids(150, 53, 1), "b": random_ids(9, 53, 2)}
    compare(eng, cfg, t, reqs, [[("a", 150), ("b", 9)]], dtype)
    compare(eng, cfg, t, reqs, [[("a", 70), ("b", 2)], [("a", 3), ("b", 1)]] + [[("a", 1), ("b", 1)]] * 6 + [[("a", 71)]], dtype)


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts(models, name, dtype):
    from ithaca_b200 import Engine
    d, t = models[name]
    eng = Engine(d, dtype=dtype, max_tokens=2048)
    for n in (1, 2, 63, 64, 65, 300):
        compare(eng, CONFIGS[name], t, {"a": random_ids(n, CONFIGS[name]["vocab"], n)}, [[("a", n)]], dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sched", list(SCHEDULES))
@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_same_logits_however_a_prompt_is_cut(models, name, sched, dtype):
    from ithaca_b200 import Engine
    d, t = models[name]
    n = 220
    ids = random_ids(n, CONFIGS[name]["vocab"], 7)
    eng = Engine(d, dtype=dtype, max_tokens=1024)
    got = compare(eng, CONFIGS[name], t, {"a": ids}, SCHEDULES[sched](n), dtype)["a"]
    if dtype == "float32":
        whole = run_schedule(eng, {"a": ids}, [[("a", n)]])["a"]
        assert np.array_equal(got, whole)                              # every sum runs in an order of its own, whatever the step


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_batches_against_each_request_alone(models, name, dtype):
    """Requests of 1 to 260 tokens start together and are decoded together; the short ones end earlier.  Then portions of
    some beside single tokens of others."""
    from ithaca_b200 import Engine
    d, t = models[name]
    V = CONFIGS[name]["vocab"]
    reqs = {r: random_ids(n, V, 40 + n) for r, n in (("a", 1), ("b", 66), ("c", 260), ("d", 13), ("e", 130))}
    eng = Engine(d, dtype=dtype, max_tokens=2048)
    first = {"a": 1, "b": 60, "c": 250, "d": 9, "e": 126}
    sched = [[(r, first[r]) for r in reqs]]
    left = {r: len(reqs[r]) - first[r] for r in reqs}
    while any(left.values()):
        sched.append([(r, 1) for r in reqs if left[r] > 0])
        left = {r: max(0, n - 1) for r, n in left.items()}
    compare(eng, CONFIGS[name], t, reqs, sched, dtype)
    mixed = [[("c", 64), ("b", 1)], [("c", 65), ("b", 2), ("e", 7)], [("b", 63), ("c", 1), ("e", 1)], [("c", 130), ("e", 122)]]
    got = compare(eng, CONFIGS[name], t, {r: reqs[r] for r in "bce"}, mixed, dtype)
    if dtype == "float32":
        alone = run_schedule(eng, {"c": reqs["c"]}, [[("c", 260)]])["c"]
        assert np.array_equal(got["c"], alone)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_pages_and_states_are_used_again(models, dtype):
    """A small cache: requests come and go, so slots, pages, key scales and states are handed out again, also to shorter
    sequences whose first tokens must see nothing of what lay there before."""
    from ithaca_b200 import Engine
    for name, pages in (("A", 6), ("C", 8)):
        d, t = models[name]
        cfg, V = CONFIGS[name], CONFIGS[name]["vocab"]
        eng = Engine(d, dtype=dtype, max_tokens=64 * pages, max_slots=2)
        for round_ in range(4):
            reqs = {"x": random_ids(230 - 60 * round_, V, 20 + round_), "y": random_ids(3 + round_, V, 30 + round_)}
            compare(eng, cfg, t, reqs, [[("x", len(reqs["x"]) - 2), ("y", 2)], [("x", 1), ("y", 1)], [("x", 1)]] + [[("y", 1)] for _ in range(round_)],
                    dtype)
            eng.cache.table.check_consistent()
            assert all(p.held() == 0 for p in eng.cache.table.pools)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(models, name, dtype):
    from ithaca_b200 import Engine
    d, t = models[name]
    V = CONFIGS[name]["vocab"]
    eng = Engine(d, dtype=dtype, max_tokens=64 * 9, max_slots=1)
    compare(eng, CONFIGS[name], t, {"a": random_ids(530, V, 77)}, [[("a", 10)]] + [[("a", 1)] for _ in range(520)], dtype)


def test_other_sizes_than_multiples_of_eight(tmp_path):
    """A width, head sizes and feed-forwards that no tensor-core kernel takes: the CUDA-core kernels serve both number types."""
    from ithaca_b200 import Engine
    cfg = _model([(_att(3, 1, 10, 0.3, 9.0, (0.2, 7)), _moe(7, 4, 2, (2, 1), 1.1, shared=5)), (_gla(3, 5, 7, 2.0, 3), _moe(21, 3, 1)), 0,
                  (_att(2, 1, 16, 0.3), None), 1], 37, 30)
    t = make_tensors(cfg, 3)
    d = _write(tmp_path, _stored(cfg), t, "odd")
    for dtype in ("float32", "bfloat16"):
        eng = Engine(d, dtype=dtype, max_tokens=512)
        compare(eng, cfg, t, {"a": random_ids(110, 37, 8)}, [[("a", 66)], [("a", 3)]] + [[("a", 1)]] * 41, dtype)


# ------------------------------------------------------------------------------------------ one token decides
D = 32


def _needle_base(cfg):
    """Token 1 (the needle) points along axis 0 and carries a mark on axis 5, token 2 (the query) points along axis 6, every other
    token along an axis of its own."""
    t = make_tensors(cfg, 9)
    g = torch.Generator().manual_seed(1)
    emb = torch.randn(40, D, generator=g) * 0.05
    for i in range(3, 40):
        emb[i, 8 + i % 20] += 1.5
    emb[1] += torch.eye(D)[0] * 1.5 + torch.eye(D)[5]
    emb[2] += torch.eye(D)[6] * 1.5
    emb[3:, :8] = 0.0
    t["embed"] = emb.bfloat16()
    for n in ("embed.norm", "l0.norm1", "l0.norm1b", "final.norm"):
        t[n], t[n + ".b"], t[n + ".alpha"] = torch.ones(D).bfloat16(), torch.zeros(D).bfloat16(), torch.tensor(1.0).bfloat16()
    t["l0.mix.o"] = (2 * torch.eye(D)).bfloat16()
    return t


def _query_rows(eng, ids, cuts):
    """The last token's logits for every way of cutting: a prompt of ``cut`` tokens, then one by one beside another request."""
    for cut in cuts:
        s, other = eng.alloc_slot(), eng.alloc_slot()
        lg = eng.step([other, s], [ids[3:10], ids[:cut]], "last")
        for x in ids[cut:]:
            lg = eng.step([s, other], [[x], [5]], "last")
        eng.free_slot(s)
        eng.free_slot(other)
        yield cut, lg.cpu().numpy()[1 if cut == len(ids) else 0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cap", [None, 50.0])
def test_the_one_key_that_matters(tmp_path, cap, dtype):
    """The needle sits at the first places, at a page's last and first place, far back and just behind the query; the query comes
    at the end of a prompt, is decoded alone after it, or a hundred decoded tokens later."""
    from ithaca_b200 import Engine
    cfg = _model([(_att(1, 1, D, 0.45, cap, (0.1, 100)), None)], 40, D, mult=1.0)
    t = _needle_base(cfg)
    wq, wk = torch.zeros(D, D), torch.eye(D)
    wq[0, 6] = 1.0                                                        # the query looks along the needle's axis
    wk[6, 6], wk[7, 6] = 0.0, 1.0
    t["l0.mix.q"], t["l0.mix.k"] = wq.bfloat16(), wk.bfloat16()
    eng = Engine(_write(tmp_path, cfg, t, "needle"), dtype=dtype, max_tokens=4096)
    n = 400
    none = [3 + (i * 7) % 37 for i in range(n - 1)] + [2]
    base = _plain(cfg, t, none)[n - 1]
    tol = REL[dtype] if dtype == "float32" else 6e-2
    for at in (0, 1, 63, 64, 127, 128, 200, 335, 336, n - 3, n - 2):
        ids = list(none)
        ids[at] = 1
        want = _plain(cfg, t, ids)[n - 1]
        assert rel_err(want, base) > 0.15, at                             # the test has teeth
        for cut, row in _query_rows(eng, ids, (n, n - 1, n - 5) + ((n - 100,) if at in (0, 63, 335) else ())):
            assert rel_err(row, want) < tol, (at, cut)
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_bias_tells_near_keys_from_far_ones(tmp_path, dtype):
    """Two needles with different marks: the nearer one wins although both match alike, at every distance; a bias that took
    distances from the wrong end, or none, would mix them."""
    from ithaca_b200 import Engine
    cfg = _model([(_att(2, 1, D, 0.45, 50.0, None), None)], 40, D, mult=1.0)
    t = _needle_base(cfg)
    wq, wk = torch.zeros(2 * D, D), torch.eye(D)
    wq[0, 6] = 1.0                                                        # the steep head asks, the flat one too
    wq[D, 6] = 1.0
    wk[6, 6], wk[7, 6] = 0.0, 1.0
    t["l0.mix.q"], t["l0.mix.k"] = wq.bfloat16(), wk.bfloat16()
    o = torch.zeros(D, 2 * D)
    o[:, :D] = 2 * torch.eye(D)                                           # slope 1/16 only
    t["l0.mix.o"] = o.bfloat16()
    t["embed"][4] = t["embed"][1]
    t["embed"][4, 5] = -t["embed"][1, 5]                                  # another needle, its mark reversed
    eng = Engine(_write(tmp_path, cfg, t, "two"), dtype=dtype, max_tokens=4096)
    n = 300
    hay = [5 + (i * 7) % 35 for i in range(n - 1)] + [2]
    tol = REL[dtype] if dtype == "float32" else 6e-2
    seen = []
    for far, near in ((0, 60), (60, 200), (64, 127), (200, 290), (290, 200)):
        ids = list(hay)
        ids[far], ids[near] = 1, 4
        want = _plain(cfg, t, ids)[n - 1]
        seen.append(want)
        for cut, row in _query_rows(eng, ids, (n, n - 1, 130)):
            assert rel_err(row, want) < tol, (far, near, cut)
    assert rel_err(seen[-1], seen[-2]) > 0.15                             # which of the two is nearer decides
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_state_carries_one_token_far(tmp_path, dtype):
    """A recurrence that hardly forgets: only the needle writes, only the query reads and opens the gate; what it reads is the
    needle's value, however long ago it was written, in a prompt, across portions and when decoded."""
    from ithaca_b200 import Engine
    cfg = _model([(_gla(1, 16, D, 16.0, 4), None)], 40, D, mult=1.0)
    t = _needle_base(cfg)
    q, k, g = torch.zeros(16, D), torch.zeros(16, D), torch.zeros(D, D)
    q[3, 6], k[3, 0], g[:, 6] = 2.0, 2.0, 4.0
    t["l0.mix.q"], t["l0.mix.k"], t["l0.mix.g"], t["l0.mix.v"] = q.bfloat16(), k.bfloat16(), g.bfloat16(), torch.eye(D).bfloat16()
    t["l0.mix.a2"], t["l0.mix.a2.b"] = torch.zeros(16, 4).bfloat16(), torch.full((16,), 8.0).bfloat16()
    t["l0.mix.norm"] = torch.ones(D).bfloat16()
    eng = Engine(_write(tmp_path, _stored(cfg), t, "state"), dtype=dtype, max_tokens=4096)
    n = 400
    none = [3 + (i * 7) % 37 for i in range(n - 1)] + [2]
    base = _plain(cfg, t, none)[n - 1]
    tol = REL[dtype] if dtype == "float32" else 6e-2
    for at in (0, 1, 63, 64, 127, 128, 300, n - 2):
        ids = list(none)
        ids[at] = 1
        want = _plain(cfg, t, ids)[n - 1]
        assert rel_err(want, base) > 0.15, at
        for cut, row in _query_rows(eng, ids, (n, n - 1, n - 5, 65)):
            assert rel_err(row, want) < tol, (at, cut)
    eng.check_status()


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_greedy_generation_through_the_engine(models, name, graphs):
    """More prompts than slots, unequal lengths, the generation loop's own batching and its graph-replayed decode steps."""
    from ithaca_b200 import Engine
    d, t = models[name]
    V = CONFIGS[name]["vocab"]
    prompts = [random_ids(n, V, 60 + n) for n in (1, 6, 125, 20)]
    eng = Engine(d, dtype="float32", max_tokens=64 * 12, max_slots=3, graphs=graphs)
    assert (eng._decoder is not None) == graphs                            # every part of the design may be replayed
    got = eng.generate(prompts, max_tokens=12, temp=0.0, rep_pen=1.0, stop_token_ids=[])

    def check(p, g):
        lgs = P.forward(CONFIGS[name], t, list(p) + g[:-1])
        for i, tok in enumerate(g):
            lg = lgs[len(p) - 1 + i]
            top2 = torch.topk(lg, 2).values
            if float(top2[0] - top2[1]) > 1e-4 * float(lg.abs().max()):
                assert tok == int(lg.argmax()), (len(p), i)
    for p, g in zip(prompts, got):
        assert len(g) == 12
        check(p, g)
    assert eng.cache.table.n_slots_in_use() == 0
    got = eng.generate(prompts[:3], max_tokens=9, temp=0.0, rep_pen=1.0, stop_token_ids=[got[0][4], got[2][6]])
    for p, g in zip(prompts, got):
        check(p, g)


def test_graph_replay_in_16_bit_gives_what_eager_steps_give(models):
    """The 16-bit decode kernels under replay, whose captured grids are shaped for longer sequences than they run on."""
    from ithaca_b200 import Engine
    d, _ = models["B"]
    prompts = [random_ids(n, 67, 80 + n) for n in (3, 70, 130)]
    outs = [Engine(d, dtype="bfloat16", max_tokens=1024, graphs=g).generate(prompts, max_tokens=80, temp=0.0, rep_pen=1.0, stop_token_ids=[])
            for g in (True, False)]
    for a, b in zip(*outs):
        same = next((i for i, (x, y) in enumerate(zip(a, b)) if x != y), len(a))
        assert same >= 20                                                  # (near ties may part the ways later on)


# ------------------------------------------------------------------------------------------ the programs
def test_trace_replay_and_command_line(models, tmp_path):
    import subprocess
    import sys
    from helpers import ROOT
    d, t = models["A"]
    V = 101
    reqs = {"p": random_ids(70, V, 90), "q": random_ids(3, V, 91), "r": random_ids(130, V, 92)}
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": reqs["p"][:66], "want": [0, 65]}, {"id": "q", "tokens": reqs["q"][:1], "want": []},
                                     {"id": "r", "tokens": reqs["r"][:126], "want": [125]}], "end": []}]
    for i in range(4):
        ent = [{"id": "p", "tokens": [reqs["p"][66 + i]], "want": [0]}, {"id": "r", "tokens": [reqs["r"][126 + i]], "want": [0]}]
        if i < 2:
            ent.insert(1, {"id": "q", "tokens": [reqs["q"][1 + i]], "want": [0] if i == 1 else []})
        steps.append({"step": 1 + i, "entries": ent, "end": (["q"] if i == 1 else []) + (["p", "r"] if i == 3 else [])})
    out = tmp_path / "out"
    want = {r: _plain(CFG_A, t, ids) for r, ids in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "210"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                           timeout=900)
        assert p.returncode == 0, p.stderr[-3000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(5)]
        got = np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V) for i in (0, 2, 4)])
        ref = np.stack([want["p"][0], want["p"][65], want["r"][125], want["p"][67], want["q"][2], want["r"][127], want["p"][69], want["r"][129]])
        if dtype == "float32":
            assert rel_err(got, ref) < REL[dtype]
        else:                                                              # (a token whose experts changed places is far off alone)
            rows = np.abs(got - ref).max(1) / np.abs(ref).max()
            assert np.median(rows) < 2 * REL[dtype]

    cli = [sys.executable, os.path.join(ROOT, "bin", "ithaca"), "--model", d, "--dtype", "float32"]
    p = subprocess.run(cli + ["--describe"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0 and p.stdout.count("sandwich:") == 7 and p.stdout.count("gla") == 4 and p.stdout.count("moe") == 6, p.stdout + p.stderr[-2000:]
    prompt = random_ids(11, V, 93)
    p = subprocess.run(cli + ["--prompt", ",".join(map(str, prompt)), "-n", "5", "--rep-pen", "1.0", "--stop-ids", ""],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    from ithaca_b200 import Engine
    eng = Engine(d, dtype="float32", max_tokens=512)
    assert [int(x) for x in p.stdout.strip().split(",")] == eng.generate([prompt], max_tokens=5, temp=0.0, rep_pen=1.0, stop_token_ids=[])[0]


def test_random_weights_written_and_made_on_the_device_agree(tmp_path):
    from ithaca_b200 import Engine
    from ithaca_b200.weights import write_random_model
    cfg = copy.deepcopy(CFG_A)
    d = write_random_model(os.path.join(str(tmp_path), "rand"), cfg, seed=5)
    ids = random_ids(40, 101, 3)
    a = Engine(d, dtype="float32", max_tokens=256)
    b = Engine.from_random(cfg, seed=5, dtype="float32", max_tokens=256)
    la = run_schedule(a, {"a": ids}, [[("a", 40)]])["a"]
    lb = run_schedule(b, {"a": ids}, [[("a", 40)]])["a"]
    assert np.array_equal(la, lb) and np.all(np.isfinite(la)) and np.abs(la).max() > 0
