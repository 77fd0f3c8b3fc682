"""The Zomipel decoder and its mechanisms against the plain implementation (tests/plain/zomipel_plain.py).

Small configurations with weights made here.  Per mechanism: the kernel against the plain function, also across several
steps where it carries a state, and one-layer models of each mixer and feed-forward.  Whole models: prompts against
token-by-token decoding, portions down to two tokens, batches of unequal requests against each alone, slots, pages and
states that are used again, long decoding, and greedy generation through the engine's own loop.  Where random weights would
hide a fault (a far key, a kept key, a window's edge, a state or an input that was lost on the way), the weights are made so
that one token decides the result.
"""
import copy
import json
import os

import numpy as np
import pytest
import torch

from helpers import REL, random_ids, rel_err, run_schedule
from plain import zomipel_plain as P
from test_gunenex_gpu import STEPS, RouterTap, _close, _ctx, _portions, _write, rows_hold, SCHEDULES

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _ssd(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _att(heads, kv, dim, vdim, scale, rot=None, mask=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if mask is not None:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return m


def _ff(n):
    return {"kind": "dense", "ff": n}


def _moe(ff, experts, top, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _model(layers, vocab, width, eps=1e-5, loop=None):
    c = {"architecture": "Zomipel", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "layers": [{"type": "mamba2" if "state" in m else "attention", "mixer": m, "mlp": f} for m, f in layers]}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# unlike layers: value sizes unlike key sizes, part of the head turned, three groups in six heads, parts of the norm that cut
# through heads, a layer without feed-forward, windows shorter and longer than a page with and without kept keys, a loop over
# two different layers
CFG_A = _model([
    (_att(4, 2, 32, 16, 0.2, rot=(16, 500.0), mask=(9, 3)), _moe(24, 5, 2, shared=40)),
    (_ssd(6, 8, 24, 3, 3, 2), _ff(88)),
    (_ssd(4, 24, 16, 1, 4, 8), None),
    (_att(2, 2, 16, 16, 0.3, rot=(16, 1000.0), mask=(70, 0)), _moe(40, 6, 1)),
], 101, 64, loop=(1, 3, 2))
# one head, one group, one tap, one expert; every expert chosen; one kept key; sizes the tensor-core kernels take; no window and
# no rotation
CFG_B = _model([
    (_att(1, 1, 64, 64, 0.15, rot=(64, 10000.0), mask=(64, 1)), _moe(32, 1, 1, shared=16)),
    (_ssd(1, 32, 8, 1, 1, 1), _moe(16, 3, 3)),
    (_ssd(8, 64, 128, 2, 2, 8), None),
    (_att(3, 1, 32, 32, 0.2), _ff(40)),
], 67, 48, eps=1e-6)
# the whole model three times over; recurrent sizes the tensor-core kernel does not take and a head wider than one block of it;
# heads of 128 in groups of four, the whole head turned, kept keys that end inside a page behind a window of three pages
CFG_C = _model([
    (_ssd(3, 20, 12, 3, 3, 5), _moe(48, 8, 3, shared=72)),
    (_att(8, 2, 128, 128, 0.09, rot=(128, 250000.0), mask=(130, 66)), _ff(56)),
    (_ssd(2, 80, 64, 1, 5, 1), _moe(64, 4, 2, shared=8)),
], 89, 64, loop=(0, 3, 3))
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
        elif name == "final.norm" or last == "norm1":
            t = 0.2 * r                                           # stored around zero
        elif last == "norm":
            t = 1.0 + 0.2 * r
        elif last == "conv":
            t = 0.6 * r
        elif last == "dt_bias":
            t = r - 1.0
        elif last == "A_log":
            t = r - 0.5
        elif last == "D":
            t = 1.0 + 0.5 * r
        elif len(shape) == 1:                                     # biases
            t = 0.4 * r
        elif last in ("router", "sg"):
            t = r * (3.0 / shape[1] ** 0.5)
        else:
            t = r * (1.2 / shape[1] ** 0.5)
        out[name] = t.bfloat16()
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("zomipel")
    out = {}
    for i, (n, c) in enumerate(CONFIGS.items()):
        t = make_tensors(c, 30 + i)
        out[n] = (_write(root, c, t, n), t)
    return out


def _plain(cfg, t, ids):
    return P.forward(cfg, t, ids).numpy()


def routed_runs(cfg):
    return sum(1 for i, _ in P.layer_runs(cfg) if (cfg["layers"][i]["mlp"] or {}).get("kind") == "moe")


def run_tapped(eng, cfg, reqs, schedule):
    """As ``run_schedule``, and beside the logits, for every request, the experts the library used in each routed run."""
    n = routed_runs(cfg)
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
    the tolerance.  bfloat16: two experts whose logits lie a few hundredths apart change places under 16-bit operands, so that
    run is held against the plain implementation made to use the experts the library chose (which experts are the right ones is
    what the float32 run and the routing kernels' own tests check)."""
    if dtype == "float32":
        got = run_schedule(eng, reqs, schedule)
        for r, ids in reqs.items():
            assert _close(got[r], _plain(cfg, t, ids)), (r, rel_err(got[r], _plain(cfg, t, ids)))
        return got
    got, used = run_tapped(eng, cfg, reqs, schedule)
    for r, ids in reqs.items():
        assert rows_hold(got[r], P.forward(cfg, t, ids, forced=used[r]).numpy()), r
    return got


# ------------------------------------------------------------------------------------------ the recurrence
def _ssd_case(H, G, N, Pv, seed, dtype, n_tok, slow):
    """Inputs of three sequences.  ``slow``: steps and rates so small that the state hardly forgets (its error would add up);
    else from hardly to completely forgotten in one token."""
    g = torch.Generator().manual_seed(seed)
    u = torch.randn(n_tok, H * Pv + 2 * G * N, generator=g).to(dtype)
    raw = torch.randn(n_tok, H, generator=g) * 2.0
    dt_bias = torch.randn(H, generator=g) - (5.0 if slow else 1.0)
    A_log = torch.randn(H, generator=g) * (0.5 if slow else 2.0) - (3.0 if slow else 0.0)
    return u, raw, dt_bias, A_log, torch.randn(H, generator=g)


def _ssd_plain(u, raw, dt_bias, A_log, D, H, G, N, Pv, state):
    u, T = u.double(), u.shape[0]
    dt = P.softplus(raw.double() + dt_bias.double())
    y, S = P.ssd(u[:, :H * Pv].reshape(T, H, Pv), u[:, H * Pv:H * Pv + G * N].reshape(T, G, N), u[:, H * Pv + G * N:].reshape(T, G, N), dt,
                 A_log.double(), D.double(), state)
    return y.reshape(T, H * Pv), S


@pytest.mark.parametrize("slow", [False, True])
@pytest.mark.parametrize("kind,dtype", [("scan", torch.float32), ("scan", torch.bfloat16), ("mma", torch.bfloat16), ("tcgen05", torch.bfloat16)])
@pytest.mark.parametrize("H,G,N,Pv", [(4, 2, 16, 24), (3, 3, 40, 8), (2, 1, 128, 64), (6, 1, 24, 16), (1, 1, 64, 136), (4, 4, 8, 32), (5, 1, 12, 10),
                                      (2, 2, 200, 33), (4, 2, 64, 64), (3, 3, 128, 192), (8, 2, 128, 64)])
def test_state_space_kernels(kind, dtype, H, G, N, Pv, slow):
    """A prompt, portions and single tokens behind it, three sequences in scattered slots with leftovers in their states; the
    state in both its places and every y."""
    from ithaca_b200.csrc import ops
    takes = {"scan": True, "mma": N <= 128 and N % 8 == 0 and Pv % 8 == 0, "tcgen05": N in (64, 128) and Pv % 64 == 0}[kind]
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    slots = [3, 0, 2]
    state = torch.randn(4, 2, H, N, Pv, device=DEV)                   # leftovers: a sequence starts from zeros all the same
    plain = {b: None for b in range(3)}
    total = [max(hi[b] for _, hi in STEPS) for b in range(3)]
    data = {b: _ssd_case(H, G, N, Pv, 10 + b, dtype, total[b], slow) for b in range(3)}
    _, _, dt_bias, A_log, D = data[0]
    A = -torch.exp(A_log.double()).float().to(DEV)
    worst = 0.0
    for lo, hi in STEPS:
        ctx = _ctx(lo, hi, slots)
        u = torch.cat([data[b][0][lo[b]:hi[b]] for b in range(3)]).to(DEV)
        raw = torch.cat([data[b][1][lo[b]:hi[b]] for b in range(3)])
        p = torch.full((u.shape[0], H + 7), 9.0)
        p[:, 5:5 + H] = raw
        args = (u, p.to(DEV), 5, dt_bias.to(DEV), A, D.to(DEV), state, ctx, G)
        if not takes:
            with pytest.raises(ops.KernelError):
                ops.ssd(*args, kind=kind)
            return
        y = ops.ssd(*args, kind=kind, status=status).cpu().double()
        assert status.item() == 0
        at = 0
        for b in range(3):
            n = hi[b] - lo[b]
            want, S = _ssd_plain(data[b][0][lo[b]:hi[b]], data[b][1][lo[b]:hi[b]], dt_bias, A_log, D, H, G, N, Pv, plain[b])
            got_S = state[slots[b], (hi[b] - 1) & 1].cpu().double()
            worst = max(worst, float((y[at:at + n] - want).abs().max() / want.abs().max()), float((got_S - S).abs().max() / S.abs().max()))
            plain[b] = S
            at += n
    # inputs are given exactly (bfloat16 values), everything behind them is float: what is left is float rounding, and for the
    # chunks the two-part operands' 2^-17
    assert worst < (3e-6 if kind == "scan" and dtype == torch.float32 else 2e-5), worst


@pytest.mark.parametrize("kind", ["mma", "tcgen05"])
def test_long_prompts_in_chunks_against_token_by_token(kind):
    """Prompts of several chunks with a ragged end, two sequences, a portion behind each: both tensor-core kernels against the
    token-by-token kernel on the same values, many heads at once."""
    from ithaca_b200.csrc import ops
    H, G, N, Pv = 24, 4, 128, 64
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    ends = [1000, 389]
    data = [_ssd_case(H, G, N, Pv, 20 + b, torch.bfloat16, ends[b], b == 0) for b in range(2)]
    dt_bias, A, D = data[0][2].to(DEV), -torch.exp(data[0][3].double()).float().to(DEV), data[0][4].to(DEV)
    states = [torch.randn(2, 2, H, N, Pv, generator=torch.Generator().manual_seed(1)).to(DEV) for _ in range(2)]
    for lo, hi in (([0, 0], [700, 256]), ([700, 256], [1000, 389])):
        ctx = _ctx(lo, hi, [1, 0])
        u = torch.cat([data[b][0][lo[b]:hi[b]] for b in range(2)]).to(DEV)
        raw = torch.cat([data[b][1][lo[b]:hi[b]] for b in range(2)]).to(DEV).contiguous()
        got, want = (ops.ssd(u, raw, 0, dt_bias, A, D, st, ctx, G, kind=k, status=status) for st, k in zip(states, (kind, "scan")))
        assert status.item() == 0 and rel_err(got.cpu().numpy(), want.cpu().numpy()) < 2e-5
        for b in range(2):
            a, w = (st[[1, 0][b], (hi[b] - 1) & 1].cpu().numpy() for st in states)
            assert rel_err(a, w) < 2e-5


def test_state_space_scan_gives_the_same_bits_however_it_is_cut():
    from ithaca_b200.csrc import ops
    H, G, N, Pv, n = 4, 2, 24, 40, 90
    u, raw, dt_bias, A_log, D = (v.to(DEV) for v in _ssd_case(H, G, N, Pv, 3, torch.float32, n, False))
    A = -torch.exp(A_log)

    def run(cuts):
        state = torch.zeros(1, 2, H, N, Pv, device=DEV)
        ys = [ops.ssd(u[a:b], raw[a:b].contiguous(), 0, dt_bias, A, D, state, _ctx([a], [b], [0]), G) for a, b in zip(cuts, cuts[1:])]
        return torch.cat(ys), state[0, (n - 1) & 1].clone()
    y, S = run([0, n])
    for cuts in ([0, 1, 3, 16, 17, 64, n], list(range(n + 1))):
        y2, S2 = run(cuts)
        assert torch.equal(y, y2) and torch.equal(S, S2)


@pytest.mark.parametrize("H,G,N,Pv,taps", [(4, 2, 16, 24, 4), (6, 2, 40, 8, 3), (2, 1, 128, 64, 2), (1, 1, 64, 136, 5), (3, 3, 7, 4, 1), (2, 1, 300, 12, 4)])
def test_decode_kernel_with_its_convolution(H, G, N, Pv, taps):
    """Token by token from position 0 in slots with leftovers, beside the convolution and the recurrence done apart; running a
    step twice changes nothing (a captured graph does)."""
    from ithaca_b200.csrc import ops
    C, n, slots = H * Pv + 2 * G * N, 12, [2, 0]
    g = torch.Generator().manual_seed(7)
    rows = [torch.randn(n, C, generator=g) for _ in slots]
    raws = [torch.randn(n, H, generator=g) for _ in slots]
    w, cb = torch.randn(C, taps, generator=g) * 0.6, torch.randn(C, generator=g)
    dt_bias, A_log, D = torch.randn(H, generator=g) - 1, torch.randn(H, generator=g), torch.randn(H, generator=g)
    state = torch.randn(3, 2, H, N, Pv, device=DEV)
    ring = torch.randn(3, taps, C, device=DEV) if taps > 1 else None
    dev = lambda x: x.to(DEV).contiguous()
    want = []
    for b in range(2):
        u = P.silu(P.causal_conv(rows[b].double(), w.double(), cb.double()))
        want.append(_ssd_plain(u, raws[b], dt_bias, A_log, D, H, G, N, Pv, None))
    for i in range(n):
        p = torch.zeros(2, 4 * ((8 + C + H + 3) // 4))
        for b in range(2):
            p[b, 8:8 + C], p[b, 8 + C:8 + C + H] = rows[b][i], raws[b][i]
        ctx = _ctx([i, i], [i + 1, i + 1], slots)
        for _ in range(2):
            y = ops.ssd_decode(dev(p), 8, dev(w.t()), dev(cb), ring, dev(dt_bias), dev(-torch.exp(A_log)), dev(D), state, ctx, G)
        for b in range(2):
            assert rel_err(y[b].cpu().numpy(), want[b][0][i].numpy()) < 1e-5, (i, b)
    for b in range(2):
        assert rel_err(state[slots[b], (n - 1) & 1].cpu().numpy(), want[b][1].numpy()) < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,C", [(2, 2048), (3, 1028), (4, 3072), (5, 1024)])
def test_short_convolution_of_long_prompts(dtype, taps, C):
    """Prompts long enough for the kernel that takes several tokens a thread: sequences that begin inside a run of tokens, one
    that goes on from its ring; the same bits as short steps give."""
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(taps)
    lens, slots = [3001, 2, 6100, 1], [2, 0, 3, 1]
    x = [torch.randn(n + 5, C, generator=g) for n in lens]
    w, cb = torch.randn(C, taps, generator=g) * 0.5, torch.randn(C, generator=g)
    ring = torch.randn(4, taps, C, generator=g).to(DEV)
    wd, bd = w.t().contiguous().to(DEV), cb.to(DEV)
    out = [[] for _ in lens]
    for lo, hi in (([0] * 4, [5, 1, 2, 1]), ([5, 1, 2, 1], [n + 1 if n > 1 else 2 for n in lens])):
        ctx = _ctx(lo, hi, slots)
        y = ops.causal_conv(torch.cat([x[b][lo[b]:hi[b]] for b in range(4)]).to(DEV), wd, bd, ring, ctx, dtype)
        for b, part in enumerate(y.split([h - l for l, h in zip(lo, hi)])):
            out[b].append(part)
    ring2 = torch.zeros_like(ring)
    for b, n in enumerate(lens):
        end = n + 1 if n > 1 else 2
        got = torch.cat(out[b])
        want = P.silu(P.causal_conv(x[b][:end].double(), w, cb))
        assert rel_err(got.float().cpu().numpy(), want.numpy()) < (2e-6 if dtype == torch.float32 else 5e-3), b
        cuts = list(range(0, end, 700)) + [end]
        again = torch.cat([ops.causal_conv(x[b][a:e].to(DEV), wd, bd, ring2, _ctx([a], [e], [0]), dtype) for a, e in zip(cuts, cuts[1:])])
        assert torch.equal(got, again), b


def test_decode_kernel_declines_odd_value_sizes():
    from ithaca_b200.csrc import ops
    z = lambda *s: torch.zeros(*s, device=DEV)
    assert ops.ssd_decode(z(1, 6 + 8 + 2), 0, z(2, 14), z(14), z(1, 2, 14), z(2), z(2), z(2), z(1, 2, 2, 4, 3), _ctx([0], [1], [0]), 1) is None


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,groups", [(64, 1), (96, 8), (30, 3), (4096, 1), (9216, 1), (4800, 6), (8192, 16), (33, 1)])
def test_gated_group_norm_kernel(dtype, d, groups):
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(d)
    y, p, w = torch.randn(5, d, generator=g), torch.randn(5, d + 12, generator=g) * 2, torch.randn(d, generator=g)
    y[3] *= 1e-4                                                      # eps matters
    got = ops.gated_group_norm(y.to(DEV), p.to(DEV)[:, 4:4 + d], w.to(DEV), groups, 1e-5, dtype)
    want = P.gated_group_norm(y.double(), p.double()[:, 4:4 + d], w.double(), groups, 1e-5)
    assert got.dtype == dtype and rel_err(got.float().cpu().numpy(), want.numpy()) < (2e-6 if dtype == torch.float32 else 5e-3)
    assert rel_err(got[3].float().cpu().numpy(), want[3].numpy()) < (2e-6 if dtype == torch.float32 else 5e-3)


# ------------------------------------------------------------------------------------------ attention
def _paged_case(nh, nkv, hd, hdv, lens, new, dtype, seed, scale, window, keep):
    """Random q, k, v of sequences laid into scrambled pages; the last ``new[b]`` positions of each are the step's queries.
    Every query's best key is one of the first ``keep`` or just outside them, so that a kept key left out (or one too many)
    shows."""
    from test_kernels_gpu import Paged
    g = torch.Generator().manual_seed(seed)
    qs = [torch.randn(l, nh, hd, generator=g).to(dtype) for l in lens]
    ks = [torch.randn(l, nkv, hd, generator=g).to(dtype) for l in lens]
    vs = [torch.randn(l, nkv, hdv, generator=g).to(dtype) for l in lens]
    pk, pv = Paged(lens, nkv, hd, dtype, seed), Paged(lens, nkv, hdv, dtype, seed)       # same seed: same block table
    pk.fill(ks, ks)
    pv.fill(vs, vs)
    ref = torch.cat([P.attention_core(q.double(), k.double(), v.double(), scale, P.visible(l, window or None, keep))[l - n:]
                     for q, k, v, l, n in zip(qs, ks, vs, lens, new)]).reshape(sum(new), nh * hdv)
    q = torch.cat([q[l - n:] for q, l, n in zip(qs, lens, new)]).reshape(sum(new), nh * hd).to(DEV)
    i32 = lambda a: torch.from_numpy(np.asarray(a).astype(np.int32)).to(DEV)
    tab = pk.dev()[2].clone()
    if window:                                                        # pages that no query of the step sees are gone
        for b, (l, n) in enumerate(zip(lens, new)):
            first = max(0, l - n + 1 - window) // 64
            tab[b, -(-keep // 64):first] = -1
    return dict(q=q, k=pk.dev()[0], v=pv.dev()[0], tab=tab, ref=ref, seq=i32(np.repeat(np.arange(len(lens)), new)),
                pos=i32(np.concatenate([np.arange(l - n, l) for l, n in zip(lens, new)])), cu=i32(np.concatenate([[0], np.cumsum(new)])), lens=i32(lens))


KEEPS = [(9, 3), (64, 1), (64, 64), (65, 65), (40, 130), (1, 1), (200, 0), (130, 66), (0, 5)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,hdv", [(4, 2, 16, 24), (3, 1, 40, 40)])
@pytest.mark.parametrize("window,keep", KEEPS)
def test_kept_keys_in_the_cuda_core_attention(dtype, nh, nkv, hd, hdv, window, keep):
    from ithaca_b200.csrc import ops
    lens, new = [1, 70, 300, 129, 64, 500], [1, 70, 170, 1, 64, 3]
    c = _paged_case(nh, nkv, hd, hdv, lens, new, dtype, 40, 0.7, window, keep)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    got = ops.attention_simt(c["q"], c["k"], c["v"], c["seq"], c["pos"], c["tab"], nh, 0.7, window, status, keep=keep)
    assert status.item() == 0
    assert rel_err(got.float().cpu().numpy(), c["ref"].numpy()) < (3e-6 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("nh,nkv,hd,kind", [(4, 4, 16, "mma"), (6, 2, 32, "mma"), (8, 2, 64, "tc"), (8, 4, 128, "tc"), (6, 2, 128, "mma")])
@pytest.mark.parametrize("window,keep", KEEPS)
def test_kept_keys_in_the_tensor_core_attention(nh, nkv, hd, kind, window, keep):
    """Prefill (both kernels) and decode with chunks of one to four pages, in a table whose unseen pages are gone."""
    from ithaca_b200.csrc import attention_bf16 as A
    scale = 2.0 / hd ** 0.5
    lens, new = [1, 70, 300, 129, 64, 700], [1, 70, 67, 129, 5, 450]
    c = _paged_case(nh, nkv, hd, hd, lens, new, torch.bfloat16, 41, scale, window, keep)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    got = A.prefill(c["q"], c["k"], c["v"], c["cu"], c["lens"], c["tab"], len(lens), max(new), nh, scale, window, status, kind=kind, keep=keep)
    assert status.item() == 0
    assert rel_err(got.float().cpu().numpy(), c["ref"].numpy()) < 8e-3
    d = _paged_case(nh, nkv, hd, hd, lens, [1] * len(lens), torch.bfloat16, 42, scale, window, keep)
    for chunk in (1, 2, 4):
        got = A.decode(d["q"], d["k"], d["v"], d["lens"], d["tab"], len(lens), 1000, nh, scale, window, status, chunk_pages=chunk, keep=keep)
        assert status.item() == 0
        assert rel_err(got.float().cpu().numpy(), d["ref"].numpy()) < 8e-3
    if window == 9:                                                   # the test has teeth: without the kept keys another result
        other = A.decode(d["q"], d["k"], d["v"], d["lens"], d["tab"], len(lens), max(lens), nh, scale, window, status)
        assert rel_err(other.float().cpu().numpy(), d["ref"].numpy()) > 5e-2


@pytest.mark.parametrize("T", [1, 5, 12, 40, 300])
@pytest.mark.parametrize("hd,nh,nkv,pairing", [(64, 4, 2, 0), (32, 3, 1, 0), (128, 2, 2, 0)])
def test_biases_in_the_fused_projection(T, hd, nh, nkv, pairing):
    """The 16-bit mixer whose product adds the biases, rotates and appends in its epilogue, against the plain mixer."""
    from ithaca_b200.cache.cache import SequenceCache
    from ithaca_b200.config.spec import PartSpec
    from ithaca_b200.engine.context import ContextBuilder
    from ithaca_b200.parts import MIXERS, POSITIONS, Runtime
    d, window, keep = 72, 50, 7
    m = _att(nh, nkv, hd, hd, hd ** -0.5, rot=(hd, 700.0), mask=(window, keep))
    t = {n[len("l0.mix."):]: v for n, v in make_tensors(_model([(m, None)], 11, d), 5).items() if n.startswith("l0.mix.")}
    for r in "qkv":
        t[r + ".b"] = (t[r + ".b"].float() * 4).bfloat16()            # biases as large as the projections
    rt = Runtime("bfloat16", DEV)
    pos = POSITIONS.get("rotary")(PartSpec("rotary", {"rotary_dim": hd, "theta": 700.0, "pairing": "half"}), {}, rt)
    w = {r: r for r in "qkvo"}
    w.update({r + "_bias": r + ".b" for r in "qkv"})
    spec = PartSpec("attention", {"hidden_size": d, "n_heads": nh, "n_kv_heads": nkv, "head_dim": hd, "scale": hd ** -0.5, "bias": "qkv",
                                  "window": window, "keep_first": keep}, w)
    mix = MIXERS.get("attention")(spec, t, rt, position=pos)
    assert mix.fused_rope and not mix.wide
    x = torch.randn(T, d, generator=torch.Generator().manual_seed(T)).bfloat16()
    cache = SequenceCache({0: mix.cache_requests()}, max_tokens=512, max_slots=2)
    s = cache.alloc_slot()
    cache.reserve([s], [T])
    ctx = ContextBuilder(DEV).build([s], [[0] * T], [0], [[]], [cache.table.table_rows(0, [s], 8)])
    out = torch.ones(T, d, device=DEV)
    mix.forward(x.to(DEV), ctx, cache.layer(0), out)
    want = 1.0 + P.attention_mixer(x.double(), m, {k: v.double() for k, v in t.items()}, "")
    assert int(rt.status.item()) == 0 and rel_err(out.cpu().numpy(), want.numpy()) < REL["bfloat16"]
    free = {k: (torch.zeros_like(v) if k.endswith(".b") else v).double() for k, v in t.items()}
    assert rel_err(1.0 + P.attention_mixer(x.double(), m, free, "").numpy(), want.numpy()) > 0.1


# ------------------------------------------------------------------------------------------ experts, norm
@pytest.mark.parametrize("E,top,K,T", [(5, 2, 48, 3), (12, 4, 256, 70), (1, 1, 64, 9), (40, 40, 128, 20), (7, 3, 30, 65), (33, 5, 2052, 130)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_biased_router_and_the_shared_experts_weight(E, top, K, T, dtype):
    """Choice, weights and the extra row's sigmoid, from the fused kernel and from ready-made logits; the bias decides some
    choices."""
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(E)
    x, wr, b = torch.randn(T, K, generator=g).to(dtype), torch.randn(E + 1, K, generator=g) / K ** 0.5, torch.randn(E, generator=g) * 2
    z = x.double() @ wr.double().T
    e, w = P.route(x.double(), top, wr[:E], b)
    gate = torch.empty(T, device=DEV)
    got = ops.moe_router(x.to(DEV), wr.to(DEV), top, renorm=True, bias=b.to(DEV), gate=gate)
    assert (got is None) == (K % 4 != 0)
    if got is not None:
        assert rel_err(gate.cpu().numpy(), torch.sigmoid(z[:, E]).numpy()) < 1e-5
        assert torch.equal(got[0].cpu().long(), e) and rel_err(got[1].cpu().numpy(), w.numpy()) < 1e-5
    gate = torch.empty(T, device=DEV)
    got = ops.moe_route(z.float().to(DEV), top, renorm=True, bias=b.to(DEV), gate=gate)
    assert torch.equal(got[0].cpu().long(), e) and rel_err(got[1].cpu().numpy(), w.numpy()) < 1e-5
    assert rel_err(gate.cpu().numpy(), torch.sigmoid(z[:, E]).numpy()) < 1e-5
    if 1 < top < E:
        assert not torch.equal(P.route(x.double(), top, wr[:E], torch.zeros(E))[0], e)


def test_combine_adds_one_more_result_and_the_stream():
    from ithaca_b200.csrc import ops
    g = torch.Generator().manual_seed(1)
    parts, w, ex, ew, y = (torch.randn(s, generator=g) for s in ((12, 20), (6, 2), (6, 20), (6,), (6, 20)))
    want = (parts.view(6, 2, 20) * w[:, :, None]).sum(1)
    dev = lambda v: v.to(DEV)
    assert rel_err(ops.moe_combine(dev(parts), dev(w)).cpu().numpy(), want.numpy()) < 1e-6
    assert rel_err(ops.moe_combine(dev(parts), dev(w), extra=dev(ex)).cpu().numpy(), (want + ex).numpy()) < 1e-6
    out = dev(y)
    ops.moe_combine(dev(parts), dev(w), out=out, extra=dev(ex), extra_weight=dev(ew), accumulate=True)
    assert rel_err(out.cpu().numpy(), (y + want + ex * ew[:, None]).numpy()) < 1e-6
    out = dev(y)
    ops.moe_combine(dev(parts), dev(w), out=out, extra=dev(ex), extra_weight=dev(ew))
    assert rel_err(out.cpu().numpy(), (want + ex * ew[:, None]).numpy()) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,ff,E,top,shared,T", [(64, 24, 5, 2, 40, 9), (48, 40, 1, 1, None, 3), (128, 96, 16, 4, 64, 300), (72, 16, 3, 3, 200, 1),
                                                 (256, 64, 12, 3, 72, 1500), (30, 7, 4, 2, 21, 20), (64, 32, 9, 2, None, 600)])
def test_routed_feed_forward_with_a_shared_expert(dtype, d, ff, E, top, shared, T):
    from ithaca_b200.config import config_from_dict
    from ithaca_b200.parts import FEED_FORWARDS, Runtime
    fc = _moe(ff, E, top, shared)
    cfg = _model([(_ssd(1, 8, 8), fc)], 13, d)
    t = make_tensors(cfg, 3)
    rt = Runtime(dtype, DEV)
    part = FEED_FORWARDS.get("moe")(config_from_dict(cfg)[1].model_spec().layers[0].feed_forward, t, rt)
    x = torch.randn(T, d, generator=torch.Generator().manual_seed(2)).bfloat16()
    base = torch.randn(T, d, generator=torch.Generator().manual_seed(4))
    for accumulate in (True, False):
        res = base.to(DEV)
        with RouterTap() as tap:
            part.forward(x.to(DEV).to(rt.act_dtype), None, res, accumulate=accumulate)
        chosen = tap.calls[0].cpu().long()
        want = P.moe_ff(x.double(), fc, {k: v.double() for k, v in t.items()}, "l0.mlp.", chosen) + (base if accumulate else 0)
        assert rel_err(res.cpu().numpy(), want.numpy()) < (REL["float32"] if dtype == "float32" else 1.5e-2)
    free, _ = P.route(x.double(), top, t["l0.mlp.router"], t["l0.mlp.router.b"])
    same = (chosen.sort(1).values == free.sort(1).values).all(1).double().mean()
    assert same == 1.0 if dtype == "float32" else same > 0.98


def test_norm_weights_are_stored_around_zero():
    from ithaca_b200.config.spec import PartSpec
    from ithaca_b200.parts import NORMS, Runtime
    g = torch.Generator().manual_seed(0)
    x, w = torch.randn(4, 96, generator=g), (torch.randn(96, generator=g) * 0.3).bfloat16()
    rt = Runtime("float32", DEV)
    n = NORMS.get("rmsnorm")(PartSpec("rmsnorm", {"size": 96, "eps": 1e-3, "unit_offset": True}, {"weight": "w"}), {"w": w}, rt)
    assert rel_err(n.forward(x.to(DEV)).cpu().numpy(), P.norm(x.double(), w.double(), 1e-3).numpy()) < 1e-6


# ------------------------------------------------------------------------------------------ one-layer models
ONE_LAYER = {
    "recurrence": _model([(_ssd(4, 16, 24, 2, 4, 2), None)], 53, 48),
    "recurrence, one tap": _model([(_ssd(2, 8, 8, 2, 1, 1), _ff(32))], 53, 48),
    "recurrence, no tensor-core sizes": _model([(_ssd(3, 6, 10, 1, 3, 9), None)], 53, 48),
    "recurrence, long taps, many parts": _model([(_ssd(2, 64, 128, 1, 7, 16), None)], 53, 64),
    "window and kept": _model([(_att(4, 2, 16, 24, 0.25, rot=(8, 100.0), mask=(20, 6)), None)], 53, 48),
    "window and kept, fused": _model([(_att(4, 1, 64, 64, 0.12, rot=(64, 10000.0), mask=(66, 65)), _ff(40))], 53, 64),
    "no window": _model([(_att(3, 3, 8, 8, 0.4), None)], 53, 48),
    "kept longer than the window": _model([(_att(2, 2, 32, 32, 0.2, rot=(32, 50.0), mask=(10, 90)), None)], 53, 48),
    "routed and shared": _model([(_ssd(1, 8, 8), _moe(24, 7, 2, shared=16))], 53, 48),
    "routed": _model([(_att(2, 1, 24, 8, 0.3, mask=(7, 0)), _moe(24, 4, 4))], 53, 48),
    "looped": _model([(_ssd(2, 16, 8, 1, 3, 1), _ff(24))], 53, 48, loop=(0, 1, 4)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ONE_LAYER))
def test_one_layer_models(tmp_path, name, dtype):
    from ithaca_b200 import Engine
    cfg = ONE_LAYER[name]
    t = make_tensors(cfg, 11)
    eng = Engine(_write(tmp_path, cfg, t, "one"), dtype=dtype, max_tokens=1024)
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


def test_slots_pages_and_states_are_used_again(models):
    """A small cache: requests come and go, so slots, pages, states and rings are handed out again, also to shorter sequences
    whose first tokens must see nothing of what lay there before; windows give pages back on the way."""
    from ithaca_b200 import Engine
    for name, pages in (("A", 6), ("C", 8)):
        d, t = models[name]
        cfg, V = CONFIGS[name], CONFIGS[name]["vocab"]
        eng = Engine(d, dtype="float32", max_tokens=64 * pages, max_slots=2)
        for round_ in range(4):
            reqs = {"x": random_ids(230 - 60 * round_, V, 20 + round_), "y": random_ids(3 + round_, V, 30 + round_)}
            got = run_schedule(eng, reqs, [[("x", len(reqs["x"]) - 2), ("y", 2)], [("x", 1), ("y", 1)], [("x", 1)]]
                               + [[("y", 1)] for _ in range(round_)])
            for r, ids in reqs.items():
                assert _close(got[r], _plain(cfg, t, ids)), (name, round_, r)
            eng.cache.table.check_consistent()
            assert all(p.held() == 0 for p in eng.cache.table.pools)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(models, name, dtype):
    """Windows pass over decoded tokens and give their pages back; a cache with room for little more than a window's pages."""
    from ithaca_b200 import Engine
    d, t = models[name]
    V = CONFIGS[name]["vocab"]
    eng = Engine(d, dtype=dtype, max_tokens=64 * 7, max_slots=1)
    compare(eng, CONFIGS[name], t, {"a": random_ids(530, V, 77)}, [[("a", 10)]] + [[("a", 1)] for _ in range(520)], dtype)


def test_other_sizes_than_multiples_of_eight(tmp_path):
    """A width, head sizes and feed-forwards that no tensor-core kernel takes: the CUDA-core kernels serve both number types."""
    from ithaca_b200 import Engine
    cfg = _model([(_att(3, 1, 10, 6, 0.3, rot=(6, 77.0), mask=(21, 2)), _moe(7, 4, 2, shared=5)), (_ssd(3, 5, 7, 1, 2, 3), _ff(21)),
                  (_att(2, 1, 16, 16, 0.3, rot=(16, 77.0), mask=(33, 4)), None)], 37, 30, loop=(1, 2, 2))
    t = make_tensors(cfg, 3)
    d = _write(tmp_path, cfg, t, "odd")
    for dtype in ("float32", "bfloat16"):
        eng = Engine(d, dtype=dtype, max_tokens=512)
        compare(eng, cfg, t, {"a": random_ids(110, 37, 8)}, [[("a", 66)], [("a", 3)]] + [[("a", 1)]] * 41, dtype)


# ------------------------------------------------------------------------------------------ one token decides
D = 32


def _needle_base(cfg):
    """Token 1 (the needle) and token 2 (the query) point along axis 0, every other token along an axis of its own; the
    needle carries a mark on axis 5.  The mixer's result outweighs the token's own embedding."""
    t = make_tensors(cfg, 9)
    g = torch.Generator().manual_seed(1)
    emb = torch.randn(40, D, generator=g) * 0.05
    for i in range(3, 40):
        emb[i, 8 + i % 20] += 4.0
    emb[1] += torch.eye(D)[0] * 4 + torch.eye(D)[5] * 2
    emb[2] += torch.eye(D)[0] * 4 - torch.eye(D)[5] * 2
    emb[3:, 0] = 0.0
    t["embed"] = emb.bfloat16()
    t["l0.norm1"] = t["final.norm"] = torch.zeros(D).bfloat16()
    t["l0.mix.o"] = (3 * torch.eye(D)).bfloat16()
    return t


def _needle_attention(mask):
    cfg = _model([(_att(1, 1, D, D, 0.05, mask=mask), None)], 40, D)
    t = _needle_base(cfg)
    pick = torch.zeros(D, D)
    pick[0, 0] = 4.0
    t["l0.mix.q"] = t["l0.mix.k"] = pick.bfloat16()
    t["l0.mix.v"] = torch.eye(D).bfloat16()
    for r in "qkv":
        t[f"l0.mix.{r}.b"] = torch.zeros_like(t[f"l0.mix.{r}.b"])
    return cfg, t


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
@pytest.mark.parametrize("mask", [(75, 20), (64, 1), (130, 66), (70, 0), (12, 128), None], ids=str)
def test_the_one_key_that_matters(tmp_path, mask, dtype):
    """The needle sits just inside and just outside the window and the kept keys, at a page's last and first place and far
    back; the query comes at the end of a prompt, is decoded alone after it, or a hundred decoded tokens later (the window has
    then passed over decoded tokens)."""
    from ithaca_b200 import Engine
    cfg, t = _needle_attention(mask)
    eng = Engine(_write(tmp_path, cfg, t, "needle"), dtype=dtype, max_tokens=4096)
    n = 400
    hay = [3 + (i * 7) % 37 for i in range(n)]
    places = {0, 1, 63, 64, 127, 128, n - 2}
    if mask:
        places |= {n - 1 - mask[0], n - mask[0], n - mask[0] + 1, mask[1] - 1, mask[1], mask[1] + 1}
    none = list(hay)
    none[n - 1] = 2
    base = _plain(cfg, t, none)[n - 1]
    tol = REL[dtype] if dtype == "float32" else 6e-2
    for at in sorted(p for p in places if 0 <= p < n - 1):
        ids = list(none)
        ids[at] = 1
        want = _plain(cfg, t, ids)[n - 1]
        seen = mask is None or n - 1 - at < mask[0] or at < mask[1]
        assert (rel_err(want, base) > 0.15) == seen, at                  # the test has teeth: seen or not, other logits
        for cut, row in _query_rows(eng, ids, (n, n - 1, n - 5) + ((n - 100,) if at in (0, n - 400, n - 1 - (mask or (64,))[0]) else ())):
            assert rel_err(row, want) < tol, (at, cut)
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_state_carries_one_token_far(tmp_path, dtype):
    """A recurrence that hardly forgets: only the needle writes, only the query reads and opens the gate; what it reads is the
    needle's value, however long ago it was written, in a prompt, across portions and when decoded."""
    from ithaca_b200 import Engine
    cfg = _model([(_ssd(1, D, 8, 1, 2, 1), None)], 40, D)
    t = _needle_base(cfg)
    w = torch.zeros(D + D + 16 + 1, D)
    w[:D, 0] = 4.0                                                        # z: the gates open for needle and query
    w[D:2 * D] = torch.eye(D) * 2.0                                       # x: the normed token itself, without the axis that
    w[D, 0] = 0.0                                                         # needle and query share
    w[2 * D, 0] = 1.0                                                     # B and C: axis 0 only (silu(0) = 0 for the others)
    w[2 * D + 8, 0] = 1.0
    t["l0.mix.in"] = w.bfloat16()
    taps = torch.zeros(D + 16, 2)
    taps[:, 1] = 1.0                                                      # the convolution passes the current token through
    t["l0.mix.conv"], t["l0.mix.conv.b"] = taps.bfloat16(), torch.zeros(D + 16).bfloat16()
    t["l0.mix.dt_bias"], t["l0.mix.A_log"] = torch.full((1,), -5.0).bfloat16(), torch.full((1,), -1.0).bfloat16()
    t["l0.mix.D"] = torch.zeros(1).bfloat16()
    t["l0.mix.norm"] = torch.ones(D).bfloat16()
    eng = Engine(_write(tmp_path, cfg, t, "state"), dtype=dtype, max_tokens=4096)
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


@pytest.mark.parametrize("taps,back", [(2, 1), (4, 3), (3, 1)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_token_some_places_before_decides(tmp_path, taps, back, dtype):
    """A convolution whose only open tap lies ``back`` places before the token, and a state that forgets at once: a token's
    result depends on that one earlier token alone, within a portion, across portions, when decoded one by one, and in a slot
    that was used before; the first tokens read zeros."""
    from ithaca_b200 import Engine
    cfg = _model([(_ssd(1, D, 8, 1, taps, 1), None)], 40, D)
    t = _needle_base(cfg)
    w = torch.zeros(D + D + 16 + 1, D)
    w[:D] = torch.randn(D, D, generator=torch.Generator().manual_seed(3)) * 0.3
    w[D:2 * D] = torch.eye(D) * 2.0
    t["l0.mix.in"] = w.bfloat16()
    c = torch.zeros(D + 16, taps)
    c[:D, taps - 1 - back] = 1.0
    bias = torch.zeros(D + 16)
    bias[D:] = 1.0                                                        # B and C are constants
    t["l0.mix.conv"], t["l0.mix.conv.b"] = c.bfloat16(), bias.bfloat16()
    t["l0.mix.dt_bias"], t["l0.mix.A_log"] = torch.full((1,), 1.0).bfloat16(), torch.full((1,), 4.0).bfloat16()
    t["l0.mix.norm"] = torch.ones(D).bfloat16()
    eng = Engine(_write(tmp_path, cfg, t, "conv"), dtype=dtype, max_tokens=1024, max_slots=2)
    ids = [1, 2, 2, 1, 7, 2, 1] + [3 + (i * 5) % 30 for i in range(60)] + [1, 2, 9, 1]
    want = _plain(cfg, t, ids)
    assert rel_err(_plain(cfg, t, [2] + ids[1:])[back], want[back]) > 0.15
    tol = REL[dtype] if dtype == "float32" else 6e-2
    for sched in ([[("a", len(ids))]], [[("a", 1)]] * len(ids), [[("a", 2)], [("a", 1)], [("a", 3)], [("a", 58)], [("a", 1)], [("a", 6)]]):
        assert rel_err(run_schedule(eng, {"a": ids}, sched)["a"], want) < tol


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
        got0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(3, V)
        got2 = np.fromfile(out / "2.f32", dtype="<f4").reshape(3, V)
        got4 = np.fromfile(out / "4.f32", dtype="<f4").reshape(2, V)
        got = np.concatenate([got0, got2, got4])
        ref = np.stack([want["p"][0], want["p"][65], want["r"][125], want["p"][67], want["q"][2], want["r"][127], want["p"][69], want["r"][129]])
        if dtype == "float32":
            assert rel_err(got, ref) < REL[dtype]
        else:                                                              # (a token whose experts changed places is far off alone)
            rows = np.abs(got - ref).max(1) / np.abs(ref).max()
            assert np.median(rows) < 2 * REL[dtype]

    cli = [sys.executable, os.path.join(ROOT, "bin", "ithaca"), "--model", d, "--dtype", "float32"]
    p = subprocess.run(cli + ["--describe"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0 and p.stdout.count("parallel:") == 6 and p.stdout.count("mamba2") == 4 and p.stdout.count("moe") == 2 \
        and p.stdout.count("input added first") == 1, p.stdout + p.stderr[-2000:]
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
