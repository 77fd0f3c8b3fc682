"""A plain, slow Zomipel decoder: whole sequences, no cache, one function per mechanism.

Nothing here is shared with the library under test.  It reads ``config.json`` keys from a plain dictionary and
tensors from a plain name -> tensor mapping and computes on the CPU in the dtype it is given (float64 by default,
so that it is the more exact side of a comparison).

The design in this file's notation (T tokens at positions 0 .. T-1, width d):

* N(x, w) = x / sqrt(mean(x^2) + eps) * (1 + w).
* x0 = E[ids].  A layer: h = N(x, w_layer); x <- x + mixer(h) + ff(h); ff may be absent.
* layers lo..hi-1 are run R times in a row with the same weights; before every pass after the first, x += x0.
  Then the remaining layers, the final N and the head, which is E.
* mixer ``mamba2``: [z | x | B | C | dt] = Win h.  [x | B | C] through a causal convolution over time per channel with
  bias, then silu.  dt = softplus(dt + c_h).  Head h (its B and C from group h // (H / G)), state S [N, P], zero at first:
  S <- exp(-exp(A_h) dt) S + dt B x^T;  y = S^T C + D_h x.  y times silu(z), then every one of ``norm_groups`` equal parts
  divided by its own root mean square (eps inside), times a weight; Wo.
* mixer ``attention``: q, k, v = W h + b; the leading r dimensions of every q and k head turn in pairs (i, i + r/2) by
  p * base^(-2i/r); scores (q . k) * c; position i sees j when j <= i and (i - j < window or j < keep); softmax; Wo.
* feed-forward ``dense``: Wd gelu_tanh(Wu h).  ``moe``: z = Wr h + b; the ``top`` largest; weights = softmax over those;
  expert(h) = Wd (silu(Wg h) * (Wu h)); plus sigmoid(w_s . h) * shared(h) when there is a shared expert.
"""
from __future__ import annotations

import math
from typing import List, Mapping, Optional, Sequence

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * (1.0 + w.to(x.dtype))


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def causal_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: y[t] = b + sum_j w[:, j] * u[t - taps + 1 + j], zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], dim=0)
    y = b.to(u.dtype).expand_as(u).clone()
    for j in range(taps):
        y = y + w[:, j].to(u.dtype) * padded[j:j + u.shape[0]]
    return y


def ssd(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, A_log: torch.Tensor, D: torch.Tensor,
        state: Optional[torch.Tensor] = None):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (behind softplus) -> (y [T, H, P], state [H, N, P])."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.zeros_like(x)
    group = torch.arange(H) // (H // G)
    rate = -torch.exp(A_log.to(x.dtype))
    for t in range(T):
        a = torch.exp(rate * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t][group][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t][group][:, :, None]).sum(1) + D.to(x.dtype)[:, None] * x[t]
    return y, S


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """The gate first, then every one of ``groups`` equal parts by its own root mean square, then the weight."""
    T, d = y.shape
    g = (y * silu(z)).view(T, groups, d // groups)
    return rms(g, eps).reshape(T, d) * w.to(y.dtype)


def mamba2_mixer(h: torch.Tensor, m: Mapping, t: Mapping[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T, dt_ = h.shape[0], h.dtype
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = h @ t[p + "in"].to(dt_).T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, t[p + "conv"], t[p + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + t[p + "dt_bias"].to(dt_))
    y, _ = ssd(x, B, C, dt, t[p + "A_log"], t[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, t[p + "norm"], m["norm_groups"], eps) @ t[p + "o"].to(dt_).T


def rotate_halves(x: torch.Tensor, positions: Sequence[int], r: int, base: float) -> torch.Tensor:
    """x [T, heads, dim]: the pair (i, i + r/2) of every head's leading r dimensions turns by p * base^(-2i/r).
    Positions and angles are 32-bit numbers in the design: frequency and product are rounded to float32."""
    y = x.clone()
    p = torch.tensor(list(positions), dtype=torch.float32)[:, None]
    f = torch.tensor([float(base) ** (-2.0 * i / r) for i in range(r // 2)], dtype=torch.float64).to(torch.float32)[None, :]
    a = (p * f).to(x.dtype)
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :r // 2], x[..., r // 2:r]
    y[..., :r // 2] = u * c - v * s
    y[..., r // 2:r] = v * c + u * s
    return y


def visible(T: int, window: Optional[int], keep: int) -> torch.Tensor:
    """[T, T] bool: row i, column j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if window is not None:
        seen = seen & ((i - j < window) | (j < keep))
    return seen


def attention_core(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv] of one sequence -> [T, H, Dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for hh in range(H):
        g = hh // (H // G)
        s = ((q[:, hh] @ k[:, g].T) * float(scale)).masked_fill(~seen, float("-inf"))
        out[:, hh] = torch.softmax(s, dim=-1) @ v[:, g]
    return out


def attention_mixer(h: torch.Tensor, m: Mapping, t: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    T, dt = h.shape[0], h.dtype
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ t[p + r].to(dt).T + t[p + r + ".b"].to(dt) for r in "qkv")
    q, k, v = q.view(T, H, D), k.view(T, G, D), v.view(T, G, Dv)
    rot = m.get("rot")
    if rot is not None and rot["dims"] > 0:
        q, k = rotate_halves(q, range(T), rot["dims"], rot["base"]), rotate_halves(k, range(T), rot["dims"], rot["base"])
    mask = m.get("mask")
    seen = visible(T, mask["size"] if mask else None, (mask.get("keep_first") or 0) if mask else 0)
    return attention_core(q, k, v, m["scale"], seen).reshape(T, H * Dv) @ t[p + "o"].to(dt).T


def dense_ff(h: torch.Tensor, t: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    return gelu_tanh(h @ t[p + "up"].to(h.dtype).T) @ t[p + "down"].to(h.dtype).T


def expert_ff(h: torch.Tensor, t: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ t[p + "gate"].to(h.dtype).T) * (h @ t[p + "up"].to(h.dtype).T)) @ t[p + "down"].to(h.dtype).T


def route(h: torch.Tensor, top: int, w: torch.Tensor, b: torch.Tensor):
    """Returns (chosen experts [T, top], their weights [T, top])."""
    z = h @ w.to(h.dtype).T + b.to(h.dtype)
    best = z.topk(top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def moe_ff(h: torch.Tensor, fc: Mapping, t: Mapping[str, torch.Tensor], p: str, forced: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``forced`` [T, top]: use these experts instead of the best ones (their weights still are the softmax over their logits)."""
    chosen, weight = route(h, fc["router"]["top"], t[p + "router"], t[p + "router.b"])
    if forced is not None:
        z = h @ t[p + "router"].to(h.dtype).T + t[p + "router.b"].to(h.dtype)
        chosen = forced
        weight = torch.softmax(z.gather(1, forced), dim=-1)
    out = torch.zeros_like(h)
    for e in range(fc["router"]["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weight[rows, place][:, None] * expert_ff(h[rows], t, f"{p}e{e}.")
    if fc.get("shared"):
        out = out + sigmoid(h @ t[p + "shared.sg"].to(h.dtype).T) * expert_ff(h, t, p + "shared.")
    return out


def layer(x: torch.Tensor, i: int, cfg: Mapping, t: Mapping[str, torch.Tensor], forced=None) -> torch.Tensor:
    lc, eps, p = cfg["layers"][i], float(cfg["norm"]["eps"]), f"l{i}."
    h = norm(x, t[p + "norm1"], eps)
    if lc["type"] == "mamba2":
        y = mamba2_mixer(h, lc["mixer"], t, p + "mix.", eps)
    elif lc["type"] == "attention":
        y = attention_mixer(h, lc["mixer"], t, p + "mix.")
    else:
        raise ValueError(f"unknown mixer {lc['type']!r}")
    mlp = lc.get("mlp")
    if mlp is None:
        return x + y
    if mlp["kind"] == "dense":
        return x + (y + dense_ff(h, t, p + "mlp."))
    if mlp["kind"] == "moe":
        return x + (y + moe_ff(h, mlp, t, p + "mlp.", forced))
    raise ValueError(f"unknown feed-forward {mlp['kind']!r}")


def layer_runs(cfg: Mapping) -> List[tuple]:
    """(layer, adds the embedding's output first) for every run, in order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    lo, hi = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(lo)]
    for r in range(loop["times"]):
        runs += [(i, r > 0 and i == lo) for i in range(lo, hi)]
    return runs + [(i, False) for i in range(hi, n)]


def forward(cfg: Mapping, t: Mapping[str, torch.Tensor], ids: Sequence[int], dtype=torch.float64, trace=None, forced=None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``trace``: a list that receives x after every layer run.  ``forced``: the
    experts [T, top] to use in each run whose feed-forward is routed, in the order of those runs."""
    x0 = t["embed"].to(dtype)[torch.as_tensor(list(ids), dtype=torch.long)]
    x = x0.clone()
    routed = 0
    for i, add in layer_runs(cfg):
        if add:
            x = x + x0
        mlp = cfg["layers"][i].get("mlp")
        f = None
        if mlp is not None and mlp["kind"] == "moe" and forced is not None:
            f = forced[routed]
            routed += 1
        x = layer(x, i, cfg, t, f)
        if trace is not None:
            trace.append(x.clone())
    return norm(x, t["final.norm"], float(cfg["norm"]["eps"])) @ t["embed"].to(dtype).T
