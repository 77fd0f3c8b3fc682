"""A plain, slow Vovalorn decoder: whole sequences, no cache, one function per mechanism.

Nothing here is shared with the library under test.  It reads ``config.json`` keys from a plain dictionary and
tensors from a plain name -> tensor mapping and computes on the CPU in the dtype it is given (float64 by default,
so that it is the more exact side of a comparison).

The design in this file's notation (T tokens at positions 0 .. T-1, width d, c the residual constant):

* D(x; a, w, b) = tanh(a x) * w + b, a one number, w and b of size d.  R(x) = x / sqrt(mean(x^2) + eps).
* x = D(E[ids]; embed.norm).  A layer: x <- x + c D1b(mixer(D1(x))); x <- x + c D2b(ff(D2(x))); ff may be absent.  A layer that
  borrows another one's tensors runs them with a state of its own.  Then D(x; final.norm) and the head.
* mixer ``gla``: q = Wq h / sqrt(dim), k = Wk h, v = Wv h, a = sigmoid(Wa2 (Wa1 h) + b)^(1/tau) per head and key channel.  Per head
  S <- diag(a) S + k v^T, o = S^T q.  o is R-normed over its values times a weight the heads share, times silu(Wg h); Wo.
* mixer ``attention``: q = Wq h, k = Wk h, v = k; then q and k are R-normed per head and q is multiplied by
  1 + coef ln(floor((p + 1) / every) + 1).  s = cap tanh((q . k) scale / cap) - 2^(-8 (n + 1) / H) (i - j) for query head n;
  j <= i; softmax; Wo.
* ff: s = sigmoid(Wr h); picks by s + correction: groups of neighbouring experts rank by the sum of their two best picks, the
  ``keep`` best groups' experts compete, the ``top`` best win.  Weights: their s over the sum of those (+ 1e-20), times ``scale``.
  expert(h) = Wd (silu(Wg h) * (Wu h)); plus shared(h).
"""
from __future__ import annotations

import math
from typing import Mapping, Optional, Sequence

import torch


def dynamic_tanh(x: torch.Tensor, t: Mapping[str, torch.Tensor], name: str) -> torch.Tensor:
    dt = x.dtype
    return torch.tanh(t[name + ".alpha"].to(dt) * x) * t[name].to(dt) + t[name + ".b"].to(dt)


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


def channel_decay(z: torch.Tensor, tau: float) -> torch.Tensor:
    """sigmoid(z)^(1/tau) through its logarithm, -log(1 + e^-z) / tau."""
    log_sig = torch.where(z > 0, -torch.log1p(torch.exp(-z.abs())), z - torch.log1p(torch.exp(-z.abs())))
    return torch.exp(log_sig / float(tau))


def gla(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, a: torch.Tensor, state: Optional[torch.Tensor] = None):
    """q, k, a [T, H, K], v [T, H, V] -> (o [T, H, V], state [H, K, V])."""
    T, H, K = q.shape
    V = v.shape[2]
    S = torch.zeros(H, K, V, dtype=q.dtype) if state is None else state.clone()
    o = torch.zeros(T, H, V, dtype=q.dtype)
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def gla_mixer(h: torch.Tensor, m: Mapping, t: Mapping[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T, dt = h.shape[0], h.dtype
    H, K, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ t[p + "q"].to(dt).T).view(T, H, K) * K ** -0.5
    k = (h @ t[p + "k"].to(dt).T).view(T, H, K)
    v = (h @ t[p + "v"].to(dt).T).view(T, H, V)
    z = (h @ t[p + "a1"].to(dt).T) @ t[p + "a2"].to(dt).T + t[p + "a2.b"].to(dt)
    o, _ = gla(q, k, v, channel_decay(z, m["tau"]).view(T, H, K))
    o = (rms(o, eps) * t[p + "norm"].to(dt)).reshape(T, H * V)
    return (o * silu(h @ t[p + "g"].to(dt).T)) @ t[p + "o"].to(dt).T


def temperature(positions: torch.Tensor, coef: float, every: int, dtype=torch.float64) -> torch.Tensor:
    return 1.0 + float(coef) * torch.log((torch.div(positions + 1, int(every), rounding_mode="floor") + 1).to(dtype))


def slopes(n_heads: int) -> list:
    return [2.0 ** (-8.0 * (n + 1) / n_heads) for n in range(n_heads)]


def attention_core(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: Optional[float], first: int = 0) -> torch.Tensor:
    """q [T, H, D] at positions first .. first + T - 1, k [N, G, D] and v [N, G, Dv] from position 0 -> [T, H, Dv]."""
    T, H, _ = q.shape
    N, G = k.shape[:2]
    i, j = torch.arange(first, first + T)[:, None], torch.arange(N)[None, :]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for n, slope in enumerate(slopes(H)):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T) * float(scale)
        if cap:
            s = float(cap) * torch.tanh(s / float(cap))
        s = (s - slope * (i - j).to(s.dtype)).masked_fill(j > i, float("-inf"))
        out[:, n] = torch.softmax(s, dim=-1) @ v[:, g]
    return out


def attention_mixer(h: torch.Tensor, m: Mapping, t: Mapping[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T, dt = h.shape[0], h.dtype
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ t[p + "q"].to(dt).T).view(T, H, D)
    k = (h @ t[p + "k"].to(dt).T).view(T, G, D)
    v = k.clone()
    q, k = rms(q, eps), rms(k, eps)
    if m.get("q_temp"):
        q = q * temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"], dt)[:, None, None]
    return attention_core(q, k, v, m["scale"], m.get("softcap")).reshape(T, H * D) @ t[p + "o"].to(dt).T


def expert_ff(h: torch.Tensor, t: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ t[p + "gate"].to(h.dtype).T) * (h @ t[p + "up"].to(h.dtype).T)) @ t[p + "down"].to(h.dtype).T


def choose(s: torch.Tensor, correction: torch.Tensor, r: Mapping) -> torch.Tensor:
    """s [T, E] scores -> chosen experts [T, top]."""
    pick = s + correction.to(s.dtype)
    T, E = pick.shape
    g = r.get("groups")
    if g and g["count"] > 1:
        per = E // g["count"]
        by_group = pick.view(T, g["count"], per)
        rank = by_group.topk(min(2, per), dim=-1).values.sum(-1)
        kept = torch.zeros(T, g["count"], dtype=torch.bool).scatter(1, rank.topk(g["keep"], dim=-1).indices, True)
        pick = by_group.masked_fill(~kept[:, :, None], float("-inf")).reshape(T, E)
    return pick.topk(r["top"], dim=-1).indices


def weigh(s: torch.Tensor, chosen: torch.Tensor, r: Mapping) -> torch.Tensor:
    w = s.gather(1, chosen)
    return w / (w.sum(-1, keepdim=True) + 1e-20) * float(r.get("scale", 1.0))


def moe_ff(h: torch.Tensor, fc: Mapping, t: Mapping[str, torch.Tensor], p: str, forced: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``forced`` [T, top]: use these experts instead of the best ones (weighted by their own scores)."""
    r = fc["router"]
    s = sigmoid(h @ t[p + "router"].to(h.dtype).T)
    chosen = choose(s, t[p + "correction"], r) if forced is None else forced
    weight = weigh(s, chosen, r)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weight[rows, place][:, None] * expert_ff(h[rows], t, f"{p}e{e}.")
    return out + expert_ff(h, t, p + "shared.") if fc.get("shared") else out


def owner(cfg: Mapping, i: int) -> int:
    """The layer whose tensors layer i runs."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer(x: torch.Tensor, i: int, cfg: Mapping, t: Mapping[str, torch.Tensor], forced=None) -> torch.Tensor:
    lc, eps, c = cfg["layers"][i], float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    p = f"l{owner(cfg, i)}."
    mixer = {"gla": gla_mixer, "attention": attention_mixer}[lc["type"]]
    x = x + c * dynamic_tanh(mixer(dynamic_tanh(x, t, p + "norm1"), lc["mixer"], t, p + "mix.", eps), t, p + "norm1b")
    if lc.get("mlp") is None:
        return x
    return x + c * dynamic_tanh(moe_ff(dynamic_tanh(x, t, p + "norm2"), lc["mlp"], t, p + "mlp.", forced), t, p + "norm2b")


def forward(cfg: Mapping, t: Mapping[str, torch.Tensor], ids: Sequence[int], dtype=torch.float64, trace=None, forced=None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``trace``: a list that receives x after every layer.  ``forced``: the
    experts [T, top] to use in each layer that has a feed-forward, in the order of those layers."""
    x = dynamic_tanh(t["embed"].to(dtype)[torch.as_tensor(list(ids), dtype=torch.long)], t, "embed.norm")
    routed = 0
    for i, lc in enumerate(cfg["layers"]):
        f = None
        if lc.get("mlp") is not None and forced is not None:
            f = forced[routed]
            routed += 1
        x = layer(x, i, cfg, t, f)
        if trace is not None:
            trace.append(x.clone())
    return dynamic_tanh(x, t, "final.norm") @ t["head"].to(dtype).T
