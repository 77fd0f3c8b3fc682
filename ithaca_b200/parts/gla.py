"""Gated linear attention: linear attention whose matrix state decays by a number per key channel.

q = Wq x and k = Wk x (``n_heads`` heads of ``head_dim``), v = Wv x (heads of ``v_head_dim``), and one decay per head and key
channel, a = sigmoid(Wa2 (Wa1 x) + b)^(1 / tau) with Wa1 of ``decay_rank`` rows.  Per head, with S of size head_dim x v_head_dim and
zero before the sequence's first token:

    S <- diag(a) S + k v^T;    o = ``scale`` S^T q

so the read-out sees the current token's write.  Every head's o is RMS-normed over its values (``norm_eps`` inside the root) with one
weight of size v_head_dim that the heads share; the heads side by side are multiplied by silu(Wg x) and projected out.

Per sequence and cache entry the mixer keeps S as float32 [2, heads, v_head_dim, head_dim] (two copies by the parity of the
position the state belongs to, as the other recurrences do, so that a decode step never overwrites what it read).  One product gives
[q | k | v | g | Wa1 x] in float; the decay's second factor, the sigmoid and the root are one kernel on its last columns.  Decays, the
state, its sums and the norm are float32 on both paths; only the products' operands are 16-bit on the bfloat16 path.

A prompt on the bfloat16 path runs recurrence, norm and gate by chunks of 64 tokens on the tensor cores (``csrc/gla_chunk.cu``), a decode
step runs everything between the products as one kernel (``csrc/gla_decode.cu``); a few tokens at a time, the float32 path and sizes that kernel does not take run the recurrence token by token.
"""
from __future__ import annotations

from typing import Dict, List, Mapping

import torch

from ..cache.cache import LayerCache, StateRequest
from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorReq
from .base import Runtime, as_float32, register_mixer, to_device
from .linear import Linear

STATE = "gla_state"
CHUNKED_FROM = 8            # tokens the longest sequence of a step brings


class GatedLinearAttention:
    graph_safe = True       # slots, positions and lengths come from device arrays; the state is kept by parity

    @classmethod
    def manifest(cls, spec: PartSpec) -> Dict[str, TensorReq]:
        d, H, dk, dv, r = (spec[k] for k in ("hidden_size", "n_heads", "head_dim", "v_head_dim", "decay_rank"))
        w = spec.weights
        return {w["q"]: TensorReq((H * dk, d)), w["k"]: TensorReq((H * dk, d)), w["v"]: TensorReq((H * dv, d)), w["g"]: TensorReq((H * dv, d)),
                w["a1"]: TensorReq((r, d)), w["a2"]: TensorReq((H * dk, r), std=r ** -0.5), w["a2_bias"]: TensorReq((H * dk,), std=0.5),
                w["norm"]: TensorReq((dv,), init="ones"), w["o"]: TensorReq((d, H * dv))}

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        self.n_heads = int(spec["n_heads"])
        self.head_dim = int(spec["head_dim"])
        self.v_head_dim = int(spec["v_head_dim"])
        self.rank = int(spec["decay_rank"])
        self.power = 1.0 / float(spec["tau"])
        self.scale = float(spec.get("scale", 1.0))
        self.norm_eps = float(spec["norm_eps"])
        if self.head_dim > 512:
            raise ValueError(f"gla: the kernel holds a state column's rows in the registers of up to 32 lanes, 16 each; found {self.head_dim}")
        w = spec.weights
        self.in_proj = Linear([tensors[w[r]] for r in ("q", "k", "v", "g", "a1")], runtime)
        self.o = Linear([tensors[w["o"]]], runtime)
        self.k_off = self.n_heads * self.head_dim
        self.v_off = 2 * self.k_off
        self.g_off = self.v_off + self.n_heads * self.v_head_dim
        self.a_off = self.g_off + self.n_heads * self.v_head_dim
        self.a2 = to_device(tensors[w["a2"]], runtime).to(torch.float32).t().contiguous()        # [rank, heads * head_dim]
        self.a2_bias = as_float32(tensors[w["a2_bias"]], runtime)
        self.norm_w = as_float32(tensors[w["norm"]], runtime)
        self.runtime = runtime

    def cache_requests(self) -> List[object]:
        return [StateRequest(STATE, (2, self.n_heads, self.v_head_dim, self.head_dim), "float32")]

    def forward(self, x: torch.Tensor, ctx, cache: LayerCache, residual: torch.Tensor, writes_cache: bool = True,
                accumulate: bool = True) -> None:
        if not writes_cache:
            raise ValueError("gla: a run cannot read another run's state without advancing it")
        rt, H, dk, dv, T = self.runtime, self.n_heads, self.head_dim, self.v_head_dim, x.shape[0]
        # rows on 16-byte boundaries, whatever the rank
        n = self.in_proj.out_features
        p = torch.empty((T, -(-n // 4) * 4), dtype=torch.float32, device=x.device)[:, :n]
        self.in_proj(x, out=p)                                                # [T, q | k | v | g | a1]
        mid = None
        if rt.dtype == "bfloat16" and ctx.is_decode:
            mid = ops.gla_decode(p, 0, self.k_off, self.v_off, self.g_off, self.a_off, self.a2, self.a2_bias, self.power, cache.state(STATE), ctx, H, dk,
                                 dv, self.norm_w, self.norm_eps, self.scale)
        elif rt.dtype == "bfloat16" and ctx.max_new >= CHUNKED_FROM:
            decay = ops.lowrank_decay(p, self.a_off, self.a2, self.a2_bias, self.power, log2=True)
            mid = ops.gla_chunks(p, 0, self.k_off, self.v_off, self.g_off, decay, cache.state(STATE), ctx, H, dk, dv, self.norm_w, self.norm_eps,
                                 self.scale)
        if mid is None:
            decay = ops.lowrank_decay(p, self.a_off, self.a2, self.a2_bias, self.power)
            o = ops.row_decay("plain", p, 0, self.k_off, self.v_off, decay, None, None, cache.state(STATE), ctx, H, H, dk, dv, self.scale)
            mid = ops.head_norm_gate(o, self.norm_w, self.norm_eps, p, self.g_off, H, rt.act_dtype, gate="silu")
        self.o(mid, out=residual, accumulate=accumulate)


register_mixer("gla", GatedLinearAttention)
