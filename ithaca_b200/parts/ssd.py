"""The state-space duality mixer ("mamba2").

[z | x | B | C | dt] = W_in h with H heads of P values (``inner`` = H P columns of z and of x), G groups of N states (G N columns
of B and of C) and one step per head.  x, B and C together pass a causal convolution over time per channel (``conv_taps``
taps, with bias; the last column of the stored [channels, taps] matrix meets the current token, zeros stand before the
sequence's start) and silu.  dt = softplus(dt + dt_bias).  Per head h, whose B and C are those of group h // (H / G), with a
state S of N x P:

    S <- exp(-exp(A_log_h) dt) S + dt B x^T;    y = S^T C + D_h x

All heads together, y * silu(z) is RMS-normed in ``norm_groups`` equal parts (each by its own root mean square, ``norm_eps``
inside the root), multiplied by a weight of size ``inner``, and projected by W_o.

Per sequence and cache entry the mixer keeps S as float32 [2, H, N, P] (two copies by the parity of the position the state
belongs to, so that a decode step never overwrites what it read) and a ring of the last ``conv_taps`` inputs of the
convolution, float32.  Steps, decays, the state, its sums, the skip, the gate and the norm are float32 on both paths; the
projections' operands and, for a prompt, the convolution's output are 16-bit on the bfloat16 path.

A prompt on the bfloat16 path runs convolution, then chunks of 128 tokens on tcgen05 (``csrc/ssd_tcgen05.cu``) or, for sizes that
kernel does not take, of 64 tokens on the warp-level tensor path (``csrc/ssd.cu``); a decode step
runs convolution, step, decay, update and read-out in one kernel; the float32 path runs the convolution and the recurrence
token by token, for prompts and single tokens alike.
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

STATE, RING = "ssd_state", "ssd_conv_ring"


class StateSpaceDuality:
    graph_safe = True       # slots, positions and lengths come from device arrays; state by parity, ring by position

    @classmethod
    def manifest(cls, spec: PartSpec) -> Dict[str, TensorReq]:
        d, H, P, N, G, taps = (spec[k] for k in ("hidden_size", "n_heads", "v_head_dim", "state", "n_groups", "conv_taps"))
        inner, channels = H * P, H * P + 2 * G * N
        w = spec.weights
        return {w["in"]: TensorReq((inner + channels + H, d)), w["conv"]: TensorReq((channels, taps), std=1.0 / taps),
                w["conv_bias"]: TensorReq((channels,)), w["dt_bias"]: TensorReq((H,), std=0.5), w["A_log"]: TensorReq((H,), std=0.5),
                w["D"]: TensorReq((H,), init="ones"), w["norm"]: TensorReq((inner,), init="ones"), w["o"]: TensorReq((d, inner))}

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        self.hidden = int(spec["hidden_size"])
        self.n_heads = int(spec["n_heads"])
        self.v_head_dim = int(spec["v_head_dim"])
        self.n_state = int(spec["state"])
        self.n_groups = int(spec["n_groups"])
        self.taps = int(spec["conv_taps"])
        self.norm_groups = int(spec.get("norm_groups") or 1)
        self.norm_eps = float(spec["norm_eps"])
        self.inner = self.n_heads * self.v_head_dim
        self.channels = self.inner + 2 * self.n_groups * self.n_state
        if self.n_heads % self.n_groups:
            raise ValueError(f"mamba2: {self.n_heads} heads cannot share {self.n_groups} groups evenly")
        if self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.inner} channels do not form {self.norm_groups} equal parts")
        if self.n_state > 512:
            raise ValueError(f"mamba2: the kernels hold a column's states in one block's registers, up to 512 of them; found {self.n_state}")
        w = spec.weights
        self.in_proj = Linear([tensors[w["in"]]], runtime)
        self.o = Linear([tensors[w["o"]]], runtime)
        self.conv_w = to_device(tensors[w["conv"]], runtime).to(torch.float32).t().contiguous()      # tap-major [taps, channels]
        self.conv_b = as_float32(tensors[w["conv_bias"]], runtime)
        self.dt_bias = as_float32(tensors[w["dt_bias"]], runtime)
        self.A = (-torch.exp(as_float32(tensors[w["A_log"]], runtime).double())).to(torch.float32).contiguous()
        self.D = as_float32(tensors[w["D"]], runtime)
        self.norm_w = as_float32(tensors[w["norm"]], runtime)
        self.runtime = runtime

    def cache_requests(self) -> List[object]:
        out: List[object] = [StateRequest(STATE, (2, self.n_heads, self.n_state, self.v_head_dim), "float32")]
        if self.taps > 1:
            out.append(StateRequest(RING, (self.taps, self.channels), "float32"))
        return out

    def forward(self, x: torch.Tensor, ctx, cache: LayerCache, residual: torch.Tensor, writes_cache: bool = True,
                accumulate: bool = True) -> None:
        if not writes_cache:
            raise ValueError("mamba2: a run cannot read another run's state without advancing it")
        rt, T = self.runtime, x.shape[0]
        # rows on 16-byte boundaries, whatever the number of heads
        n = self.in_proj.out_features
        p = torch.empty((T, -(-n // 4) * 4), dtype=torch.float32, device=x.device)[:, :n]
        self.in_proj(x, out=p)
        state = cache.state(STATE)
        ring = cache.state(RING) if self.taps > 1 else None
        y = None
        if ctx.is_decode and rt.act_dtype != torch.float32:
            y = ops.ssd_decode(p, self.inner, self.conv_w, self.conv_b, ring, self.dt_bias, self.A, self.D, state, ctx, self.n_groups)
        if y is None:
            u = ops.causal_conv(p[:, self.inner:self.inner + self.channels], self.conv_w, self.conv_b, ring, ctx, rt.act_dtype, act=True)
            y = ops.ssd(u, p, self.inner + self.channels, self.dt_bias, self.A, self.D, state, ctx, self.n_groups,
                        status=rt.status)
        mid = ops.gated_group_norm(y, p[:, :self.inner], self.norm_w, self.norm_groups, self.norm_eps, rt.act_dtype)
        self.o(mid, out=residual, accumulate=accumulate)


register_mixer("mamba2", StateSpaceDuality)
