"""Token embedding and the output head.

x[t, :] = E[id_t, :] * scale (src/model.cpp:1381-1383).  The reference clamps an id
outside the vocabulary; here the step function rejects it before anything runs.
With a norm of its own (``normed_embedding``, parameter ``norm``: the norm's record) the stream starts as norm(E[id] * scale).
logits = W_out xn, where W_out is the embedding matrix when the model has no
output matrix of its own (src/model.cpp:132, 1590-1592).  A head may scale its logits by a constant
(``scale``) and cap them, cap * tanh(logit / cap) (``softcap``), both in float.
"""
from __future__ import annotations

from typing import Dict, Mapping

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorReq
from .base import NORMS, Runtime, register_embedding, register_head, to_device
from .linear import Linear


class Embedding:
    @classmethod
    def manifest(cls, spec: PartSpec) -> Dict[str, TensorReq]:
        return {spec.weights["weight"]: TensorReq((spec["vocab_size"], spec["hidden_size"]))}

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        self.vocab_size = int(spec["vocab_size"])
        self.hidden = int(spec["hidden_size"])
        self.scale = float(spec.get("scale", 1.0))
        self.table = to_device(tensors[spec.weights["weight"]], runtime).contiguous()
        self.runtime = runtime

    def forward(self, ids: torch.Tensor, ctx=None) -> torch.Tensor:
        return ops.embed(ids, self.table, self.scale, self.runtime.status)


class NormedEmbedding(Embedding):
    @classmethod
    def manifest(cls, spec: PartSpec) -> Dict[str, TensorReq]:
        out = super().manifest(spec)
        out.update(NORMS.get(spec["norm"].kind).manifest(spec["norm"]))
        return out

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        self.norm = NORMS.get(spec["norm"].kind)(spec["norm"], tensors, runtime)

    def forward(self, ids: torch.Tensor, ctx=None) -> torch.Tensor:
        if hasattr(self.norm, "embed"):
            return self.norm.embed(ids, self.table, self.scale)
        return self.norm.forward(super().forward(ids, ctx), out_dtype=torch.float32)


class OutputHead:
    @classmethod
    def manifest(cls, spec: PartSpec) -> Dict[str, TensorReq]:
        return {spec.weights["weight"]: TensorReq((spec["vocab_size"], spec["hidden_size"]))}

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        self.vocab_size = int(spec["vocab_size"])
        self.linear = Linear([tensors[spec.weights["weight"]]], runtime)
        self.scale = float(spec.get("scale") or 1.0)
        self.softcap = float(spec.get("softcap") or 0.0)

    def forward(self, xn: torch.Tensor) -> torch.Tensor:
        logits = self.linear(xn, out_dtype=torch.float32)
        if self.scale != 1.0 or self.softcap > 0.0:
            ops.scale_softcap_(logits, self.scale, self.softcap)
        return logits


register_embedding("embedding", Embedding)
register_embedding("normed_embedding", NormedEmbedding)
register_head("lm_head", OutputHead)
