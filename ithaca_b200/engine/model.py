"""The generic decoder: embedding, the scheduled runs of the layers, final norm, head.

It is built from a ``ModelSpec`` alone.  The schedule is data: a list of runs,
each naming a layer and the cache entry its mixer works on (the reference's layer
loop is ``for L in layers`` with per-layer flags, src/model.cpp:1130-1259, 1457-1566).
Final norm and head run only on the rows whose logits are wanted, as the reference
does for the last row (src/model.cpp:1588-1594).
"""
from __future__ import annotations

import dataclasses
from typing import Dict, List, Mapping, Optional

import torch

from ..cache.cache import KVRequest, SequenceCache
from ..config import ConfigError, config_from_model_dir
from ..config.spec import ModelSpec, validate_schedule
from ..csrc import ops
from ..parts import BLOCKS, EMBEDDINGS, HEADS, NORMS, Runtime
from ..parts.block import _merge
from ..weights.loader import TensorReq, WeightError, check_tensors, load_checkpoint, read_model_tensors, _storage_form


def weight_manifest(spec: ModelSpec) -> Dict[str, TensorReq]:
    """Every tensor the model needs, with its shape."""
    out: Dict[str, TensorReq] = {}
    _merge(out, EMBEDDINGS.get(spec.embedding.kind).manifest(spec.embedding))
    for b in spec.layers:
        _merge(out, BLOCKS.get(b.kind).manifest(b))
    _merge(out, NORMS.get(spec.final_norm.kind).manifest(spec.final_norm))
    _merge(out, HEADS.get(spec.head.kind).manifest(spec.head))
    return out


def streamed_tensor_names(spec: ModelSpec) -> List[str]:
    """The tensors a step reads in full whatever it brings: what the layers' mixers and feed-forwards and the
    head ask for (their manifests), each once.  Norm vectors are left out (a few KB), and so is the embedding
    matrix, of which a step reads one row per token, unless the head shares it."""
    names: List[str] = []
    for e in spec.schedule:
        b = spec.layers[e.layer]
        from ..parts import FEED_FORWARDS, MIXERS
        for part, reg in ((b.mixer, MIXERS), (b.feed_forward, FEED_FORWARDS)):
            if part is not None:
                names += list(reg.get(part.kind).manifest(part))
    names += list(HEADS.get(spec.head.kind).manifest(spec.head))
    return list(dict.fromkeys(names))


class DecoderModel:
    def __init__(self, spec: ModelSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        validate_schedule(spec)
        if spec.streams > 0 and (any(b.kind != "hyper" for b in spec.layers) or any(e.adds_input for e in spec.schedule)):
            raise ConfigError("a model with residual streams of its blocks' own needs 'hyper' blocks and cannot add its input again")
        if spec.streams == 0 and any(b.kind == "hyper" for b in spec.layers):
            raise ConfigError("'hyper' blocks need the model to say how many residual streams there are")
        self.spec = spec
        self.runtime = runtime
        # bytes of the matrices a step streams, in the form the kernels read them: 16-bit on the bfloat16 path
        # (a matrix stored in 32-bit is rounded once when it is loaded), as stored on the float32 path
        self._streamed_bytes = sum(
            tensors[n].numel() * (2 if runtime.dtype == "bfloat16" and tensors[n].dtype.is_floating_point
                                  else tensors[n].element_size())
            for n in streamed_tensor_names(spec) if n in tensors)
        self.embedding = EMBEDDINGS.get(spec.embedding.kind)(spec.embedding, tensors, runtime)
        self.layers = [BLOCKS.get(b.kind)(b, tensors, runtime) for b in spec.layers]
        self.final_norm = NORMS.get(spec.final_norm.kind)(spec.final_norm, tensors, runtime)
        shared = set(spec.head.weights.values()) & set(spec.embedding.weights.values())
        if shared and hasattr(self.embedding, "table"):
            tensors = dict(tensors)
            for name in shared:
                tensors[name] = self.embedding.table                        # one copy on the device for both
        self.head = HEADS.get(spec.head.kind)(spec.head, tensors, runtime)
        # the norm that reads the stream behind each run: a block that takes it may form it at its own end
        self.following = [None] * len(spec.schedule)
        for n, e in enumerate(spec.schedule[1:]):
            if not e.adds_input and hasattr(self.layers[spec.schedule[n].layer], "entry_norm"):
                self.following[n] = getattr(self.layers[e.layer], "entry_norm", None)

    @property
    def graph_safe(self) -> bool:
        """True when every mixer and feed-forward says that a captured step may be replayed for
        other slots and positions (they read those from the step's device arrays, never from
        host values).  A part that does not say so is stepped eagerly."""
        return all(getattr(l.mixer, "graph_safe", False)
                   and (l.feed_forward is None or getattr(l.feed_forward, "graph_safe", False)) for l in self.layers)

    def cache_requests(self) -> Dict[int, List[object]]:
        """What every cache entry keeps: its writer's requests.  A run that only reads an entry may reach further back
        than the writer does; the entry then keeps keys for the widest window among its readers and writer."""
        out: Dict[int, List[object]] = {}
        for e in self.spec.schedule:
            if e.writes_cache:
                out[e.cache] = self.layers[e.layer].cache_requests()
        for e in self.spec.schedule:
            if e.writes_cache:
                continue
            for r in self.layers[e.layer].cache_requests():
                if not isinstance(r, KVRequest):
                    continue
                for n, have in enumerate(out[e.cache]):
                    if isinstance(have, KVRequest) and have.window is not None and (r.window is None or r.window > have.window):
                        have = out[e.cache][n] = dataclasses.replace(have, window=r.window)
                    if isinstance(have, KVRequest) and r.keep_first > have.keep_first:
                        out[e.cache][n] = dataclasses.replace(have, keep_first=r.keep_first)
        return out

    def forward(self, ctx, cache: SequenceCache) -> Optional[torch.Tensor]:
        """Runs the step's tokens through every scheduled run; returns float32 logits
        [wanted rows, vocab], or None when no row is wanted."""
        h = self.embedding.forward(ctx.token_ids, ctx)
        for made in ("stream_copy", "stream_normed"):
            ctx.shared.pop(made, None)                         # nothing of an earlier pass over this description counts
        h0 = h.clone() if any(e.adds_input for e in self.spec.schedule) else None
        if self.spec.streams > 0:
            h = ops.hyper_start(h, self.spec.streams)          # [T, streams, d]; the final norm reads the streams' sum
        for e, following in zip(self.spec.schedule, self.following):
            if e.adds_input:
                ops.add_(h, h0)
                ctx.shared.pop("stream_copy", None)            # a block's 16-bit copy of the stream is stale now
            if following is not None:
                self.layers[e.layer].forward(h, ctx, cache.layer(e.cache), e.writes_cache, next_norm=following)
            else:
                self.layers[e.layer].forward(h, ctx, cache.layer(e.cache), e.writes_cache)
        if ctx.n_logit_rows == 0:
            return None
        xn = self.final_norm.forward(h, rows=ctx.logit_rows)
        return self.head.forward(xn)

    def weight_bytes(self) -> int:
        """Bytes of weights a step reads once (the matrices of the scheduled layers and the head, each
        counted once; for roofline figures)."""
        return self._streamed_bytes


def build_model(arch, config, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
    spec = config.model_spec()
    if arch.build_model is not None:
        return arch.build_model(spec, tensors, runtime)
    return DecoderModel(spec, tensors, runtime)


def load_model(model_dir: str, runtime: Runtime):
    """Reads ``config.json``, picks the architecture from the registry, checks the
    folder's tensors against what the architecture's parts ask for, and builds the
    model on the runtime's device.  Returns (model, config)."""
    arch, config = config_from_model_dir(model_dir)
    found = read_model_tensors(model_dir)
    if hasattr(config, "with_tensor_shapes"):
        # sizes that the file leaves to the tensors (the rank of a low-rank factor)
        config = config.with_tensor_shapes({n: tuple(t.shape) for n, t in found.items()})
    spec = config.model_spec()
    manifest = weight_manifest(spec)
    ignore = []
    for name, same_as in spec.aliases.items():
        if name in found and name not in manifest:
            # a tensor that repeats another one may be stored; it must then hold the same values
            if same_as in found and found[name].shape == found[same_as].shape and torch.equal(found[name], found[same_as]):
                ignore.append(name)
            else:
                raise WeightError(f"the configuration says that '{name}' repeats '{same_as}', but the folder holds a "
                                  f"different '{name}'")
    check_tensors(found, manifest, ignore)
    tensors = {n: _storage_form(n, found[n], manifest[n]) for n in manifest if n in found}
    return build_model(arch, config, tensors, runtime), config
