"""Typed configuration of the Vovalorn decoder, read from ``config.json``.

A Vovalorn model lists its layers one by one; every size and constant that can differ between two models of the design is
in the file or in a tensor's shape.  The keys:

* ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` (what a sublayer's result is multiplied by when it joins the stream);
* ``layers``: per layer ``type`` (the mixer: ``gla`` or ``attention``), ``mixer`` (its sizes and constants) and ``mlp`` (``kind: moe``
  with ``expert.ff``, ``router.experts``, ``router.top``, ``router.scale``, ``router.groups.count``, ``router.groups.keep`` and, if
  there is one, ``shared.ff``; or null for none).  ``weights_of: j``: the layer has no tensors of its own and runs layer j's, with a
  cache or state of its own.

A layer is a sandwich: a norm in front of and behind each sublayer.  The norm is a dynamic tanh, tanh(alpha x) * w + b with one
alpha; ``norm.eps`` serves the root mean squares inside the mixers.  The embedding's output passes a norm of the same kind.
``gla``: gated linear attention with a decay per key channel (``heads``, ``dim``, ``vdim``, ``tau``; the rank of the decay's first
factor is the first size of its tensor).  ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim`` (equal to ``dim``: the values are the
keys as projected), ``scale``, ``softcap``, ``q_temp.coef`` and ``q_temp.every``; no rotation, a distance bias of one slope per head.
The feed-forward's experts are gated with silu; sigmoid scores, choice by corrected scores within the best groups.

Tensor names: ``embed``, ``embed.norm``, ``final.norm``, ``head``, and per layer i ``l<i>.{norm1,norm1b,norm2,norm2b}`` (every norm with
``.alpha`` and ``.b``), ``l<i>.mix.{q,k,v,g,o,norm,a1,a2,a2.b}`` or ``l<i>.mix.{q,k,o}``, ``l<i>.mlp.{router,correction}``,
``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, need_float, need_int
from .spec import BlockSpec, ModelSpec, PartSpec, ScheduleEntry

# no key of the file bounds a sequence's length; this sizes nothing, it only stops a runaway caller
MAX_POSITION = 1 << 20
DEFAULT_DECAY_RANK = 16            # of random models; a folder's tensors say their own
WEIGHT_EPS = 1e-20                 # joins the sum that the chosen experts' scores are divided by

TYPES = ("gla", "attention")


def _obj(d: Dict[str, Any], key: str, where: str, optional: bool = False) -> Optional[Dict[str, Any]]:
    v = d.get(key)
    if v is None and optional:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object, found {v!r}")
    return v


def _check_gla(m: Dict[str, Any], where: str) -> None:
    need_int(m, "heads"), need_int(m, "dim"), need_int(m, "vdim")
    if need_float(m, "tau") <= 0:
        raise ConfigError(f"config.json: {where}.tau must be positive")
    if "rank" in m:
        need_int(m, "rank")


def _check_attention(m: Dict[str, Any], where: str) -> None:
    heads, kv = need_int(m, "heads"), need_int(m, "kv_heads")
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} heads cannot share {kv} kv_heads evenly")
    dim = need_int(m, "dim")
    if need_int(m, "vdim", dim) != dim:
        raise ConfigError(f"config.json: {where}: the values are the keys, so vdim must equal dim, found {m['vdim']} and {dim}")
    need_float(m, "scale")
    if m.get("softcap") is not None and need_float(m, "softcap") <= 0:
        raise ConfigError(f"config.json: {where}.softcap must be positive")
    temp = _obj(m, "q_temp", where + ".", optional=True)
    if temp is not None:
        need_float(temp, "coef"), need_int(temp, "every")


def _check_mlp(mlp: Any, where: str) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}mlp.kind {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not supported "
                          "(moe, or null for none)")
    need_int(_obj(mlp, "expert", where + "mlp."), "ff")
    router = _obj(mlp, "router", where + "mlp.")
    experts, top = need_int(router, "experts"), need_int(router, "top")
    if top > experts:
        raise ConfigError(f"config.json: {where}mlp.router.top cannot exceed the number of experts")
    need_float(router, "scale", 1.0)
    groups = _obj(router, "groups", where + "mlp.router.", optional=True)
    if groups is not None:
        count, keep = need_int(groups, "count"), need_int(groups, "keep")
        if experts % count or keep > count:
            raise ConfigError(f"config.json: {where}mlp.router.groups: {experts} experts do not form {count} equal groups of which {keep} are kept")
        if top > keep * (experts // count):
            raise ConfigError(f"config.json: {where}mlp.router.groups: the kept groups hold fewer experts than a token is to use")
    shared = _obj(mlp, "shared", where + "mlp.", optional=True)
    if shared is not None:
        need_int(shared, "ff")


@dataclass(frozen=True)
class VovalornConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[Dict[str, Any], ...]        # as validated from the file
    raw: Dict[str, Any] = field(default_factory=dict, compare=False)

    ARCHITECTURE = "Vovalorn"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "VovalornConfig":
        width = need_int(d, "width")
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        for i, l in enumerate(layers):
            where = f"layers[{i}]."
            if not isinstance(l, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            if l.get("type") not in TYPES:
                raise ConfigError(f"config.json: {where}type {l.get('type')!r} is not supported ({', '.join(TYPES)})")
            m = _obj(l, "mixer", where)
            (_check_gla if l["type"] == "gla" else _check_attention)(m, where + "mixer")
            if l.get("mlp") is not None:
                _check_mlp(l["mlp"], where)
        out = cls(architecture=cls.ARCHITECTURE, vocab_size=need_int(d, "vocab"), hidden_size=width,
                  norm_eps=need_float(_obj(d, "norm", ""), "eps"), residual_mult=need_float(d, "residual_mult", 1.0),
                  layers=tuple(copy.deepcopy(layers)), raw=copy.deepcopy(d))
        for i, l in enumerate(layers):
            src = layers[out.owner(i)]
            for key in ("type", "mixer", "mlp"):
                if l.get(key) != src.get(key):
                    raise ConfigError(f"config.json: layers[{i}] runs the tensors of layer {out.owner(i)}, but its '{key}' differs")
        return out

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i runs."""
        seen = {i}
        while self.layers[i].get("weights_of") is not None:
            j = need_int(self.layers[i], "weights_of", minimum=0)
            if j >= len(self.layers) or j in seen:
                raise ConfigError(f"config.json: layers[{i}].weights_of does not lead to a layer with tensors of its own, found {j}")
            seen.add(j)
            i = j
        return i

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "layers": copy.deepcopy(list(self.layers))}

    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "VovalornConfig":
        """The same configuration with the decay factors' ranks taken from tensor shapes (name -> shape): the file does not
        state them, the folder's tensors do."""
        layers = copy.deepcopy(list(self.layers))
        for i, l in enumerate(layers):
            name = f"l{self.owner(i)}.mix.a1"
            if l["type"] == "gla" and name in shapes:
                l["mixer"]["rank"] = int(shapes[name][0])
        return VovalornConfig(self.architecture, self.vocab_size, self.hidden_size, self.norm_eps, self.residual_mult, tuple(layers), self.raw)

    # -- the architecture-neutral description --------------------------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("dynamic_tanh", {"size": self.hidden_size}, {"weight": name, "bias": f"{name}.b", "alpha": f"{name}.alpha"})

    def _gla(self, p: str, m: Dict[str, Any]) -> PartSpec:
        w = {r: f"{p}.{r}" for r in ("q", "k", "v", "g", "o", "norm", "a1", "a2")}
        w["a2_bias"] = f"{p}.a2.b"
        return PartSpec("gla", {
            "hidden_size": self.hidden_size, "n_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "tau": m["tau"],
            "scale": float(m["dim"]) ** -0.5, "decay_rank": m.get("rank", DEFAULT_DECAY_RANK), "norm_eps": self.norm_eps}, w)

    def _attention(self, p: str, m: Dict[str, Any]) -> PartSpec:
        heads, temp = m["heads"], m.get("q_temp")
        return PartSpec("attention", {
            "hidden_size": self.hidden_size, "n_heads": heads, "n_kv_heads": m["kv_heads"], "head_dim": m["dim"], "scale": m["scale"],
            "softcap": m.get("softcap"), "window": None, "qk_norm": "unit", "norm_eps": self.norm_eps, "values": "keys",
            "q_temp": None if temp is None else (temp["coef"], temp["every"]),
            "distance_slopes": tuple(2.0 ** (-8.0 * (n + 1) / heads) for n in range(heads))}, {r: f"{p}.{r}" for r in "qko"})

    def _feed_forward(self, p: str, mlp: Dict[str, Any]) -> PartSpec:
        r = mlp["router"]
        groups, shared = r.get("groups"), mlp.get("shared")
        w = {"router": f"{p}.router", "correction": f"{p}.correction"}
        w.update({role: p + ".e{e}." + role for role in ("gate", "up", "down")})
        if shared is not None:
            w.update({f"shared_{role}": f"{p}.shared.{role}" for role in ("gate", "up", "down")})
        return PartSpec("moe", {
            "hidden_size": self.hidden_size, "intermediate_size": mlp["expert"]["ff"], "n_experts": r["experts"], "top": r["top"],
            "n_groups": groups["count"] if groups else 0, "group_keep": groups["keep"] if groups else 0, "group_score": "best_two",
            "score": "sigmoid", "renormalize": True, "weight_eps": WEIGHT_EPS, "weight_scale": r.get("scale", 1.0),
            "activation": "silu", "shared": shared["ff"] if shared is not None else 0}, w)

    def model_spec(self) -> ModelSpec:
        d = self.hidden_size
        owners = sorted({self.owner(i) for i in range(len(self.layers))})
        blocks = []
        for i in owners:
            l, p = self.layers[i], f"l{i}"
            mixer = self._gla(p + ".mix", l["mixer"]) if l["type"] == "gla" else self._attention(p + ".mix", l["mixer"])
            norms = {"mixer": self._norm(f"{p}.norm1"), "mixer_out": self._norm(f"{p}.norm1b")}
            ff = None
            if l.get("mlp") is not None:
                ff = self._feed_forward(p + ".mlp", l["mlp"])
                norms.update({"feed_forward": self._norm(f"{p}.norm2"), "feed_forward_out": self._norm(f"{p}.norm2b")})
            blocks.append(BlockSpec(kind="sandwich", mixer=mixer, feed_forward=ff, norms=norms, position=None,
                                    params={"residual_mult": self.residual_mult}))
        schedule = tuple(ScheduleEntry(layer=owners.index(self.owner(i)), cache=i) for i in range(len(self.layers)))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab_size, hidden_size=d,
            embedding=PartSpec("normed_embedding", {"vocab_size": self.vocab_size, "hidden_size": d, "norm": self._norm("embed.norm")},
                               {"weight": "embed"}),
            layers=tuple(blocks), schedule=schedule, final_norm=self._norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab_size, "hidden_size": d}, {"weight": "head"}),
            max_position=MAX_POSITION,
        )
