"""Typed configuration of the Zomipel decoder, read from ``config.json``.

A Zomipel model lists its layers one by one; every size and constant that can differ between two models of the design is in
the file.  The keys:

* ``vocab``, ``width``, ``norm.eps``;
* ``layers``: per layer ``type`` (the mixer: ``mamba2`` or ``attention``), ``mixer`` (its sizes and constants) and ``mlp`` (``kind:
  dense`` with ``ff``; ``kind: moe`` with ``expert.ff``, ``router.experts``, ``router.top`` and, if there is one, ``shared.ff``; or
  null for none);
* ``loop``: layers ``start`` .. ``stop`` - 1 run ``times`` times in a row with the same weights, each pass with a cache or state
  of its own; before every pass after the first the embedding's output joins the stream.

A layer is parallel: one RMS norm (its stored weight is the distance from one), and mixer and feed-forward both read it and
both add to the stream.  ``mamba2``: ``heads`` of ``vdim`` values, ``groups`` of ``state`` states, ``conv`` taps, ``norm_groups``
parts of the gated norm.  ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, biases on q, k and v, ``rot.dims``
leading dimensions turned in halves with ``rot.base``, a window of ``mask.size`` keys behind which the first
``mask.keep_first`` keys of a sequence stay visible.  The dense feed-forward is ungated with the tanh form of gelu; the routed
one has gated experts chosen by biased logits, their weights the softmax over the chosen logits, and an expert for every token
whose result a sigmoid weighs.  The output matrix is the embedding matrix.

Tensor names: ``embed``, ``final.norm``, and per layer i ``l<i>.norm1``,
``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``, ``l<i>.mix.{q,k,v,o}`` with ``.b`` for the biases of q, k, v,
``l<i>.mlp.{up,down}``, ``l<i>.mlp.router`` (+ ``.b``), ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down,sg}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, need_float, need_int
from .spec import BlockSpec, ModelSpec, PartSpec, ScheduleEntry

# no key of the file bounds a sequence's length; this sizes nothing, it only stops a runaway caller
MAX_POSITION = 1 << 20

TYPES = ("mamba2", "attention")


def _obj(d: Dict[str, Any], key: str, where: str, optional: bool = False) -> Optional[Dict[str, Any]]:
    v = d.get(key)
    if v is None and optional:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object, found {v!r}")
    return v


def _check_mamba2(m: Dict[str, Any], where: str) -> None:
    heads, groups = need_int(m, "heads"), need_int(m, "groups")
    if heads % groups:
        raise ConfigError(f"config.json: {where}: {heads} heads cannot share {groups} groups evenly")
    need_int(m, "state"), need_int(m, "conv")
    parts = need_int(m, "norm_groups", 1)
    if heads * need_int(m, "vdim") % parts:
        raise ConfigError(f"config.json: {where}.norm_groups must divide heads * vdim, found {parts}")


def _check_attention(m: Dict[str, Any], where: str) -> None:
    heads, kv = need_int(m, "heads"), need_int(m, "kv_heads")
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} heads cannot share {kv} kv_heads evenly")
    dim = need_int(m, "dim")
    need_int(m, "vdim"), need_float(m, "scale")
    mask = _obj(m, "mask", where + ".", optional=True)
    if mask is not None:
        need_int(mask, "size"), need_int(mask, "keep_first", 0, minimum=0)
    rot = _obj(m, "rot", where + ".", optional=True)
    if rot is not None:
        dims = need_int(rot, "dims", minimum=0)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim, found {dims}")
        if need_float(rot, "base") <= 0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive")


def _check_mlp(mlp: Any, where: str) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where}mlp.kind {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not supported "
                          "(dense, moe, or null for none)")
    if mlp["kind"] == "dense":
        need_int(mlp, "ff")
        return
    need_int(_obj(mlp, "expert", where + "mlp."), "ff")
    router = _obj(mlp, "router", where + "mlp.")
    if need_int(router, "top") > need_int(router, "experts"):
        raise ConfigError(f"config.json: {where}mlp.router.top cannot exceed the number of experts")
    shared = _obj(mlp, "shared", where + "mlp.", optional=True)
    if shared is not None:
        need_int(shared, "ff")


@dataclass(frozen=True)
class ZomipelConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[Dict[str, Any], ...]        # as validated from the file
    loop_start: int
    loop_stop: int
    loop_times: int
    raw: Dict[str, Any] = field(default_factory=dict, compare=False)

    ARCHITECTURE = "Zomipel"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ZomipelConfig":
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
            (_check_mamba2 if l["type"] == "mamba2" else _check_attention)(m, where + "mixer")
            if l.get("mlp") is not None:
                _check_mlp(l["mlp"], where)
        loop = _obj(d, "loop", "", optional=True) or {"start": 0, "stop": 0, "times": 1}
        lo, hi = need_int(loop, "start", minimum=0), need_int(loop, "stop", minimum=0)
        times = need_int(loop, "times", minimum=1)
        if not lo <= hi <= len(layers):
            raise ConfigError(f"config.json: loop {lo}..{hi} does not lie within the {len(layers)} layers")
        return cls(architecture=cls.ARCHITECTURE, vocab_size=need_int(d, "vocab"), hidden_size=width,
                   norm_eps=need_float(_obj(d, "norm", ""), "eps"), layers=tuple(copy.deepcopy(layers)),
                   loop_start=lo, loop_stop=hi, loop_times=times, raw=copy.deepcopy(d))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers)),
                "loop": {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}}

    # -- the architecture-neutral description --------------------------------------------------
    def layer_runs(self) -> List[Tuple[int, bool]]:
        """(layer, joins the embedding's output first) for every run, in order."""
        lo, hi = self.loop_start, self.loop_stop
        runs = [(i, False) for i in range(lo)]
        for r in range(self.loop_times if hi > lo else 0):
            runs += [(i, r > 0 and i == lo) for i in range(lo, hi)]
        return runs + [(i, False) for i in range(hi, len(self.layers))]

    def _mamba2(self, p: str, m: Dict[str, Any]) -> PartSpec:
        w = {r: f"{p}.{r}" for r in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}
        w["conv_bias"] = f"{p}.conv.b"
        return PartSpec("mamba2", {
            "hidden_size": self.hidden_size, "n_heads": m["heads"], "v_head_dim": m["vdim"], "state": m["state"],
            "n_groups": m["groups"], "conv_taps": m["conv"], "norm_groups": m.get("norm_groups", 1), "norm_eps": self.norm_eps}, w)

    def _attention(self, p: str, m: Dict[str, Any]) -> Tuple[PartSpec, Optional[PartSpec]]:
        rot, position, mask = m.get("rot"), None, m.get("mask") or {}
        if rot is not None and rot["dims"] > 0:
            position = PartSpec("rotary", {"rotary_dim": rot["dims"], "theta": rot["base"], "pairing": "half", "max_position": MAX_POSITION})
        w = {r: f"{p}.{r}" for r in "qkvo"}
        w.update({f"{r}_bias": f"{p}.{r}.b" for r in "qkv"})
        return PartSpec("attention", {
            "hidden_size": self.hidden_size, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "v_head_dim": m["vdim"], "scale": m["scale"], "bias": "qkv", "window": mask.get("size"),
            "keep_first": mask.get("keep_first") or 0}, w), position

    def _feed_forward(self, p: str, mlp: Dict[str, Any]) -> PartSpec:
        d = self.hidden_size
        if mlp["kind"] == "dense":
            return PartSpec("mlp", {"hidden_size": d, "intermediate_size": mlp["ff"], "activation": "gelu_tanh"},
                            {"up": f"{p}.up", "down": f"{p}.down"})
        w = {"router": f"{p}.router", "router_bias": f"{p}.router.b"}
        w.update({r: p + ".e{e}." + r for r in ("gate", "up", "down")})
        shared = mlp.get("shared")
        if shared is not None:
            w.update({f"shared_{r}": f"{p}.shared.{r}" for r in ("gate", "up", "down")})
            w["shared_weight"] = f"{p}.shared.sg"
        return PartSpec("moe", {
            "hidden_size": d, "intermediate_size": mlp["expert"]["ff"], "n_experts": mlp["router"]["experts"],
            "top": mlp["router"]["top"], "score": "softmax", "renormalize": True, "activation": "silu",
            "shared": shared["ff"] if shared is not None else 0}, w)

    def model_spec(self) -> ModelSpec:
        d = self.hidden_size

        def norm(name: str) -> PartSpec:
            return PartSpec("rmsnorm", {"size": d, "eps": self.norm_eps, "unit_offset": True}, {"weight": name})

        blocks = []
        for i, l in enumerate(self.layers):
            p, position = f"l{i}", None
            if l["type"] == "mamba2":
                mixer = self._mamba2(p + ".mix", l["mixer"])
            else:
                mixer, position = self._attention(p + ".mix", l["mixer"])
            ff = self._feed_forward(p + ".mlp", l["mlp"]) if l.get("mlp") is not None else None
            blocks.append(BlockSpec(kind="parallel", mixer=mixer, feed_forward=ff, norms={"mixer": norm(f"{p}.norm1")}, position=position))
        schedule = tuple(ScheduleEntry(layer=i, cache=n, adds_input=add) for n, (i, add) in enumerate(self.layer_runs()))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab_size, hidden_size=d,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab_size, "hidden_size": d}, {"weight": "embed"}),
            layers=tuple(blocks), schedule=schedule, final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab_size, "hidden_size": d, "tied": True}, {"weight": "embed"}),
            max_position=MAX_POSITION,
        )
