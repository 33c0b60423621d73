"""Gekilix: a decoder whose ``config.json`` lists its layers one by one.

Every layer is a pre-norm block: x += mixer(norm1(x)); x += feed_forward(norm2(x)), RMS norms with weights stored around
zero.  The mixer is one of

* ``mamba2``: a state space with one decay per head and token (``StateSpaceSpec``);
* ``attention``: grouped-query softmax attention over a sliding window that keeps the sequence's first keys visible, value
  heads of their own size, an RMS norm of q and of k over all their lanes at once (plain weights), and a rotation of
  neighbouring lanes of a head's first ``rot.dims`` with frequencies rescaled between two wavelengths.

The feed-forward is routed experts with a shared one, or absent: sigmoid scores that multiply the experts' input as they
are, SiLU-gated experts, and a shared expert times the sigmoid of one more product per token.  The output is the model's
norm and the matrix ``head``.

``config.json``::

    {"architecture": "Gekilix", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "mamba2", "mixer": {"heads", "vdim", "state", "groups", "conv", "norm_groups"},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k}, "shared": {"ff": S}}},
                {"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"},
                           "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"}}},
                 "mlp": null}, ...]}

``mask``, ``mask.keep_first``, ``rot``, ``rot.scaling``, ``mlp`` and ``mlp.shared`` may be absent (or null).

Tensor names: ``embed``, ``final.norm``, ``head`` and per layer i ``l<i>.norm1`` / ``norm2``, ``l<i>.mix.in / .conv / .conv.b /
.dt_bias / .A_log / .D / .norm / .o`` or ``l<i>.mix.q / .k / .v / .o / .q.norm / .k.norm``, and ``l<i>.mlp.e<j>.gate / .up /
.down``, ``.router``, ``.shared.gate / .up / .down / .sg``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import List, Optional, Tuple

from ..errors import BadFormat, UnsupportedModel
from .registry import register_architecture
from .specs import (AttentionSpec, BlockSpec, EmbeddingSpec, GatedMlpSpec, ModelSpec, NormSpec, OutputSpec, PositionSpec,
                    RoutedExpertsSpec, ScheduleEntry, StateSpaceSpec)


def _int(d: dict, key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int):
        raise BadFormat(f'config.json: {where} needs an integer "{key}", not {v!r}')
    if v < minimum:
        raise BadFormat(f'config.json: {where}: "{key}" is {v}, expected at least {minimum}')
    return v


def _num(d: dict, key: str, where: str) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or v <= 0:
        raise BadFormat(f'config.json: {where} needs a positive number "{key}", not {v!r}')
    return float(v)


def _obj(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise BadFormat(f'config.json: {where} needs an object "{key}", not {v!r}')
    return v


@dataclass(frozen=True)
class GekilixMamba:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "GekilixMamba":
        g = cls(*(_int(m, k, where) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        if g.heads % g.groups:
            raise BadFormat(f"config.json: {where}: {g.heads} heads are no multiple of {g.groups} groups")
        if (g.heads * g.vdim) % g.norm_groups:
            raise BadFormat(f"config.json: {where}: {g.heads} heads of {g.vdim} lanes are no {g.norm_groups} equal parts")
        return g

    def to_dict(self) -> dict:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class GekilixAttention:
    """``window`` 0: every earlier key; ``rot_dims`` 0: no rotation; ``factor`` 0: plain frequencies."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    keep_first: int = 0
    rot_base: float = 0.0
    rot_dims: int = 0
    factor: float = 0.0
    low: float = 0.0
    high: float = 0.0
    original: float = 0.0

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "GekilixAttention":
        heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
        if heads % kv:
            raise BadFormat(f"config.json: {where}: {heads} heads are no multiple of {kv} key/value heads")
        dim = _int(m, "dim", where)
        window = keep = 0
        if m.get("mask") is not None:
            mask = _obj(m, "mask", where)
            window = _int(mask, "size", f"{where}.mask")
            keep = 0 if mask.get("keep_first") is None else _int(mask, "keep_first", f"{where}.mask", minimum=0)
        base, dims, sc = 0.0, 0, (0.0, 0.0, 0.0, 0.0)
        if m.get("rot") is not None:
            rot = _obj(m, "rot", where)
            base, dims = _num(rot, "base", f"{where}.rot"), _int(rot, "dims", f"{where}.rot", minimum=2)
            if dims % 2 or dims > dim:
                raise BadFormat(f"config.json: {where}.rot turns {dims} of a head's {dim} lanes: an even number of at most "
                                "all of them is needed")
            if rot.get("scaling") is not None:
                s, at = _obj(rot, "scaling", f"{where}.rot"), f"{where}.rot.scaling"
                sc = tuple(_num(s, k, at) for k in ("factor", "low", "high", "original"))
                if sc[1] > sc[2]:
                    raise BadFormat(f'config.json: {at}: "low" is {sc[1]:g}, above "high" {sc[2]:g}')
        return cls(heads, kv, dim, _int(m, "vdim", where), _num(m, "scale", where), window, keep, base, dims, *sc)

    def to_dict(self) -> dict:
        m = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window:
            m["mask"] = {"size": self.window, "keep_first": self.keep_first}
        if self.rot_dims:
            m["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.factor:
                m["rot"]["scaling"] = {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}
        return m


@dataclass(frozen=True)
class GekilixMoe:
    """``shared_ff`` 0: no shared expert."""
    ff: int
    experts: int
    top: int
    shared_ff: int = 0

    @classmethod
    def from_dict(cls, d, where: str) -> Optional["GekilixMoe"]:
        if d is None:
            return None
        if not isinstance(d, dict):
            raise BadFormat(f"config.json: {where} is neither null nor an object")
        if d.get("kind") != "moe":
            raise UnsupportedModel(f'config.json: {where} has "kind": {d.get("kind")!r} (supported: "moe")')
        ro = _obj(d, "router", where)
        experts, top = _int(ro, "experts", f"{where}.router"), _int(ro, "top", f"{where}.router")
        if top > experts:
            raise BadFormat(f"config.json: {where}.router takes the top {top} of {experts} experts")
        shared = 0 if d.get("shared") is None else _int(_obj(d, "shared", where), "ff", f"{where}.shared")
        return cls(_int(_obj(d, "expert", where), "ff", f"{where}.expert"), experts, top, shared)

    def to_dict(self) -> dict:
        d = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class GekilixLayer:
    """One entry of ``layers``, checked: ``type`` "mamba2" (``mamba``) or "attention" (``attention``)."""
    type: str
    mamba: Optional[GekilixMamba] = None
    attention: Optional[GekilixAttention] = None
    mlp: Optional[GekilixMoe] = None

    @classmethod
    def from_dict(cls, i: int, d: dict) -> "GekilixLayer":
        where = f"layers[{i}]"
        if not isinstance(d, dict):
            raise BadFormat(f"config.json: {where} is not an object")
        kind = d.get("type")
        m = _obj(d, "mixer", where)
        mlp = GekilixMoe.from_dict(d.get("mlp"), f"{where}.mlp")
        if kind == "mamba2":
            return cls("mamba2", mamba=GekilixMamba.from_dict(m, f"{where}.mixer"), mlp=mlp)
        if kind == "attention":
            return cls("attention", attention=GekilixAttention.from_dict(m, f"{where}.mixer"), mlp=mlp)
        raise UnsupportedModel(f'config.json: {where} has "type": {kind!r} (supported: "mamba2", "attention")')

    def to_dict(self) -> dict:
        m = (self.mamba if self.type == "mamba2" else self.attention).to_dict()
        return {"type": self.type, "mixer": m, "mlp": None if self.mlp is None else self.mlp.to_dict()}


@register_architecture("Gekilix")
@dataclass
class GekilixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[GekilixLayer, ...]
    max_positions: int = 1 << 20  # the design has no table of positions: rotary angles are computed, nothing runs out
    eos_token_id: Tuple[int, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, d: dict) -> "GekilixConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise BadFormat('config.json needs a non-empty list "layers"')
        eos = d.get("eos_token_id")
        eos = tuple(eos) if isinstance(eos, list) else (() if eos is None else (eos,))
        cfg = cls(vocab=_int(d, "vocab", "the model"), width=_int(d, "width", "the model"),
                  norm_eps=_num(_obj(d, "norm", "the model"), "eps", "norm"),
                  layers=tuple(GekilixLayer.from_dict(i, l) for i, l in enumerate(layers)),
                  max_positions=_int(d, "max_positions", "the model") if d.get("max_positions") is not None else 1 << 20,
                  eos_token_id=eos)
        for e in cfg.eos_token_id:
            if isinstance(e, bool) or not isinstance(e, int) or not 0 <= e < cfg.vocab:
                raise BadFormat(f'config.json: "eos_token_id" holds {e!r}')
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [l.to_dict() for l in self.layers]}
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    def model_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps

        def norm(name: str) -> NormSpec:
            return NormSpec("rmsnorm", w, eps, name, suffix="", offset=1.0)

        blocks: List[BlockSpec] = []
        for i, l in enumerate(self.layers):
            p = f"l{i}"
            if l.type == "mamba2":
                m = l.mamba
                mixer = StateSpaceSpec(kind="state_space", name=f"{p}.mix", hidden_size=w, n_heads=m.heads, value_dim=m.vdim,
                                       state=m.state, n_groups=m.groups, conv=m.conv, norm_groups=m.norm_groups, eps=eps)
            else:
                a = l.attention
                position = None
                if a.rot_dims:
                    position = PositionSpec("rope_pairs", a.rot_base, a.rot_dims, scaling_factor=a.factor,
                                            scaling_original=a.original, scaling_fast=a.high, scaling_slow=a.low,
                                            scaling_kind="bands")
                mixer = AttentionSpec(kind="attention", name=f"{p}.mix", hidden_size=w, n_heads=a.heads, n_kv_heads=a.kv_heads,
                                      head_dim=a.dim, v_head_dim=a.vdim, scale=a.scale, window=a.window,
                                      keep_first=a.keep_first, position=position, tensor_names="short",
                                      qk_norm=NormSpec("rmsnorm", a.heads * a.dim, eps, f"{p}.mix"), qk_norm_whole=True)
            ff = None
            if l.mlp is not None:
                f = l.mlp
                shared = None
                if f.shared_ff:
                    shared = GatedMlpSpec(kind="gated_mlp", name=f"{p}.mlp.shared", hidden_size=w, intermediate_size=f.shared_ff,
                                          tensor_names="short")
                ff = RoutedExpertsSpec(kind="routed_experts", name=f"{p}.mlp", hidden_size=w, intermediate_size=f.ff,
                                       n_experts=f.experts, top=f.top, activation="silu", shared=shared, scores="sigmoid",
                                       router_bias=False, weight_on="input", shared_gate=shared is not None)
            blocks.append(BlockSpec(kind="prenorm", norm1=norm(f"{p}.norm1"), mixer=mixer, norm2=norm(f"{p}.norm2"),
                                    feed_forward=ff))
        return ModelSpec(
            architecture=self.architecture, hidden_size=w, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=EmbeddingSpec("embed", self.vocab, w, suffix=""), layers=tuple(blocks),
            schedule=tuple(ScheduleEntry(i) for i in range(len(self.layers))),
            output=OutputSpec(norm=norm("final.norm"), name="head", tied=False, vocab_size=self.vocab, hidden_size=w, suffix=""),
            stop_token_ids=tuple(self.eos_token_id))
