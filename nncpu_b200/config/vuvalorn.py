"""Vuvalorn: a decoder whose ``config.json`` lists its layers one by one and may run a range of them several times.

Every layer is a "sandwich" block, RMS norms with plain weights before and after each sublayer:
x += norm1b(mixer(norm1(x))); x += norm2b(feed_forward(norm2(x))).  The mixer is causal grouped-query attention without a
value projection: q and k pass a short causal convolution per channel right after their projections, a position's value is
its convolved key, then come an RMS norm per head and a rotation of neighbouring lanes of a head's first ``rot.dims``.
Scores are capped, c tanh(z / c), and every head's output is multiplied by the sigmoid of one logit of its own.

The feed-forward is one clamped gated layer, or routed experts (softmax over all of the router's outputs, the choice by score
plus a correction, the chosen scores as they are; the last ``identity`` outputs hand the input on), or absent.

The embedding is multiplied by a constant; the output is the model's norm and the embedding table, times another.
``loop`` names a range of layers that runs ``times`` times in a row with the same weights and a cache and state per pass; row t
of ``loop.step`` is added to the stream before pass t (the first too).

``config.json``::

    {"architecture": "Vuvalorn", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": a}, "logit_scale": b,
     "loop": {"start": i, "stop": j, "times": n},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "conv", "scale", "softcap", "rot": {"base", "dims"}},
                 "mlp": {"kind": "dense", "ff": F, "limit": c}},
                {"type": "attention", "mixer": {...},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "identity": I, "top": k}}}, ...]}

``embedding``, ``logit_scale``, ``loop``, ``softcap``, ``rot``, ``identity`` and a layer's ``mlp`` may be absent (or null).

Tensor names: ``embed``, ``loop.step``, ``final.norm`` and per layer i ``l<i>.norm1 / norm1b / norm2 / norm2b``,
``l<i>.mix.q / .k / .g / .o / .q.conv / .k.conv / .q.norm / .k.norm``, ``l<i>.mlp.gate / .up / .down`` or
``l<i>.mlp.e<j>.gate / .up / .down``, ``.router``, ``.correction``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional, Tuple

from ..errors import BadFormat, UnsupportedModel
from .fields import integer, number, obj
from .registry import register_architecture
from .specs import (AttentionSpec, BlockSpec, EmbeddingSpec, GatedMlpSpec, ModelSpec, NormSpec, OutputSpec, PositionSpec,
                    RoutedExpertsSpec, ScheduleEntry, StreamInjection)

LOOP_TABLE = "loop.step"


@dataclass(frozen=True)
class VuvalornAttention:
    """``softcap`` 0: scores as they are; ``rot_dims`` 0: no rotation."""
    heads: int
    kv_heads: int
    dim: int
    conv: int
    scale: float
    softcap: float = 0.0
    rot_base: float = 0.0
    rot_dims: int = 0

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "VuvalornAttention":
        heads, kv, dim = (integer(m, k, where) for k in ("heads", "kv_heads", "dim"))
        if heads % kv:
            raise BadFormat(f"config.json: {where}: {heads} heads are no multiple of {kv} key/value heads")
        if m.get("vdim") is not None and integer(m, "vdim", where) != dim:
            raise BadFormat(f"config.json: {where}: values are the keys, of {dim} lanes, not {m['vdim']}")
        base, dims = 0.0, 0
        if m.get("rot") is not None:
            rot = obj(m, "rot", where)
            base, dims = number(rot, "base", f"{where}.rot"), integer(rot, "dims", f"{where}.rot", minimum=2)
            if dims % 2 or dims > dim:
                raise BadFormat(f"config.json: {where}.rot turns {dims} of a head's {dim} lanes: an even number of at most "
                                "all of them is needed")
        cap = 0.0 if m.get("softcap") is None else number(m, "softcap", where)
        return cls(heads, kv, dim, integer(m, "conv", where), number(m, "scale", where), cap, base, dims)

    def to_dict(self) -> dict:
        m = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim, "conv": self.conv,
             "scale": self.scale}
        if self.softcap:
            m["softcap"] = self.softcap
        if self.rot_dims:
            m["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return m


@dataclass(frozen=True)
class VuvalornMlp:
    """``kind`` "dense": ``ff`` and ``limit``.  ``kind`` "moe": ``ff`` of an expert, and the router's ``experts``, ``identity``
    and ``top``."""
    kind: str
    ff: int
    limit: float = 0.0
    experts: int = 0
    identity: int = 0
    top: int = 0

    @classmethod
    def from_dict(cls, d, where: str) -> Optional["VuvalornMlp"]:
        if d is None:
            return None
        if not isinstance(d, dict):
            raise BadFormat(f"config.json: {where} is neither null nor an object")
        kind = d.get("kind")
        if kind == "dense":
            return cls("dense", integer(d, "ff", where), number(d, "limit", where))
        if kind == "moe":
            ro, at = obj(d, "router", where), f"{where}.router"
            experts, top = integer(ro, "experts", at), integer(ro, "top", at)
            identity = 0 if ro.get("identity") is None else integer(ro, "identity", at, minimum=0)
            if top > experts + identity:
                raise BadFormat(f"config.json: {at} takes the top {top} of {experts + identity} experts")
            return cls("moe", integer(obj(d, "expert", where), "ff", f"{where}.expert"), 0.0, experts, identity, top)
        raise UnsupportedModel(f'config.json: {where} has "kind": {kind!r} (supported: "dense", "moe")')

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff, "limit": self.limit}
        return {"kind": "moe", "expert": {"ff": self.ff},
                "router": {"experts": self.experts, "identity": self.identity, "top": self.top}}


@dataclass(frozen=True)
class VuvalornLayer:
    attention: VuvalornAttention
    mlp: Optional[VuvalornMlp] = None

    @classmethod
    def from_dict(cls, i: int, d: dict) -> "VuvalornLayer":
        where = f"layers[{i}]"
        if not isinstance(d, dict):
            raise BadFormat(f"config.json: {where} is not an object")
        if d.get("type") != "attention":
            raise UnsupportedModel(f'config.json: {where} has "type": {d.get("type")!r} (supported: "attention")')
        return cls(VuvalornAttention.from_dict(obj(d, "mixer", where), f"{where}.mixer"),
                   VuvalornMlp.from_dict(d.get("mlp"), f"{where}.mlp"))

    def to_dict(self) -> dict:
        return {"type": "attention", "mixer": self.attention.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@register_architecture("Vuvalorn")
@dataclass
class VuvalornConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[VuvalornLayer, ...]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    has_loop: bool = False
    max_positions: int = 1 << 20  # the design has no table of positions: rotary angles are computed, nothing runs out
    eos_token_id: Tuple[int, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, d: dict) -> "VuvalornConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise BadFormat('config.json needs a non-empty list "layers"')
        scale = 1.0 if d.get("embedding") is None else number(obj(d, "embedding", "the model"), "scale", "embedding", 1.0)
        start, stop, times, has_loop = 0, 0, 1, False
        if d.get("loop") is not None:
            lp = obj(d, "loop", "the model")
            start, stop = integer(lp, "start", "loop", minimum=0), integer(lp, "stop", "loop", minimum=0)
            times, has_loop = integer(lp, "times", "loop"), True
            if not start < stop <= len(layers):
                raise BadFormat(f"config.json: loop runs layers {start} to {stop - 1} of {len(layers)}")
        eos = d.get("eos_token_id")
        eos = tuple(eos) if isinstance(eos, list) else (() if eos is None else (eos,))
        cfg = cls(vocab=integer(d, "vocab", "the model"), width=integer(d, "width", "the model"),
                  norm_eps=number(obj(d, "norm", "the model"), "eps", "norm"),
                  layers=tuple(VuvalornLayer.from_dict(i, l) for i, l in enumerate(layers)), embedding_scale=scale,
                  logit_scale=number(d, "logit_scale", "the model", 1.0), loop_start=start, loop_stop=stop, loop_times=times,
                  has_loop=has_loop,
                  max_positions=integer(d, "max_positions", "the model") if d.get("max_positions") is not None else 1 << 20,
                  eos_token_id=eos)
        for e in cfg.eos_token_id:
            if isinstance(e, bool) or not isinstance(e, int) or not 0 <= e < cfg.vocab:
                raise BadFormat(f'config.json: "eos_token_id" holds {e!r}')
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale,
             "layers": [l.to_dict() for l in self.layers]}
        if self.has_loop:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    def schedule(self) -> Tuple[ScheduleEntry, ...]:
        """The layers in running order; the first layer of pass t of the loop carries the addition of row t of
        ``loop.step`` to the stream."""
        n = len(self.layers)
        if not self.has_loop:
            return tuple(ScheduleEntry(i) for i in range(n))
        a, b, times = self.loop_start, self.loop_stop, self.loop_times
        runs: List[ScheduleEntry] = [ScheduleEntry(i) for i in range(a)]
        for t in range(times):
            runs += [ScheduleEntry(i, inject=StreamInjection(table=LOOP_TABLE, n_rows=times, row=t) if i == a else None)
                     for i in range(a, b)]
        return tuple(runs + [ScheduleEntry(i) for i in range(b, n)])

    def model_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps

        def norm(name: str, gain: float = 1.0) -> NormSpec:
            return NormSpec("rmsnorm", w, eps, name, suffix="", gain=gain)

        blocks: List[BlockSpec] = []
        for i, l in enumerate(self.layers):
            p, a, f = f"l{i}", l.attention, l.mlp
            mixer = AttentionSpec(
                kind="attention", name=f"{p}.mix", hidden_size=w, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim,
                scale=a.scale, qk_norm=NormSpec("rmsnorm", a.dim, eps, f"{p}.mix"), tensor_names="short", values_are_keys=True,
                position=PositionSpec("rope_pairs", a.rot_base, a.rot_dims) if a.rot_dims else None, score_cap=a.softcap,
                head_gate=True, conv=a.conv)
            ff = None
            if f is not None and f.kind == "dense":
                ff = GatedMlpSpec(kind="gated_mlp", name=f"{p}.mlp", hidden_size=w, intermediate_size=f.ff,
                                  activation="swish_clamp", limit=f.limit, tensor_names="short")
            elif f is not None:
                ff = RoutedExpertsSpec(kind="routed_experts", name=f"{p}.mlp", hidden_size=w, intermediate_size=f.ff,
                                       n_experts=f.experts, identity=f.identity, top=f.top, activation="silu", scores="plain",
                                       correction=True, router_bias=False)
            blocks.append(BlockSpec(kind="sandwich", norm1=norm(f"{p}.norm1"), mixer=mixer, norm1_post=norm(f"{p}.norm1b"),
                                    norm2=norm(f"{p}.norm2"), feed_forward=ff, norm2_post=norm(f"{p}.norm2b")))
        return ModelSpec(
            architecture=self.architecture, hidden_size=w, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=EmbeddingSpec("embed", self.vocab, w, scale=self.embedding_scale, suffix=""), layers=tuple(blocks),
            schedule=self.schedule(),
            # a constant on the logits is a factor on the final norm's output
            output=OutputSpec(norm=norm("final.norm", gain=self.logit_scale), name="embed", tied=True, vocab_size=self.vocab,
                              hidden_size=w, suffix=""),
            stop_token_ids=tuple(self.eos_token_id))
