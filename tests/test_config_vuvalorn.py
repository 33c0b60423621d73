"""Vuvalorn's configuration on the CPU: the keys of its ``config.json``, the registry's choice by the ``architecture``
key, the tensors its parts ask for, the schedule with its injections, what the cache keeps (pages and one state row per
layer run), and the plain model's own consistency."""
import json

import numpy as np
import pytest
import torch

import plain_vuvalorn as P
from nncpu_b200.config import VuvalornConfig, config_from_dict
from nncpu_b200.config.specs import AttentionSpec, NormSpec, PositionSpec, RoutedExpertsSpec
from nncpu_b200.engine.model import parameter_list
from nncpu_b200.errors import BadFormat, UnsupportedModel
from nncpu_b200.kernels import ops
from nncpu_b200.parts import base
from nncpu_b200.weights import check_tensors, write_model_folder

CFG = {"architecture": "Vuvalorn", "vocab": 97, "width": 40, "norm": {"eps": 2e-6}, "embedding": {"scale": 3.5}, "logit_scale": 0.7,
       "loop": {"start": 1, "stop": 3, "times": 2},
       "layers": [{"type": "attention", "mixer": {"heads": 6, "kv_heads": 3, "dim": 8, "vdim": 8, "conv": 4, "scale": 0.25, "softcap": 9.0,
                                                  "rot": {"base": 1234.0, "dims": 6}},
                   "mlp": {"kind": "dense", "ff": 20, "limit": 1.5}},
                  {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 5, "vdim": 5, "conv": 2, "scale": 0.5, "softcap": 30.0,
                                                  "rot": {"base": 100.0, "dims": 2}},
                   "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 6, "identity": 3, "top": 2}}},
                  {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 4, "vdim": 4, "conv": 1, "scale": 0.5}, "mlp": None},
                  {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 6, "conv": 3, "scale": 0.4, "softcap": 4.0},
                   "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 3, "identity": 0, "top": 3}}}]}


def test_keys_round_trip_and_specs():
    cfg = config_from_dict(CFG)
    assert isinstance(cfg, VuvalornConfig)
    assert config_from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == CFG
    spec = cfg.model_spec()
    a, b, c, d = spec.layers
    assert {x.kind for x in spec.layers} == {"sandwich"}
    for x in spec.layers:
        assert all((n.kind, n.size, n.eps, n.offset, n.gain) == ("rmsnorm", 40, 2e-6, 0.0, 1.0)
                   for n in (x.norm1, x.norm1_post, x.norm2, x.norm2_post))
    m = a.mixer
    assert (m.n_heads, m.n_kv_heads, m.head_dim, m.scale, m.score_cap, m.conv) == (6, 3, 8, 0.25, 9.0, 4)
    assert m.values_are_keys and m.head_gate and not m.out_gate and not m.qkv_bias and not m.qk_norm_whole and m.qk_norm.size == 8
    assert (m.position.kind, m.position.theta, m.position.rotary_dim) == ("rope_pairs", 1234.0, 6)
    assert c.mixer.position is None and c.mixer.score_cap == 0.0 and c.feed_forward is None
    f = a.feed_forward
    assert (f.kind, f.activation, f.intermediate_size, f.limit) == ("gated_mlp", "swish_clamp", 20, 1.5)
    f = b.feed_forward
    assert (f.n_experts, f.identity, f.top, f.scores, f.correction, f.activation, f.router_bias, f.weight_on, f.weight_scale) == \
        (6, 3, 2, "plain", True, "silu", False, "output", 1.0)
    assert d.feed_forward.identity == 0
    assert spec.embedding.scale == 3.5 and spec.output.tied and spec.output.norm.gain == 0.7


def test_the_loop_adds_a_vector_before_every_pass():
    spec = config_from_dict(CFG).model_spec()
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 2, 3]
    marks = [(i, e.inject.row, e.inject.n_rows, e.inject.table) for i, e in enumerate(spec.schedule) if e.inject is not None]
    assert marks == [(1, 0, 2, "loop.step"), (3, 1, 2, "loop.step")]
    assert all(not e.inject.embedding and e.inject.mix is None for e in spec.schedule if e.inject is not None)
    assert [(l, t) for l, t in P.runs(CFG)] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    plain = {k: v for k, v in CFG.items() if k not in ("loop", "embedding", "logit_scale")}
    spec = config_from_dict(plain).model_spec()
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3] and spec.embedding.scale == spec.output.norm.gain == 1.0
    assert "loop.step" not in {p.name for p in parameter_list(spec)}


def test_tensor_names_and_shapes():
    params = parameter_list(config_from_dict(CFG).model_spec())
    names = {p.name: p.shape for p in params}
    want = {"embed": (97, 40), "final.norm": (40,), "loop.step": (2, 40), "l0.norm1": (40,), "l0.norm1b": (40,), "l0.norm2": (40,),
            "l0.norm2b": (40,), "l0.mix.q": (48, 40), "l0.mix.k": (24, 40), "l0.mix.g": (6, 40), "l0.mix.o": (40, 48),
            "l0.mix.q.norm": (8,), "l0.mix.k.norm": (8,), "l0.mix.q.conv": (48, 4), "l0.mix.k.conv": (24, 4), "l0.mlp.gate": (20, 40),
            "l0.mlp.up": (20, 40), "l0.mlp.down": (40, 20), "l1.mlp.router": (9, 40), "l1.mlp.correction": (9,), "l1.mlp.e5.down": (40, 16),
            "l2.mix.k.conv": (8, 1), "l3.mlp.router": (3, 40), "l3.mlp.e2.gate": (12, 40)}
    for n, shape in want.items():
        assert names[n] == shape, n
    for n in ("l0.mix.v", "head", "l1.mlp.e6.gate", "l1.mlp.router.b", "l0.mix.sink", "l2.mlp.router"):
        assert n not in names, n
    assert not any(p.required for p in params if p.name in ("l2.norm2", "l2.norm2b"))
    check_tensors({k: v for k, v in names.items() if k not in ("l2.norm2", "l2.norm2b")}, params, "file")
    wrong = dict(names)
    wrong["l0.mix.q.conv"] = (48, 3)
    with pytest.raises(BadFormat, match="l0.mix.q.conv"):
        check_tensors(wrong, params, "file")


@pytest.mark.parametrize("change,error", [
    (lambda d: d["layers"][0].update(type="conv"), UnsupportedModel),
    (lambda d: d["layers"][0]["mlp"].update(kind="other"), UnsupportedModel),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), BadFormat),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), BadFormat),
    (lambda d: d["layers"][0]["mixer"].update(vdim=4), BadFormat),
    (lambda d: d["layers"][0]["mixer"].update(conv=0), BadFormat),
    (lambda d: d["layers"][0]["mixer"].update(softcap=-1.0), BadFormat),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), BadFormat),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=5), BadFormat),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=10), BadFormat),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=10), BadFormat),
    (lambda d: d["layers"][1]["mlp"]["router"].update(identity=-1), BadFormat),
    (lambda d: d["layers"][1]["mlp"].pop("expert"), BadFormat),
    (lambda d: d["loop"].update(stop=5), BadFormat),
    (lambda d: d["loop"].update(times=0), BadFormat),
    (lambda d: d.update(logit_scale=0), BadFormat),
    (lambda d: d.pop("norm"), BadFormat),
    (lambda d: d.update(layers=[]), BadFormat),
])
def test_refusals(change, error):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(error):
        config_from_dict(d).model_spec()


def test_parts_refuse_what_they_cannot_do():
    att = dict(kind="attention", name="m", hidden_size=16, n_heads=2, n_kv_heads=1, head_dim=8, scale=1.0, tensor_names="short")
    for more in (dict(conv=3), dict(conv=3, values_are_keys=True, position=PositionSpec("rope_neox", 1e4, 8)),
                 dict(conv=3, values_are_keys=True, q_temp_coef=0.5), dict(head_gate=True, out_gate=True),
                 dict(conv=3, values_are_keys=True, qk_norm=NormSpec("rmsnorm", 16, 1e-6, "m"), qk_norm_whole=True)):
        with pytest.raises(UnsupportedModel):
            base.build("mixer", AttentionSpec(**att, **more))
    with pytest.raises(UnsupportedModel):
        base.build("mixer", AttentionSpec(**att, conv=3, values_are_keys=True), reads_other_cache=True)
    moe = dict(kind="routed_experts", name="f", hidden_size=16, intermediate_size=8, n_experts=4, top=2, router_bias=False)
    for more in (dict(correction=True), dict(identity=2, weight_on="input"), dict(scores="plain", n_groups=2, keep_groups=1), dict(top=5)):
        with pytest.raises(UnsupportedModel):
            base.build("feed_forward", RoutedExpertsSpec(**{**moe, **more}))
    base.build("feed_forward", RoutedExpertsSpec(**{**moe, "top": 5, "identity": 1}))


def test_cache_requests():
    spec = config_from_dict(CFG).model_spec()
    reqs = [base.build("block", b).cache_requests()[0] for b in spec.layers]
    for (kv, st), (G, d, taps, C) in zip(reqs, ((3, 8, 4, 72), (1, 5, 2, 15), (2, 4, 1, 16), (2, 6, 3, 36))):
        assert (kv.n_kv_heads, kv.head_dim, kv.v_head_dim, kv.window) == (G, d, 0, 0)
        # two copies of the last taps - 1 inputs of every channel of q and k, and how long the sequence was at each
        assert st.dtype == torch.float32 and st.shape == (ops.conv_state_floats(taps, C),) and st.shape[0] >= 2 * (taps - 1) * C + 2
        assert st.shape[0] % 4 == 0


def test_random_weights_folder_and_the_plain_model_reads_it(tmp_path):
    folder = write_model_folder(tmp_path / "m", config_from_dict(CFG), 1, torch.float32)
    cfg, w = P.load(folder)
    t = np.random.RandomState(0).randint(0, 97, size=24)
    logits, streams = P.forward(cfg, w, t, True)
    assert logits.shape == (24, 97) and len(streams) == 6 and np.isfinite(logits).all()
    t2 = t.copy()
    t2[17] = (t2[17] + 1) % 97
    again = P.forward(cfg, w, t2)       # causal: what comes later changes nothing earlier
    assert np.allclose(again[:17], logits[:17], atol=1e-12) and not np.allclose(again[17:], logits[17:])


def test_plain_mechanisms():
    u, w = np.arange(1.0, 6.0)[:, None], np.array([[10.0, 1.0, 0.1]])
    assert np.allclose(P.short_conv(u, w)[:, 0], [0.1, 1.2, 12.3, 23.4, 34.5])
    x = np.array([[[1.0, 0.0, 0.0, 2.0, 5.0]]])
    y = P.rotate_pairs(x, [3], {"base": 100.0, "dims": 4})
    assert np.allclose(y[0, 0], [np.cos(3), np.sin(3), -2 * np.sin(0.3), 2 * np.cos(0.3), 5.0])
    assert np.allclose(P.capped(np.array([1e-3, 1e9, -1e9]), 5.0), [1e-3, 5.0, -5.0]) and P.capped(7.0, None) == 7.0
    ids, weights = P.route(np.array([0.5, 0.3, 0.2]), np.array([0.0, 0.0, 0.4]), 2)
    assert ids.tolist() == [2, 0] and weights.tolist() == [0.2, 0.5]
    h = np.array([[2.0, -3.0]])
    zeros = {f"m.e0.{k}": np.zeros((2, 2)) for k in ("gate", "up", "down")}
    out = P.routed_experts(h, {"router": {"experts": 1, "identity": 1, "top": 2}},
                           {"m.router": np.zeros((2, 2)), "m.correction": np.array([9.0, 0.0]), **zeros}, "m")
    assert np.allclose(out, 0.5 * h)        # half the weight on an expert of zeros, half on the input itself
    big = P.clamped_gated(np.array([[10.0]]), {"m.gate": np.ones((1, 1)), "m.up": -np.ones((1, 1)), "m.down": np.ones((1, 1))}, "m", 2.0)
    assert np.allclose(big, 2.0 / (1 + np.exp(-3.404)) * -1.0)
