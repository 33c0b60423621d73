"""Gekilix's configuration on the CPU: the keys of its ``config.json``, the registry's choice by the ``architecture``
key, the tensors its parts ask for, what the cache keeps (pages for the window and the kept first keys, one state row per
recurrent layer), and the plain model's own consistency."""
import json

import numpy as np
import pytest
import torch

import plain_gekilix as P
from nncpu_b200.cache import PAGE, Cache, KVRequest
from nncpu_b200.config import GekilixConfig, config_from_dict
from nncpu_b200.engine.model import parameter_list
from nncpu_b200.errors import BadFormat, InvalidArgument, UnsupportedModel
from nncpu_b200.kernels import ops
from nncpu_b200.parts import base
from nncpu_b200.weights import check_tensors, write_model_folder

CFG = {"architecture": "Gekilix", "vocab": 97, "width": 40, "norm": {"eps": 2e-6},
       "layers": [{"type": "mamba2", "mixer": {"heads": 6, "vdim": 5, "state": 7, "groups": 3, "conv": 3, "norm_groups": 2},
                   "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 6, "top": 2}, "shared": {"ff": 24}}},
                  {"type": "attention",
                   "mixer": {"heads": 6, "kv_heads": 3, "dim": 8, "vdim": 12, "scale": 0.25, "mask": {"size": 9, "keep_first": 4},
                             "rot": {"base": 1234.0, "dims": 6, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 100.0}}},
                   "mlp": {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 3, "top": 3}}},
                  {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 4, "vdim": 4, "scale": 0.5}, "mlp": None}]}


def test_keys_round_trip_and_specs():
    cfg = config_from_dict(CFG)
    assert isinstance(cfg, GekilixConfig)
    assert config_from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == CFG
    spec = cfg.model_spec()
    a, b, c = spec.layers
    assert {x.kind for x in spec.layers} == {"prenorm"} and [e.layer for e in spec.schedule] == [0, 1, 2]
    assert all(x.norm1.offset == 1.0 and x.norm1.eps == 2e-6 for x in spec.layers) and spec.output.norm.offset == 1.0
    m = a.mixer
    assert (m.kind, m.n_heads, m.value_dim, m.state, m.n_groups, m.conv, m.norm_groups, m.eps) == ("state_space", 6, 5, 7, 3, 3, 2, 2e-6)
    m = b.mixer
    assert (m.n_heads, m.n_kv_heads, m.head_dim, m.v_head_dim, m.scale, m.window, m.keep_first) == (6, 3, 8, 12, 0.25, 9, 4)
    p = m.position
    assert (p.kind, p.theta, p.rotary_dim, p.scaling_kind) == ("rope_pairs", 1234.0, 6, "bands")
    assert (p.scaling_factor, p.scaling_slow, p.scaling_fast, p.scaling_original) == (4.0, 1.0, 3.0, 100.0)
    assert m.qk_norm_whole and m.qk_norm.offset == 0.0 and not m.qkv_bias
    assert c.mixer.window == c.mixer.keep_first == 0 and c.mixer.position is None and c.feed_forward is None
    f = a.feed_forward
    assert (f.n_experts, f.top, f.scores, f.weight_on, f.router_bias, f.shared_gate, f.shared.intermediate_size) == \
        (6, 2, "sigmoid", "input", False, True, 24)
    assert b.feed_forward.shared is None and not b.feed_forward.shared_gate


def test_tensor_names_and_shapes():
    params = parameter_list(config_from_dict(CFG).model_spec())
    names = {p.name: p.shape for p in params}
    want = {"embed": (97, 40), "final.norm": (40,), "head": (97, 40), "l0.norm1": (40,), "l0.norm2": (40,),
            "l0.mix.in": (2 * 30 + 2 * 21 + 6, 40), "l0.mix.conv": (72, 3), "l0.mix.conv.b": (72,), "l0.mix.dt_bias": (6,),
            "l0.mix.A_log": (6,), "l0.mix.D": (6,), "l0.mix.norm": (30,), "l0.mix.o": (40, 30), "l0.mlp.router": (6, 40),
            "l0.mlp.shared.gate": (24, 40), "l0.mlp.shared.up": (24, 40), "l0.mlp.shared.down": (40, 24), "l0.mlp.shared.sg": (1, 40),
            "l0.mlp.e5.gate": (16, 40), "l0.mlp.e5.down": (40, 16), "l1.mix.q": (48, 40), "l1.mix.k": (24, 40), "l1.mix.v": (36, 40),
            "l1.mix.q.norm": (48,), "l1.mix.k.norm": (24,), "l1.mix.o": (40, 72), "l1.mlp.e2.up": (20, 40), "l2.mix.q.norm": (8,)}
    for n, shape in want.items():
        assert names[n] == shape, n
    for n in ("l1.mlp.shared.gate", "l1.mlp.shared.sg", "l0.mlp.router.b", "l1.mix.q.b", "l2.mlp.router", "l0.mix.q"):
        assert n not in names, n
    assert not next(p for p in params if p.name == "l2.norm2").required
    check_tensors({k: v for k, v in names.items() if k != "l2.norm2"}, params, "file")
    wrong = dict(names)
    wrong["l0.mix.conv"] = (72, 4)
    with pytest.raises(BadFormat, match="l0.mix.conv"):
        check_tensors(wrong, params, "file")


@pytest.mark.parametrize("change,error", [
    (lambda d: d["layers"][0].update(type="conv"), UnsupportedModel),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), UnsupportedModel),
    (lambda d: d["layers"][0]["mixer"].update(groups=4), BadFormat),
    (lambda d: d["layers"][0]["mixer"].update(norm_groups=4), BadFormat),
    (lambda d: d["layers"][0]["mixer"].pop("conv"), BadFormat),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), BadFormat),
    (lambda d: d["layers"][0]["mlp"].update(shared={}), BadFormat),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=4), BadFormat),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=5), BadFormat),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=10), BadFormat),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("low"), BadFormat),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].update(low=4.0), BadFormat),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=-1), BadFormat),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), BadFormat),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), BadFormat),
    (lambda d: d.pop("norm"), BadFormat),
    (lambda d: d.update(layers=[]), BadFormat),
])
def test_refusals(change, error):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(error):
        config_from_dict(d).model_spec()


def test_cache_requests():
    spec = config_from_dict(CFG).model_spec()
    reqs = [base.build("block", b).cache_requests()[0] for b in spec.layers]
    kv, st = reqs[0]
    # S of every head, then as many inputs of the convolutions as they have taps
    assert kv is None and st.dtype == torch.float32 and st.shape == (ops.ssm_state_floats(6, 5, 3, 7, 3),)
    assert st.shape[0] >= 6 * 7 * 5 + 3 * 72
    kv, st = reqs[1]
    assert st is None and (kv.n_kv_heads, kv.head_dim, kv.v_head_dim, kv.window, kv.keep_first) == (3, 8, 12, 9, 4)


def test_a_windowed_group_keeps_the_pages_of_the_first_keys():
    cache = Cache([(KVRequest(1, 8, 70, keep_first=65), None), (KVRequest(1, 8, 70), None)], [None, None], PAGE * 10, torch.float32, "cpu")
    s = cache.alloc_slot()
    for n in (1, 64, 135, 1, 199):
        cache.prepare([s], [n])
        cache.commit([s], [n])
        length = cache.length(s)
        for g in cache.groups:
            keep, table = g.request.keep_first, g.tables[s]
            for j in range(length):         # a key that some later query sees is in a page that is held, and no other page is
                if length - j < 70 or j < keep:
                    assert table[j // PAGE] >= 0, (length, j)
            for p, page in enumerate(table):
                needed = any(length - j < 70 or j < keep for j in range(p * PAGE, (p + 1) * PAGE))
                assert (page >= 0) == needed, (length, p)
    assert [g.pool.n_held for g in cache.groups] == [4, 2]
    with pytest.raises(InvalidArgument, match="window has already moved"):
        cache.truncate(s, 200)
    cache.check()
    cache.free_slot(s)
    assert all(g.pool.n_held == 0 for g in cache.groups)


def test_rewinding_within_the_kept_pages():
    """Pages that the window moved past but that the kept keys hold can be gone back to."""
    cache = Cache([(KVRequest(1, 8, 10, keep_first=100), None)], [None], PAGE * 4, torch.float32, "cpu")
    s = cache.alloc_slot()
    cache.prepare([s], [120])
    cache.commit([s], [120])
    cache.truncate(s, 40)
    assert cache.length(s) == 40 and cache.groups[0].pool.n_held == 2


def test_random_weights_folder_and_the_plain_model_reads_it(tmp_path):
    folder = write_model_folder(tmp_path / "m", config_from_dict(CFG), 1, torch.float32)
    cfg, w = P.load(folder)
    assert cfg["layers"][2]["mlp"] is None
    t = np.random.RandomState(0).randint(0, 97, size=24)
    logits, streams = P.forward(cfg, w, t, True)
    assert logits.shape == (24, 97) and len(streams) == 3 and np.isfinite(logits).all()
    t2 = t.copy()
    t2[17] = (t2[17] + 1) % 97
    again = P.forward(cfg, w, t2)       # causal: what comes later changes nothing earlier
    assert np.allclose(again[:17], logits[:17], atol=1e-12) and not np.allclose(again[17:], logits[17:])


def test_plain_frequencies_and_visibility():
    r = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 70.0}}
    plain = P.frequencies({"base": 100.0, "dims": 8})
    got = P.frequencies(r)
    assert got[0] == plain[0] and got[3] == plain[3] / 4.0          # wavelengths 6 (short) and 199 (long)
    assert all(plain[i] / 4.0 < got[i] < plain[i] for i in (1, 2))
    see = [[P.visible(i, j, {"size": 3, "keep_first": 2}) for j in range(8)] for i in range(8)]
    assert see[7] == [True, True, False, False, False, True, True, True] and see[1] == [True, True] + [False] * 6
