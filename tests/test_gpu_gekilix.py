"""The Gekilix design against its plain statement (``plain_gekilix``): every mechanism alone, then the model through
``Engine.step`` cut in every way (whole prompts, token by token, portions down to two tokens, unequal batches, slots,
pages and state rows used again, windows and pages crossed while decoding), and greedy generation through
``Session.generate``, the command line and the trace replay.  Configurations and weights are made here; where random
weights would hide a fault (a window's edge, a kept first key, a key far back, a write the recurrence must remember) the
weights or inputs are made so that it shows."""
import json

import numpy as np
import pytest
import torch

import plain_gekilix as P
from gpu_util import DEV, TOL, check
from nncpu_b200 import Engine, GenerateParams, Model, SamplerParams, Session, SessionParams
from nncpu_b200.cache import PAGE
from nncpu_b200.config import config_from_dict
from nncpu_b200.config.specs import PositionSpec
from nncpu_b200.engine.model import parameter_list
from nncpu_b200.kernels import ops
from nncpu_b200.parts import Runtime, build
from nncpu_b200.weights import random_tensors, write_safetensors

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
STORE = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def rot(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def att(heads, kv, dim, vdim, scale, window=None, keep=0, r=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if r:
        m["rot"] = r
    return {"type": "attention", "mixer": m, "mlp": mlp}


def ssm(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                                    "norm_groups": norm_groups}}


CONFIGS = {
    # odd sizes everywhere and a width that is no multiple of 8 (no tensor-core product takes it); the recurrent layer first;
    # a norm part that ends inside a head; a window of 5 that keeps 2, one of 70 that keeps 130 (three pages); odd value
    # heads; a layer without a feed-forward, one without a shared expert
    "A": {"architecture": "Gekilix", "vocab": 211, "width": 76, "norm": {"eps": 3e-6},
          "layers": [ssm(6, 10, 11, 3, 3, 4, mlp=moe(6, 2, 20, 28)),
                     att(6, 2, 24, 11, 0.3, 5, 2, rot(1e4, 16, (4.0, 1.0, 3.0, 64)), mlp=moe(5, 3, 12)),
                     att(4, 4, 16, 16, 0.25, 70, 130, rot(300.0, 6)),
                     ssm(3, 36, 20, 1, 2, 1, mlp=moe(4, 1, 20, 9))]},
    # sizes the tensor-core paths take: key rows of 64 and 128 lanes, values of the same size, smaller and larger, heads
    # that fill their rows and heads that do not, states of 64, 128 and 200 rows, experts of 64 and 128
    "B": {"architecture": "Gekilix", "vocab": 640, "width": 256, "norm": {"eps": 1e-5},
          "layers": [ssm(8, 64, 128, 2, 4, 2, mlp=moe(8, 2, 64, 128)),
                     att(8, 2, 128, 64, 0.09, 100, 70, rot(1e6, 128, (8.0, 1.0, 4.0, 256)), mlp=moe(12, 3, 128, 64)),
                     ssm(4, 40, 64, 4, 4, 1, mlp=moe(8, 1, 64, 64)),
                     att(4, 1, 64, 64, 0.125, 64, 64, rot(1e4, 32), mlp=None),
                     att(6, 3, 96, 40, 0.1, 77, 1, rot(4e5, 64, (3.0, 0.5, 2.0, 100)), mlp=moe(8, 8, 64, 128)),
                     ssm(2, 96, 200, 1, 2, 6, mlp=moe(4, 2, 136)),
                     att(4, 2, 48, 112, 0.14, None, 0, rot(1e4, 48), mlp=moe(16, 4, 72, 64))]},
    # values at the edges: a window of one key that keeps one, 32 query heads on one key/value head, values of one lane,
    # states of one row and of one column, a convolution of one tap and one of nine, one expert, every expert chosen, norm
    # parts of one lane, no rotation, attention without a window
    "C": {"architecture": "Gekilix", "vocab": 97, "width": 100, "norm": {"eps": 1e-5},
          "layers": [att(32, 1, 8, 1, 0.5, 1, 1, rot(100.0, 2), mlp=moe(1, 1, 8, 4)),
                     ssm(1, 9, 1, 1, 1, 1, mlp=moe(4, 4, 12, 12)),
                     ssm(4, 1, 70, 2, 9, 4, mlp=moe(3, 2, 8)),
                     att(3, 3, 10, 10, 0.3, None, 0, None, mlp=moe(2, 1, 36, 36))]},
}


def write_folder(path, cfg_dict, seed, store, sharpen=None):
    """A model folder with random weights, scaled so that every part of a layer moves the stream; the query and key norms'
    weights are scaled up so that attention is not close to uniform and a key wrongly seen or missed changes the logits
    (less so for a bfloat16 run, whose rounding a sharp softmax and the choice of experts make larger in every layer)."""
    sharpen = sharpen or (4.0 if store == torch.float32 else 2.0)
    config = config_from_dict(cfg_dict)
    tensors = random_tensors(parameter_list(config.model_spec()), seed, store)
    for name in list(tensors):
        if name.endswith((".q.norm", ".k.norm")):
            tensors[name] = (tensors[name].float() * sharpen ** 0.5).to(store)
        elif tensors[name].dim() == 2 and not name.endswith((".conv", ".router", ".sg", ".down")):
            tensors[name] = (tensors[name].float() * 3.0).to(store)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(config.to_dict()))
    write_safetensors(path / "model.safetensors", tensors, {"format": "pt"})
    return path


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("gekilix")
    return {(name, dtype): write_folder(root / f"{name}_{dtype}", cfg, 31 + i, STORE[dtype])
            for i, (name, cfg) in enumerate(CONFIGS.items()) for dtype in DTYPES}


def toks(cfg, n, seed):
    return np.random.RandomState(seed).randint(0, cfg["vocab"], size=n).tolist()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def f32(x):
    return torch.tensor(np.asarray(x), dtype=torch.float32, device=DEV)


# -- attention alone ------------------------------------------------------------------------------

@pytest.mark.parametrize("r", [rot(1e4, 64), rot(2e5, 48, (6.0, 1.0, 4.0, 1024)), rot(5e5, 128, (32.0, 1.0, 4.0, 8192)),
                               rot(300.0, 10, (3.0, 0.5, 2.0, 40)), rot(100.0, 2, (4.0, 1.0, 1.0, 16))])
def test_rotation_frequencies_and_table(r):
    sc = r.get("scaling") or {}
    spec = PositionSpec("rope_pairs", r["base"], r["dims"], scaling_factor=sc.get("factor", 0.0),
                        scaling_original=sc.get("original", 0.0), scaling_fast=sc.get("high", 0.0),
                        scaling_slow=sc.get("low", 0.0), scaling_kind="bands")
    part = build("position", spec)
    part.bind({}, Runtime(DEV, torch.float32))
    f = P.frequencies(r)
    np.testing.assert_allclose(part.inv_freq.cpu().numpy(), f, rtol=1e-6)
    pos = [0, 1, 7, 63, 64, 1000]
    table = torch.empty(len(pos), len(f), 2, device=DEV)
    ops.rope_table(i32(pos), part.inv_freq, table, 1.0, False, part.stretch)
    want = np.stack([np.cos(np.outer(pos, f)), np.sin(np.outer(pos, f))], axis=-1)
    check(table, want, 2e-4, "table")


def cos_sin(pos, r):
    f = P.frequencies(r)
    return f32(np.stack([np.cos(np.outer(pos, f)), np.sin(np.outer(pos, f))], axis=-1))


def pages_of(lens, n_kv, hd, vd, k_row, v_row, dtype, seed):
    """Random keys and values in shuffled pages whose rows are longer than the heads (zeros behind)."""
    g = torch.Generator().manual_seed(seed)
    n_pages = sum((n + PAGE - 1) // PAGE for n in lens) + 2
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((len(lens), max((n + PAGE - 1) // PAGE for n in lens)), -1, dtype=torch.int32)
    kp = torch.zeros(n_pages, n_kv, PAGE, k_row, dtype=dtype)
    vp = torch.zeros(n_pages, n_kv, PAGE, v_row, dtype=dtype)
    ks, vs = [], []
    for b, n in enumerate(lens):
        k = torch.randn(n, n_kv, hd, generator=g).to(dtype)
        v = torch.randn(n, n_kv, vd, generator=g).to(dtype)
        for p in range((n + PAGE - 1) // PAGE):
            page = table[b, p] = order.pop()
            a, z = p * PAGE, min(n, (p + 1) * PAGE)
            kp[page, :, :z - a, :hd] = k[a:z].transpose(0, 1)
            vp[page, :, :z - a, :vd] = v[a:z].transpose(0, 1)
        ks.append(k.double().numpy())
        vs.append(v.double().numpy())
    return kp.to(DEV), vp.to(DEV), table.to(DEV), ks, vs


def plain_rows(q, k, v, positions, scale, window, keep):
    """Attention of queries at the given positions over keys 0 .. len - 1."""
    mask = {"size": window, "keep_first": keep} if window else None
    group = q.shape[1] // k.shape[1]
    out = np.zeros((len(positions), q.shape[1], v.shape[2]))
    for i, p in enumerate(positions):
        see = [j for j in range(p + 1) if P.visible(p, j, mask)]
        for h in range(q.shape[1]):
            s = (k[see, h // group] @ q[i, h]) * scale
            w = np.exp(s - s.max())
            out[i, h] = (w / w.sum()) @ v[see, h // group]
    return out


@pytest.mark.parametrize("nh,nkv,hd,vd,window,keep", [
    (4, 2, 64, 64, 100, 70), (2, 1, 128, 64, 64, 64), (8, 2, 128, 56, 36, 24), (16, 1, 64, 7, 10, 130), (12, 4, 96, 112, 200, 1),
    (6, 2, 40, 33, 30, 3), (3, 1, 128, 128, 129, 63), (5, 5, 64, 64, 70, 65), (1, 1, 128, 40, 3, 200), (2, 2, 128, 128, 1, 1),
    (32, 1, 128, 64, 50, 128), (4, 4, 24, 8, 65, 5)])
def test_windows_with_kept_keys_and_values_of_their_own_size_in_every_kernel(nh, nkv, hd, vd, window, keep):
    """The 32-bit kernel and the three bfloat16 kernels: a portion of 9 tokens, a whole prompt of 67, a portion of 130 that
    crosses pages and windows, then one token each with the keys in one split, in several that a cluster merges, and in
    several through scratch."""
    lens, new = [150, 67, 420], [9, 67, 130]
    k_row, v_row = ops.attention_rows(hd, vd)
    g = torch.Generator().manual_seed(nh + hd + vd)
    kp, vp, table, ks, vs = pages_of(lens, nkv, hd, vd, k_row, v_row, torch.bfloat16, 3)
    q = [torch.randn(n, nh, hd, generator=g).bfloat16() for n in new]
    n = sum(new)
    qp = torch.zeros(n, nh, k_row, dtype=torch.bfloat16)
    qp[:, :, :hd] = torch.cat(q)
    qp = qp.view(n, -1).to(DEV)
    cu = i32(np.cumsum([0] + new).tolist())
    tok_pos = i32([p for b in range(3) for p in range(lens[b] - new[b], lens[b])])
    tok_seq = i32([b for b in range(3) for _ in range(new[b])])
    want = np.concatenate([plain_rows(q[b].double().numpy(), ks[b], vs[b], range(lens[b] - new[b], lens[b]), 0.2, window, keep)
                           for b in range(3)]).reshape(n, -1)
    kw = {"keep": keep, "v_lanes": vd}
    out = torch.full((n, nh * vd), float("nan"), dtype=torch.float32, device=DEV)
    ops.attention(qp.float(), kp.float(), vp.float(), table, tok_seq, tok_pos, out, nh, nkv, k_row, 0.2, window, v_row, **kw)
    check(out, want, 2e-5, "32-bit kernel")
    out = torch.full((n, nh * vd), float("nan"), dtype=torch.bfloat16, device=DEV)
    ops.attention_prefill_mma(qp, kp, vp, table, cu, tok_pos, out, 3, nh, nkv, k_row, 0.2, window, **kw)
    check(out, want, 2e-2, "portion kernel")
    out = torch.full((n, nh * vd), float("nan"), dtype=torch.bfloat16, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.attention_prefill_tc(qp, kp, vp, table, cu, tok_pos, out, status, 3, nh, nkv, k_row, 0.2, window, **kw)
    assert int(status.item()) == 0
    check(out, want, 2e-2, "tcgen05 prompt kernel")
    last = [int(cu[b + 1]) - 1 for b in range(3)]
    for n_splits, scratched in ((1, False), (2, False), (5, False), (3, True)):
        scratch = torch.empty(ops.attention_decode_scratch_floats(3, nh, nkv, v_row, n_splits), device=DEV) if scratched else None
        got = torch.full((3, nh * vd), float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.attention_decode_mma(qp[last].contiguous(), kp, vp, table, i32([0, 1, 2]), i32([l - 1 for l in lens]), got, scratch,
                                 nh, nkv, k_row, 0.2, window, n_splits, **kw)
        check(got, want[last], 2e-2, f"decode, {n_splits} splits")


@pytest.mark.parametrize("window,keep", [(1, 1), (5, 3), (64, 64), (65, 63), (100, 65), (30, 128)])
def test_a_key_just_inside_and_just_outside_a_window_and_the_kept_keys(window, keep):
    """One key stands far out: seen, it is all of the answer; unseen, none of it.  Keys on both sides of the window's edge and
    of the last kept key, in the 32-bit kernel and in the bfloat16 kernels."""
    hd = 64
    for pos in (window + keep + 3, 300):
        kp, vp, table, ks, vs = pages_of([pos + 1], 1, hd, hd, hd, hd, torch.bfloat16, 1)
        for j in sorted({0, keep - 1, keep, pos - window, pos - window + 1, pos} & set(range(pos + 1))):
            q = torch.zeros(1, 1, hd, dtype=torch.bfloat16)
            q[0, 0] = torch.tensor(np.sign(ks[0][j, 0])).bfloat16()          # its score is by far the largest
            seen = P.visible(pos, j, {"size": window, "keep_first": keep})
            want = plain_rows(q.double().numpy(), ks[0], vs[0], [pos], 1.0, window, keep).reshape(1, -1)
            if seen and pos > 20:
                assert np.abs(want - vs[0][j]).max() < 0.1, "the key does not stand out"
            args = (table, i32([0]), i32([pos]))
            cu, qd = i32([0, 1]), q.view(1, -1).to(DEV)
            out = torch.empty(1, hd, dtype=torch.float32, device=DEV)
            ops.attention(qd.float(), kp.float(), vp.float(), *args, out, 1, 1, hd, 1.0, window, keep=keep)
            check(out, want, 1e-4, f"32-bit, key {j} of {pos}")
            out = torch.empty(1, hd, dtype=torch.bfloat16, device=DEV)
            ops.attention_decode_mma(qd, kp, vp, *args, out, None, 1, 1, hd, 1.0, window, 2, keep=keep)
            check(out, want, 2e-2, f"decode, key {j} of {pos}")
            ops.attention_prefill_mma(qd, kp, vp, table, cu, args[2], out, 1, 1, 1, hd, 1.0, window, keep=keep)
            check(out, want, 2e-2, f"portion kernel, key {j} of {pos}")
            status = torch.zeros(1, dtype=torch.int32, device=DEV)
            ops.attention_prefill_tc(qd, kp, vp, table, cu, args[2], out, status, 1, 1, 1, hd, 1.0, window, keep=keep)
            check(out, want, 2e-2, f"prompt kernel, key {j} of {pos}")


@pytest.mark.parametrize("nh,nkv,hd,vd,dims", [(4, 2, 64, 64, 64), (6, 2, 24, 11, 16), (8, 2, 128, 56, 40), (3, 1, 7, 5, 2),
                                               (16, 4, 128, 128, 128), (5, 5, 96, 40, 0)])
def test_norm_over_whole_rows_rotation_of_neighbours_and_append(nh, nkv, hd, vd, dims):
    """Queries and pages from the projections, in rows of the heads' own sizes (32-bit) and in the tensor-core kernels' rows
    (bfloat16, zeros behind); then a decode step from the projections, whose pages must be the same bits."""
    n = 70
    g = torch.Generator().manual_seed(hd + vd)
    pos = list(range(40, 40 + n))
    r = rot(300.0, dims, (4.0, 1.0, 3.0, 100)) if dims else None
    ld = (nh + nkv) * hd + nkv * vd
    qkv = torch.randn(n, ld, generator=g) * 2
    qg, kg = torch.randn(nh * hd, generator=g) + 1, torch.randn(nkv * hd, generator=g) + 1
    x = qkv.double().numpy()

    def heads(a, gamma, h):
        a = (P.rms(a, 1e-5) * gamma.double().numpy()).reshape(n, h, hd)
        return P.rotate_pairs(a, pos, r) if r else a

    q = heads(x[:, :nh * hd], qg, nh)
    k = heads(x[:, nh * hd:(nh + nkv) * hd], kg, nkv)
    v = x[:, (nh + nkv) * hd:].reshape(n, nkv, vd)
    cs = cos_sin(pos, r) if r else None
    table = i32([[3, 0]])
    for dt, rows, tol in ((torch.float32, (hd, vd), 1e-5), (torch.bfloat16, ops.attention_rows(hd, vd), 8e-3)):
        kp = torch.full((4, nkv, PAGE, rows[0]), 9.0, dtype=dt, device=DEV)
        vp = torch.full((4, nkv, PAGE, rows[1]), 9.0, dtype=dt, device=DEV)
        q_out = torch.full((n, nh * rows[0]), 9.0, dtype=dt, device=DEV)
        ops.qk_whole_norm_append(qkv.to(DEV), qg.to(DEV), kg.to(DEV), 1e-5, cs, i32([0] * n), i32(pos), table, kp, vp, q_out, nh, nkv,
                                 hd, vd)
        got = q_out.view(n, nh, -1)
        check(got[..., :hd], q, tol, "queries")
        assert float(got[..., hd:].float().abs().sum()) == 0.0, "zeros behind a head"
        for t in (0, 23, 24, 69):
            page, row = (3, pos[t]) if pos[t] < PAGE else (0, pos[t] - PAGE)
            check(kp[page, :, row, :hd], k[t], tol, f"key of token {t}")
            check(vp[page, :, row, :vd], v[t], tol, f"value of token {t}")
            assert float(kp[page, :, row, hd:].float().abs().sum() + vp[page, :, row, vd:].float().abs().sum()) == 0.0
        assert float(kp[1].float().min()) == 9.0, "a page of nobody was written"
    # a decode step: three sequences, one token each
    if nh // nkv > 16:
        return
    lens, window, keep = [1, 65, 300], 50, 70
    k_row, v_row = ops.attention_rows(hd, vd)
    kp, vp, table, ks, vs = pages_of(lens, nkv, hd, vd, k_row, v_row, torch.bfloat16, 6)
    dpos = [l - 1 for l in lens]
    pos = dpos
    n = 3
    x = x[:3]
    qkv = qkv[:3].contiguous()
    q = heads(x[:, :nh * hd], qg, nh)
    k = heads(x[:, nh * hd:(nh + nkv) * hd], kg, nkv)
    want = []
    for b in range(3):
        kb, vb = ks[b].copy(), vs[b].copy()
        kb[-1], vb[-1] = k[b], x[b, (nh + nkv) * hd:].reshape(nkv, vd)
        want.append(plain_rows(q[b:b + 1], kb, vb, [dpos[b]], 0.2, window, keep).reshape(-1))
    cs = cos_sin(dpos, r) if r else None
    kp2, vp2 = kp.clone(), vp.clone()
    for n_splits in (1, 3):
        got = torch.empty(3, nh * vd, dtype=torch.bfloat16, device=DEV)
        ops.attention_decode_mma_from_qkv(qkv.to(DEV), qg.to(DEV), kg.to(DEV), 1e-5, cs, kp, vp, True, table, i32([0, 1, 2]), i32(dpos),
                                          got, None, nh, nkv, hd, 0.2, window, n_splits, keep=keep, v_head_dim=vd, whole_norm=True,
                                          rot_pairs=True)
        check(got, np.stack(want), 2e-2, f"decode from the projections, {n_splits} splits")
    q_out = torch.empty(3, nh * k_row, dtype=torch.bfloat16, device=DEV)
    ops.qk_whole_norm_append(qkv.to(DEV), qg.to(DEV), kg.to(DEV), 1e-5, cs, i32([0, 1, 2]), i32(dpos), table, kp2, vp2, q_out, nh, nkv,
                             hd, vd)
    check(kp, kp2, 8e-3, "pages of keys")        # (the two add a row's squares in different orders)
    assert torch.equal(vp, vp2), "the pages of values differ from the separate append kernel's"


# -- the state space alone ------------------------------------------------------------------------

SSM_SIZES = [(6, 10, 3, 11, 3, 4), (8, 64, 2, 128, 4, 2), (1, 9, 1, 1, 1, 1), (4, 1, 2, 70, 9, 4), (2, 96, 1, 200, 2, 6),
             (4, 40, 4, 64, 4, 1), (3, 33, 1, 256, 4, 1), (2, 16, 1, 300, 4, 2)]


def plain_mixer_core(proj, H, Pd, G, N, w):
    """From the projections to y (before gate and norm)."""
    T, inner = proj.shape[0], H * Pd
    xbc = P.silu(P.short_conv(proj[:, inner:2 * inner + 2 * G * N], w["conv"], w["b"]))
    dt = P.softplus(proj[:, 2 * inner + 2 * G * N:2 * inner + 2 * G * N + H] + w["dt_bias"])
    return P.state_space(xbc[:, :inner].reshape(T, H, Pd), xbc[:, inner:inner + G * N].reshape(T, G, N),
                         xbc[:, inner + G * N:].reshape(T, G, N), dt, w["a_log"], w["d"]).reshape(T, inner)


class SsmRunner:
    def __init__(self, H, Pd, G, N, taps, w, store, n_slots=4):
        self.sizes = (H, Pd, G, N, taps)
        self.H, self.inner = H, H * Pd
        self.store = store
        self.w = {k: f32(v) for k, v in w.items()}
        self.state = torch.full((n_slots + 1, ops.ssm_state_floats(*self.sizes)), 7.0, dtype=torch.float32, device=DEV)

    def run(self, parts, kernel="scan"):        # [(slot, start, rows)] -> y
        proj = f32(np.concatenate([rows for _, _, rows in parts]))
        n = proj.shape[0]
        pos = i32([st + j for _, st, rows in parts for j in range(len(rows))])
        seq = i32([i for i, (_, _, rows) in enumerate(parts) for _ in rows])
        cu = i32(np.cumsum([0] + [len(rows) for _, _, rows in parts]).tolist())
        slots = i32([s for s, _, _ in parts])
        y = torch.full((n, self.inner), float("nan"), dtype=torch.float32, device=DEV)
        w = self.w
        for s, st, _ in parts:
            if st == 0 and s >= 0:
                self.state[s].zero_()
        if kernel == "step":
            ops.ssm_step(proj, w["conv"], w["b"], self.state, pos, slots, w["dt_bias"], w["a_log"], w["d"], y, self.sizes)
            return y
        xc = torch.empty(n, ops.ssm_row(*self.sizes[:4]), dtype=self.store, device=DEV)
        gd = torch.empty(n, 2 * self.H, dtype=torch.float32, device=DEV)
        ops.ssm_conv(proj, w["conv"], w["b"], self.state, seq, pos, slots, cu, w["dt_bias"], w["a_log"], xc, gd, self.sizes)
        fn = ops.ssm_chunk_scan if kernel == "chunks" else ops.ssm_scan
        fn(proj, xc, gd, self.state, slots, cu, pos, w["d"], y, len(parts), self.sizes)
        return y


def ssm_weights(g, H, Pd, G, N, taps):
    C = H * Pd + 2 * G * N
    return {"conv": g.randn(C, taps) * 0.5, "b": g.randn(C) * 0.3, "dt_bias": g.randn(H) - 1.0, "a_log": g.randn(H) * 0.7 - 1.0,
            "d": g.randn(H)}


@pytest.mark.parametrize("H,Pd,G,N,taps,_ng", SSM_SIZES)
def test_state_space_alone_in_portions_batches_and_steps(H, Pd, G, N, taps, _ng):
    """Convolution, step sizes and recurrence against the plain rule: whole; in portions beside another sequence and a
    padding sequence (the same bits, 32-bit); a few tokens and then token by token through the step kernel; and in
    chunks on the tensor cores, whole and in portions that end inside chunks, then stepped on from there."""
    g = np.random.RandomState(H * 100 + N)
    w = ssm_weights(g, H, Pd, G, N, taps)
    row = 2 * H * Pd + 2 * G * N + H + 3
    seqs = [g.randn(150, row), g.randn(70, row)]
    want = [plain_mixer_core(s, H, Pd, G, N, w) for s in seqs]
    m = SsmRunner(H, Pd, G, N, taps, w, torch.float32)
    whole = m.run([(0, 0, seqs[0])]).clone()
    check(whole, want[0], 2e-5, "whole")
    pad = g.randn(3, row)
    rows, at = [], 0
    for i, k in enumerate((2, 3, 64, 1, 80)):
        other = [(2, 0, seqs[1][:41])] if i == 0 else [(2, 41, seqs[1][41:])] if i == 2 else []
        y = m.run([(1, at, seqs[0][at:at + k]), (-1, 0, pad)] + other)
        rows.append(y[:k].clone())
        assert float(y[k:k + 3].abs().max()) == 0.0, "a padding sequence"
        if i == 0:
            check(y[k + 3:], want[1][:41], 2e-5, "another sequence")
        if i == 2:
            check(y[k + 3:], want[1][41:], 2e-5, "another sequence goes on")
        at += k
    assert torch.equal(torch.cat(rows), whole), "portions beside others are not the same bits"
    assert torch.equal(m.state[0], m.state[1]), "the states differ"
    m.run([(3, 0, seqs[0][:5])])
    steps = [m.run([(3, t, seqs[0][t:t + 1]), (-1, 0, pad[:1])], "step")[:1].clone() for t in range(5, 150)]
    check(torch.cat(steps), want[0][5:], 2e-5, "token by token")
    check(m.state[3], m.state[0], 2e-5, "the state after the steps")
    if N > ops.SSM_CHUNK_MAX_STATE:
        return
    m = SsmRunner(H, Pd, G, N, taps, w, torch.bfloat16)
    y = m.run([(0, 0, seqs[0]), (-1, 0, pad), (2, 0, seqs[1])], "chunks")
    check(y[:150], want[0], 1.5e-2, "chunks, whole")
    check(y[153:], want[1], 1.5e-2, "chunks, another sequence")
    assert float(y[150:153].abs().max()) == 0.0
    scan = SsmRunner(H, Pd, G, N, taps, w, torch.bfloat16)
    y0 = scan.run([(0, 0, seqs[0])])
    check(y[:150], y0, 2e-4, "chunks against the scan on the same rounded inputs")
    check(m.state[0], scan.state[0], 2e-4, "the state after the chunks")
    rows, at = [], 0
    for k in (30, 64, 17, 39):
        rows.append(m.run([(1, at, seqs[0][at:at + k])], "chunks").clone())
        at += k
    check(torch.cat(rows), y0, 2e-4, "chunks in portions")
    check(m.state[1], scan.state[0], 2e-4, "the state after the portions")
    y1 = m.run([(1, 150, seqs[1][:1]), (0, 150, seqs[1][:1])], "step")
    check(y1[0], y1[1], 2e-4, "a step on from the portions and from the whole")


def test_a_write_far_back_that_the_last_query_asks_for():
    """Slow decays, one token's B and x large and every other one's small: 600 tokens later C asks for its B.  In order, in
    chunks and token by token."""
    H, Pd, G, N, taps = 2, 16, 1, 32, 1
    g = np.random.RandomState(4)
    T, inner = 640, H * Pd
    w = {"conv": np.ones((inner + 2 * G * N, 1)), "b": np.zeros(inner + 2 * G * N), "dt_bias": np.full(H, -3.0),
         "a_log": np.full(H, -6.0), "d": np.zeros(H)}
    proj = g.randn(T, 2 * inner + 2 * N + H) * 0.05
    proj[30, inner:2 * inner] = g.randn(inner) * 4 + 4
    b = np.abs(g.randn(N)) * 3 + 1
    proj[30, 2 * inner:2 * inner + N] = b
    proj[T - 1, 2 * inner + N:2 * inner + 2 * N] = b
    want = plain_mixer_core(proj, H, Pd, G, N, w)
    without = proj.copy()
    without[30] = 0.0
    assert np.abs(plain_mixer_core(without, H, Pd, G, N, w)[-1]).max() < 0.05 * np.abs(want[-1]).max(), "the write does not show"
    for store, kernel, tol in ((torch.float32, "scan", 2e-5), (torch.bfloat16, "chunks", 1e-2)):
        m = SsmRunner(H, Pd, G, N, taps, w, store)
        y = m.run([(0, 0, proj)], kernel)
        check(y[-1], want[-1], tol, kernel)
        m.run([(1, 0, proj[:100])], kernel)
        for t in range(100, T):
            y = m.run([(1, t, proj[t:t + 1])], "step")
        check(y[0], want[-1], tol, f"{kernel}, then token by token")


def test_strong_and_weak_decays_in_one_chunk():
    """Decays that wipe the state at once beside tokens that hardly decay at all: the sums of logarithms in a chunk reach
    hundreds, and what is asked for lies between two tokens of small decay."""
    H, Pd, G, N, taps = 3, 32, 1, 64, 2
    g = np.random.RandomState(9)
    w = ssm_weights(g, H, Pd, G, N, taps)
    w["a_log"] = np.array([1.5, 0.0, -8.0])
    proj = g.randn(200, 2 * H * Pd + 2 * G * N + H)
    proj[:, -H:] = np.where(g.rand(200, H) < 0.3, 9.0, -6.0)
    want = plain_mixer_core(proj, H, Pd, G, N, w)
    check(SsmRunner(H, Pd, G, N, taps, w, torch.float32).run([(0, 0, proj)]), want, 5e-5, "in order")
    check(SsmRunner(H, Pd, G, N, taps, w, torch.bfloat16).run([(0, 0, proj)], "chunks"), want, 1.5e-2, "chunks")


@pytest.mark.parametrize("inner,groups", [(60, 4), (512, 2), (4, 4), (9000, 1), (4096, 8), (192, 6)])
def test_gate_then_norm_in_parts(inner, groups):
    g = np.random.RandomState(inner)
    y, z, w = g.randn(9, inner) * 3, g.randn(9, inner + 5), g.randn(inner)
    want = P.gated_group_norm(y, z[:, :inner], w, groups, 1e-5)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 8e-3)):
        out = torch.empty(9, inner, dtype=dt, device=DEV)
        ops.ssm_gated_norm(f32(y), f32(z), f32(w), 1e-5, out, groups)
        check(out, want, tol, "gated norm")


# -- the feed-forward alone -----------------------------------------------------------------------

@pytest.mark.parametrize("n_experts,top", [(5, 2), (8, 3), (4, 4), (1, 1), (70, 6), (300, 1)])
def test_router_with_sigmoid_scores_and_a_gate(n_experts, top):
    g = torch.Generator().manual_seed(n_experts)
    n, width = 37, 72
    z = torch.randn(n, n_experts + 1, generator=g) * 2
    ids, ws = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
    gate = torch.empty(n, device=DEV)
    s = P.sigmoid(z.double().numpy())
    chosen = [P.route(s[t, :n_experts], top) for t in range(n)]
    ops.moe_route(z.to(DEV), top, ids, ws, ("sigmoid",), gate)
    assert ids.cpu().numpy().tolist() == [c.tolist() for c in chosen]
    check(ws, np.stack([s[t, c] for t, c in enumerate(chosen)]), 2e-6, "weights: the scores as they are")
    check(gate, s[:, -1], 2e-6, "gate")
    ops.moe_route(z[:, :n_experts].contiguous().to(DEV), top, ids, ws, ("sigmoid",))
    assert ids.cpu().numpy().tolist() == [c.tolist() for c in chosen]
    x, w = torch.randn(n, width, generator=g), torch.randn(n_experts + 1, width, generator=g) * 0.2
    s = P.sigmoid(x.double().numpy() @ w.double().numpy().T)
    ops.moe_router(x.to(DEV), w.to(DEV), None, top, ids, ws, ("sigmoid",), gate)
    chosen = [P.route(s[t, :n_experts], top) for t in range(n)]
    assert ids.cpu().numpy().tolist() == [c.tolist() for c in chosen]
    check(ws, np.stack([s[t, c] for t, c in enumerate(chosen)]), 1e-5, "weights, one launch")
    check(gate, s[:, -1], 1e-5, "gate, one launch")


def ff_part(rt, width, f, seed, store):
    """The framework's part with random weights, and the same weights for the plain statement."""
    cfg = {"architecture": "Gekilix", "vocab": 8, "width": width, "norm": {"eps": 1e-5},
           "layers": [ssm(1, 8, 8, 1, 1, 1, mlp=f)]}
    spec = config_from_dict(cfg).model_spec().layers[0].feed_forward
    part = build("feed_forward", spec)
    tensors = random_tensors(part.params(), seed, store)
    tensors = {k: (v.float() * 4.0).to(store) if not k.endswith((".router", ".sg")) else v for k, v in tensors.items()}
    plain = {k: v.double().numpy() for k, v in tensors.items()}
    part.bind({k: v.to(DEV) for k, v in tensors.items()}, rt)
    return part, plain


class Ctx:
    branch_is_fresh, out_scale, next_norm, n_tokens = False, 1.0, None, 0

    def __init__(self):
        self.memo = {}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 3, 9, 70, 300])
@pytest.mark.parametrize("width,f", [(256, moe(8, 2, 64, 128)), (88, moe(5, 1, 40, 24)), (100, moe(6, 3, 20, 28)), (128, moe(4, 2, 64)),
                                     (136, moe(8, 2, 72, 9)), (136, moe(4, 4, 9, 72))])
def test_experts_with_weighted_inputs_and_a_gated_shared_one(dtype, n, width, f):
    """Few tokens (a block per slot) and many (sorted, grouped products), with a shared expert of another size, without one, and
    sizes that only one of the two layouts of gate and up rows takes."""
    rt = Runtime(DEV, STORE[dtype])
    part, w = ff_part(rt, width, f, n + width, STORE[dtype])
    g = torch.Generator().manual_seed(n)
    x = torch.randn(n, width, generator=g).to(STORE[dtype])
    before = torch.randn(n, width, generator=g)
    out = before.clone().to(DEV)
    part.forward(Ctx(), x.to(DEV), out)
    want = P.routed_experts(x.double().numpy(), f, w, "l0.mlp")
    check(out - before.to(DEV), want, 3e-5 if dtype == "float32" else 3e-2, "feed-forward")
    rt.check_status()
    # a weight on the output answers otherwise: what multiplies the input shows
    other = np.zeros_like(want)
    s = P.sigmoid(x.double().numpy() @ w["l0.mlp.router"].T)
    for t in range(n):
        for e in P.route(s[t], f["router"]["top"]):
            other[t] += s[t, e] * P.gated_expert(x[t:t + 1].double().numpy(), w, f"l0.mlp.e{e}")[0]
    assert n < 9 or np.abs(other - want).max() > 0.05 * np.abs(want).max()


@pytest.mark.parametrize("width", [256, 1024, 4100, 8192])
def test_the_sum_of_the_experts_leaves_the_norm_that_follows(width):
    g = np.random.RandomState(width)
    n, top = 5, 2
    y, out, branch, gate = g.randn(n * top, width), g.randn(n, width), g.randn(n, width), g.rand(n)
    rows = g.permutation(n * top)
    gamma = g.randn(width) * 0.1
    xs = f32(out)
    normed = torch.empty(n, width, dtype=torch.bfloat16, device=DEV)
    ops.moe_combine(f32(y), i32(rows.tolist()), None, xs, top, f32(branch), f32(gate), (f32(gamma), 1.0, 1e-5, normed))
    want = out + y[rows].reshape(n, top, width).sum(axis=1) + gate[:, None] * branch
    check(xs, want, 1e-6, "stream")
    check(normed, P.norm(want, gamma, 1e-5), 8e-3, "norm")


@pytest.mark.parametrize("n_tokens", [1, 16, 40, 130, 600])
def test_a_norm_with_weights_around_zero_rides_on_the_products(folders, n_tokens):
    """The same step with the norms carried by products and closing kernels and with every norm a kernel of its own."""
    model = Model.load(folders["B", "bfloat16"])
    t = toks(CONFIGS["B"], n_tokens, 3)
    got = []
    for carried in (True, False):
        if not carried:
            for b in model.blocks:
                for norm in (b.norm1, b.norm2):
                    if norm is not None:
                        norm.request = lambda ctx, residual: None
        engine = Engine(model, max_tokens=1024, use_graphs=False)
        got.append(engine.step([engine.alloc_slot()], [t], [list(range(n_tokens))]).clone())
    close(got[0], got[1].double().cpu().numpy(), "bfloat16", f"{n_tokens} tokens")


# -- the model ------------------------------------------------------------------------------------

def close(got, want, dtype, what):
    """Logits against the plain model's.  float32: the largest difference within 1e-4 of the largest logit.
    bfloat16: rounding of the activations to 8 bits of mantissa is the design's own noise (and where two router scores
    are closer than that noise a token may go to another expert), so the measure is the root mean square of the
    differences over all the rows given, held to 5 % of the logits' own; a fault of the cache, the state or a window
    moves far more than that with these weights, and the float32 runs hold the same code to 1e-4."""
    if dtype == "float32":
        return check(got, want, TOL[dtype], what)
    g = got.detach().double().cpu().numpy()
    w = np.asarray(want, dtype=np.float64).reshape(g.shape)
    assert np.isfinite(g).all(), f"{what}: NaN or infinity"
    rms = float(np.sqrt(np.mean((g - w) ** 2)) / np.sqrt(np.mean(w ** 2)))
    assert rms <= 5e-2, f"{what}: root mean square of the differences {rms:.3e} of the logits' own"


class Rows:
    """Rows of logits that arrive one step at a time: float32 rows are judged as they come, bfloat16 rows together
    at the end (see ``close``)."""

    def __init__(self, dtype, what):
        self.dtype, self.what, self.got, self.want = dtype, what, [], []

    def add(self, got, want, where=""):
        if self.dtype == "float32":
            return close(got, want, self.dtype, f"{self.what} {where}")
        self.got.append(got.detach().float().reshape(-1).clone())
        self.want.append(np.asarray(want, dtype=np.float64).reshape(-1))

    def done(self):
        if self.got:
            close(torch.stack(self.got), np.stack(self.want), self.dtype, self.what)


def plain_logits(folder, tokens):
    cfg, w = P.load(folder)
    return P.forward(cfg, w, tokens)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_every_position_and_layer(folders, name, dtype):
    cfg = CONFIGS[name]
    t = toks(cfg, 150, 1)
    pcfg, w = P.load(folders[name, dtype])
    want, streams = P.forward(pcfg, w, t, True)
    model = Model.load(folders[name, dtype], dtype=dtype)
    engine = Engine(model, max_tokens=256, use_graphs=False)
    caught = []
    for b in model.blocks:
        def wrapped(ctx, residual, caches, _o=b.forward):
            _o(ctx, residual, caches)
            caught.append(residual.detach().clone())
        b.forward = wrapped
    got = engine.step([engine.alloc_slot()], [t], [list(range(150))])
    close(got, want, dtype, f"{name} whole prompt")
    assert len(caught) == len(streams)
    for i, (a, b) in enumerate(zip(caught, streams)):
        assert a.dtype == torch.float32, "the residual sum is 32-bit in both run types"
        if dtype == "float32":
            check(a, b, 5e-5, f"stream after layer {i}")
        else:
            close(a, b, dtype, f"stream after layer {i}")
    if dtype == "float32":         # the first tokens of a sequence, one by one
        for i in range(4):
            close(got[i], want[i], dtype, f"{name} token {i}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_token_by_token_against_the_whole(folders, name, dtype):
    """The same 200 tokens: whole; in portions of 2, 3, 64, 1, 65, ... tokens; a prompt of 40 and then one token a
    step for 160 steps (across page borders and windows, the states and the convolutions' inputs handed from step to step).
    All against the plain model; in float32 the three runs agree with one another far below the tolerance."""
    cfg = CONFIGS[name]
    t = toks(cfg, 200, 2)
    want = plain_logits(folders[name, dtype], t)
    model = Model.load(folders[name, dtype], dtype=dtype)
    engine = Engine(model, max_tokens=64 * 12)
    s = engine.alloc_slot()
    whole = engine.step([s], [t], [list(range(200))]).clone()
    close(whole, want, dtype, "whole")
    s2 = engine.alloc_slot()
    rows, at, sizes, i = [], 0, [2, 3, 64, 1, 65, 2, 7], 0
    while at < 200:
        n = min(sizes[i % len(sizes)], 200 - at)
        rows.append(engine.step([s2], [t[at:at + n]], [list(range(n))]).clone())
        at += n
        i += 1
    portions = torch.cat(rows)
    close(portions, want, dtype, "portions")
    engine.free_slot(s)
    s3 = engine.alloc_slot()                 # the slot, pages and state rows that the whole run used
    engine.step([s3], [t[:40]], [[]])
    decoded = torch.cat([engine.step([s3], [[t[i]]]).clone() for i in range(40, 200)])
    close(decoded, want[40:], dtype, "token by token")
    s4 = engine.alloc_slot()                 # portions that want their last place only
    at, last = 0, []
    for n in (5, 2, 33, 2, 100, 58):
        last.append(engine.step([s4], [t[at:at + n]]).clone())
        at += n
    picked = [4, 6, 39, 41, 141, 199]
    if dtype == "float32":
        close(torch.cat(last), want[picked], dtype, "portions that want their last place")
    close(torch.cat(last + [portions]), np.concatenate([want[picked], want]), dtype, "portions, and some for their last place")
    if dtype == "float32":
        check(portions, whole, 2e-5, "portions against the whole")
        check(decoded, whole[40:], 2e-5, "token by token against the whole")
    engine.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_batch_then_decoding_together_on_reused_slots(folders, name, dtype):
    """Four prompts of 1, 33, 130 and 64 tokens in one step, then one token each per step; the short ones end
    early and give their slots, pages and state rows back; a newcomer takes them while the others go on (its states
    must start at zero although the rows were used)."""
    cfg = CONFIGS[name]
    lens, tails = [1, 33, 130, 64], [3, 10, 24, 24]
    seqs = [toks(cfg, n + k, 10 + i) for i, (n, k) in enumerate(zip(lens, tails))]
    want = [plain_logits(folders[name, dtype], t) for t in seqs]
    model = Model.load(folders[name, dtype], dtype=dtype)
    engine = Engine(model, max_tokens=64 * 8)
    slots = [engine.alloc_slot() for _ in seqs]
    out = engine.step(slots, [t[:n] for t, n in zip(seqs, lens)], [[n - 1] for n in lens])
    rows = [Rows(dtype, f"sequence {b}") for b in range(4)]
    for b in range(4):
        rows[b].add(out[b], want[b][lens[b] - 1], "prompt")
    live = list(range(4))
    newcomer = toks(cfg, 90, 99)
    want_new = plain_logits(folders[name, dtype], newcomer)
    for step in range(24):
        live = [b for b in live if step < tails[b]]
        out = engine.step([slots[b] for b in live], [[seqs[b][lens[b] + step]] for b in live])
        for i, b in enumerate(live):
            rows[b].add(out[i], want[b][lens[b] + step], f"decoded token {step}")
        for b in list(range(4)):
            if step + 1 == tails[b] and b in live and tails[b] < 24:
                engine.free_slot(slots[b])
        if step == 11:                      # both short sequences are gone: their slots and pages are used again
            s = engine.alloc_slot()
            got = engine.step([s], [newcomer], [[0, 1, 63, 64, 89]])
            close(got, want_new[[0, 1, 63, 64, 89]], dtype, "a newcomer on used slots")
            engine.free_slot(s)
    for r in rows:
        r.done()
    engine.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_across_pages_and_windows(folders, dtype):
    """420 decoded tokens after a prompt of 150: pages pass by and are given back (but for those of the kept first keys), the
    windows move over decoded tokens only, and the recurrent states have been rewritten 570 times."""
    cfg = CONFIGS["B"]
    n = 570
    t = toks(cfg, n, 5)
    want = plain_logits(folders["B", dtype], t)
    model = Model.load(folders["B", dtype], dtype=dtype)
    engine = Engine(model, max_tokens=640)
    s = engine.alloc_slot()
    engine.step([s], [t[:150]], [[]])
    rows = Rows(dtype, "long decoding")
    for i in range(150, n):
        out = engine.step([s], [[t[i]]])
        if i % 7 == 0 or i % PAGE in (PAGE - 1, 0, 1) or i > n - 10:
            rows.add(out[0], want[i], f"decoded position {i}")
    rows.done()
    held = {(g.request.window, g.request.keep_first): g.pool.n_held for g in engine.cache.groups}
    assert held[100, 70] == 4 and held[64, 64] == 3 and held[77, 1] == 3, "pages between the kept ones and the window are given back"
    engine.cache.check()


def test_long_prompt_on_the_tensor_core_paths(folders):
    """600 tokens in one step through sizes that the tensor-core kernels take, then ten tokens one by one: bfloat16 and
    float32 against the plain model."""
    cfg = CONFIGS["B"]
    t = toks(cfg, 610, 3)
    rows = list(range(0, 600, 7)) + [63, 64, 76, 77, 78, 99, 100, 101, 127, 128, 129, 255, 256, 511, 512, 599]
    for dtype in ("bfloat16", "float32"):
        want = plain_logits(folders["B", dtype], t)
        model = Model.load(folders["B", dtype], dtype=dtype)
        engine = Engine(model, max_tokens=64 * 11)
        s = engine.alloc_slot()
        close(engine.step([s], [t[:600]], [rows]), want[rows], dtype, f"{dtype}: a prompt of 600 tokens")
        out = torch.cat([engine.step([s], [[t[i]]]).clone() for i in range(600, 610)])
        close(out, want[600:], dtype, f"{dtype}: ten tokens after it")
        model.rt.check_status()


@pytest.mark.parametrize("dim,vdim", [(16, 24), (64, 64)])
@pytest.mark.parametrize("window,keep", [(1, 1), (5, 2), (64, 64), (65, 10), (77, 65)])
def test_keys_just_inside_and_just_outside_a_window(tmp_path, window, keep, dim, vdim):
    """One layer whose attention is so sharp that single keys take most of a row's weight: a key that is wrongly seen or
    missed at the window's edge, or among the kept ones, changes the logits.  As a prompt across page borders, and token by
    token."""
    cfg = {"architecture": "Gekilix", "vocab": 64, "width": 48, "norm": {"eps": 1e-5},
           "layers": [att(2, 1, dim, vdim, 1.0, window, keep, rot(1e4, 8), mlp=moe(2, 1, 64, 64))]}
    for dtype in DTYPES:
        folder = write_folder(tmp_path / dtype, cfg, 3, STORE[dtype], sharpen=3.0)
        pcfg, w = P.load(folder)
        mask = pcfg["layers"][0]["mixer"]["mask"]
        for seed in range(40):               # tokens for which the same model with one key more or less answers otherwise
            t = toks(cfg, 210, seed)
            want, rows = P.forward(pcfg, w, t), set()
            for key, off in (("size", -1), ("size", 1), ("keep_first", -1), ("keep_first", 1)):
                if mask[key] + off < (1 if key == "size" else 0):
                    continue
                mask[key] += off
                change = np.abs(P.forward(pcfg, w, t) - want).max(axis=1)[:200]
                mask[key] -= off
                if change.max() < 0.05 * np.abs(want).max():
                    rows = None
                    break
                rows.add(int(change.argmax()))
            if rows is not None:
                break
        assert rows, "no tokens were found for which the edges show"
        model = Model.load(folder, dtype=dtype)
        engine = Engine(model, max_tokens=512)
        s = engine.alloc_slot()
        picks = sorted(p for p in rows | {0, 1, keep - 1, keep, window - 1, window, window + 1, window + keep, 63, 64, 65, 127, 128,
                                   128 + window, 199} if 0 <= p < 200)
        close(engine.step([s], [t[:200]], [picks]), want[picks], dtype, f"window {window}: a prompt")
        out = torch.cat([engine.step([s], [[t[i]]]).clone() for i in range(200, 210)])
        close(out, want[200:], dtype, f"window {window}: decoded after it")
        s2 = engine.alloc_slot()
        engine.step([s2], [t[:3]], [[]])
        out = torch.cat([engine.step([s2], [[t[i]]]).clone() for i in range(3, 200)])
        close(out, want[3:200], dtype, f"window {window}: decoded from the start")


@pytest.mark.parametrize("dtype", DTYPES)
def test_twenty_requests_decode_together(folders, dtype):
    """More sequences than the few-token products take (20 prompts of 1 to 150 tokens in one step, then 6 decode steps of 20
    tokens through the captured step of 32 rows, 12 of them padding) against each request alone in the plain model."""
    cfg = CONFIGS["B"]
    lens = [1 + (37 * i) % 150 for i in range(20)]
    seqs = [toks(cfg, n + 6, 200 + i) for i, n in enumerate(lens)]
    want = [plain_logits(folders["B", dtype], t) for t in seqs]
    model = Model.load(folders["B", dtype], dtype=dtype)
    engine = Engine(model, max_tokens=64 * 64)
    slots = [engine.alloc_slot() for _ in seqs]
    rows = Rows(dtype, "twenty requests")
    out = engine.step(slots, [t[:n] for t, n in zip(seqs, lens)], [[n - 1] for n in lens])
    for b in range(20):
        rows.add(out[b], want[b][lens[b] - 1], f"prompt {b}")
    for step in range(6):
        out = engine.step(slots, [[seqs[b][lens[b] + step]] for b in range(20)])
        for b in range(20):
            rows.add(out[b], want[b][lens[b] + step], f"request {b} decoded token {step}")
    rows.done()
    engine.cache.check()
    model.rt.check_status()


def test_keys_far_back(tmp_path):
    """Attention without a window beside one that keeps 20 keys, sharp queries and keys, 560 positions: most rows look far back
    and across pages."""
    cfg = {"architecture": "Gekilix", "vocab": 64, "width": 48, "norm": {"eps": 1e-5},
           "layers": [att(2, 1, 16, 16, 1.0, None, 0, rot(1e4, 8, (8.0, 1.0, 4.0, 128))),
                      att(4, 2, 64, 40, 0.4, 30, 20, rot(1e4, 32), mlp=moe(2, 1, 32, 32))]}
    t = toks(cfg, 560, 8)
    for dtype in DTYPES:
        folder = write_folder(tmp_path / dtype, cfg, 3, STORE[dtype], sharpen=3.0 if dtype == "float32" else 1.5)
        want = plain_logits(folder, t)
        model = Model.load(folder, dtype=dtype)
        engine = Engine(model, max_tokens=1280)
        s = engine.alloc_slot()
        picks = [0, 1, 19, 20, 49, 50, 51, 529, 530, 559]
        close(engine.step([s], [t], [picks]), want[picks], dtype, "a prompt with far keys")
        s2 = engine.alloc_slot()
        engine.step([s2], [t[:500]], [[]])
        out = torch.cat([engine.step([s2], [[t[i]]]).clone() for i in range(500, 535)])
        close(out, want[500:535], dtype, "decoded past far keys")


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_through_the_session(folders, name):
    """``Session.generate`` (scheduler, batches, captured decode steps) against greedy decoding of the plain model."""
    cfg = CONFIGS[name]
    folder = folders[name, "float32"]
    pcfg, w = P.load(folder)
    prompts = [toks(cfg, 70, 21), toks(cfg, 3, 22), toks(cfg, 129, 23)]
    want = [P.greedy(pcfg, w, p, 8) for p in prompts]
    model = Model.load(folder, dtype="float32")
    session = Session(model, SessionParams(n_ctx=256, seed=1, max_batch=2))
    res = session.generate(prompts, GenerateParams(8, SamplerParams.greedy()), stop_token_ids=())
    assert [r.tokens for r in res] == want
    # the same in bfloat16: the length of every reply (tokens may part ways by rounding)
    model = Model.load(folders[name, "bfloat16"], dtype="bfloat16")
    session = Session(model, SessionParams(n_ctx=256, seed=1, max_batch=3))
    res = session.generate(prompts, GenerateParams(4, SamplerParams.greedy()), stop_token_ids=())
    assert all(len(r.tokens) == 4 for r in res)


def test_a_32_bit_cache_under_a_bfloat16_run(folders):
    """Pages in 32-bit with the rows of the tensor-core kernels: the 32-bit attention kernel reads them."""
    cfg = CONFIGS["B"]
    t = toks(cfg, 90, 6)
    want = plain_logits(folders["B", "bfloat16"], t)
    model = Model.load(folders["B", "bfloat16"])
    engine = Engine(model, max_tokens=256, kv_dtype=torch.float32)
    s = engine.alloc_slot()
    got = torch.cat([engine.step([s], [t[:80]], [list(range(80))]).clone()] + [engine.step([s], [[x]]).clone() for x in t[80:]])
    close(got, want, "bfloat16", "32-bit cache")


def test_command_line_random_weights_info_and_generation(tmp_path):
    """The command line's modes on this design: a folder with random weights from a configuration file, its --info,
    the greedy token harness against the plain model, and a sampled continuation."""
    import io
    from nncpu_b200.cli import parse_options, run_gen, run_generate, run_info, run_random_weights

    def run(fn, argv):
        out = io.StringIO()
        assert fn(parse_options(argv), out) == 0
        return out.getvalue()

    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(CONFIGS["A"]))
    run(run_random_weights, ["--random-weights", str(cfg), "5", str(tmp_path / "m"), "--fp32"])
    info = json.loads(run(run_info, ["--info", str(tmp_path / "m")]))
    assert info["config"]["architecture"] == "Gekilix" and info["parameters"] > 0
    prompt = toks(CONFIGS["A"], 40, 3)
    got = [int(t) for t in run(run_gen, ["--gen", str(tmp_path / "m"), " ".join(map(str, prompt)), "6", "--fp32"]).splitlines()[0].split()]
    pcfg, w = P.load(tmp_path / "m")
    assert got == P.greedy(pcfg, w, prompt, 6)
    out = run(run_generate, ["-m", str(tmp_path / "m"), "--tokens", " ".join(map(str, prompt)), "-n", "6", "--temp", "0.8",
                             "--top-k", "20", "-s", "4", "-b", "3"]).split()
    assert len(out) >= 6 and all(0 <= int(t) < CONFIGS["A"]["vocab"] for t in out[:6])


def test_trace_replay_of_many_short_requests(folders, tmp_path):
    """``bin/trace_run`` as a subprocess on this design: eight requests of unequal lengths in one batch, decoded
    together while the shorter ones end; then a second batch on the slots, pages and state rows that were given back."""
    import subprocess
    import sys
    from conftest import ROOT
    cfg = CONFIGS["A"]
    folder = folders["A", "float32"]
    V = cfg["vocab"]
    lens, tails = [3, 5, 70, 1, 9, 64, 2, 31], [2, 6, 6, 1, 4, 6, 3, 6]
    seqs = {f"r{i}": toks(cfg, n + k, 50 + i) for i, (n, k) in enumerate(zip(lens, tails))}
    seqs.update({f"s{i}": toks(cfg, n, 70 + i) for i, n in enumerate((66, 4, 17))})
    want = {k: plain_logits(folder, t) for k, t in seqs.items()}
    steps, expect = [], {}

    def add(entries, end=()):
        n = len(steps)
        steps.append({"step": n, "entries": [{"id": k, "tokens": seqs[k][a:b], "want": w} for k, a, b, w in entries], "end": list(end)})
        if any(w for *_, w in entries):
            expect[n] = [(k, [a + i for i in w]) for k, a, b, w in entries if w]

    add([(f"r{i}", 0, n, [0, n - 1] if n > 1 else [0]) for i, n in enumerate(lens)])
    for step in range(max(tails)):
        live = [i for i in range(len(lens)) if step < tails[i]]
        add([(f"r{i}", lens[i] + step, lens[i] + step + 1, [0]) for i in live],
            end=[f"r{i}" for i in live if step + 1 == tails[i]])
    add([(f"s{i}", 0, len(seqs[f"s{i}"]), [0, len(seqs[f"s{i}"]) - 1]) for i in range(3)], end=[f"s{i}" for i in range(3)])
    out = tmp_path / "out"
    text = "".join(json.dumps(s) + "\n" for s in steps)
    p = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32",
                        "--out", str(out), "--max-tokens", str(sum(lens) + sum(tails))], input=text, capture_output=True,
                       text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    for n, rows in expect.items():
        got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, V)
        ref = np.concatenate([want[k][pos] for k, pos in rows])
        check(got, ref, 1e-4, f"step {n}")


def random_gekilix(rs):
    """A random configuration: any order of the two kinds of layer, head sizes in and out of what the tensor-core
    kernels take, any grouping of heads, windows short and long, kept keys in and beyond a page, groups of every kind."""
    width = int(rs.choice([72, 100, 136, 200, 256]))
    layers = []
    for i in range(int(rs.randint(2, 6))):
        mlp = None
        if rs.rand() < 0.85:
            E = int(rs.choice([1, 2, 4, 6, 8, 12]))
            mlp = moe(E, int(rs.randint(1, E + 1)), int(rs.choice([16, 20, 64, 80])),
                      int(rs.choice([16, 24, 36, 64])) if rs.rand() < 0.8 else None)
        if rs.rand() < 0.5:
            kv, group, dim = int(rs.choice([1, 2, 3])), int(rs.choice([1, 2, 4, 8])), int(rs.choice([16, 24, 64, 80, 128]))
            vdim = int(rs.choice([dim, 8, 41, 128]))
            window = None if rs.rand() < 0.15 else int(rs.choice([1, 3, 17, 64, 77, 100, 130]))
            scaling = (float(rs.choice([2.0, 8.0])), 1.0, float(rs.choice([1.0, 4.0])), int(rs.choice([16, 100, 2048]))) if rs.rand() < 0.7 else None
            layers.append(att(kv * group, kv, dim, vdim, float(rs.choice([dim ** -0.5, 0.2])), window,
                              int(rs.choice([0, 1, 5, 64, 70, 130])) if window else 0,
                              rot(float(rs.choice([1e4, 4e5, 300.0])), int(rs.choice([dim, dim // 2, 2])), scaling) if rs.rand() < 0.9 else None,
                              mlp=mlp))
        else:
            G, per, vdim = int(rs.choice([1, 2, 3])), int(rs.choice([1, 2, 3])), int(rs.choice([8, 20, 64, 72]))
            inner = G * per * vdim
            layers.append(ssm(G * per, vdim, int(rs.choice([8, 20, 64, 128, 130])), G, int(rs.choice([1, 2, 4, 5])),
                              int(rs.choice([k for k in (1, 2, 3, 4, 6) if inner % k == 0])), mlp=mlp))
    return {"architecture": "Gekilix", "vocab": int(rs.randint(100, 600)), "width": width,
            "norm": {"eps": float(rs.choice([1e-6, 1e-5]))}, "layers": layers}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", range(10))
def test_random_configuration_and_trace(tmp_path, seed, dtype):
    """Random configurations, each with a batch of unequal prompts (the first one cut in two steps the second time
    round), decoding with early leavers, then the same again on the slots, pages and state rows given back."""
    rs = np.random.RandomState(8000 + seed)
    cfg = random_gekilix(rs)
    folder = write_folder(tmp_path / "m", cfg, seed, STORE[dtype])
    model = Model.load(folder, dtype=dtype)
    lens = [int(rs.choice([1, 2, 17, 40, 65, 130, 260])) for _ in range(int(rs.choice([1, 2, 3, 4])))]
    if rs.rand() < 0.4:
        lens[0] = int(rs.choice([300, 520]))
    n_decode = [int(rs.randint(0, 10)) for _ in lens]
    reqs = [rs.randint(0, cfg["vocab"], size=n + d).tolist() for n, d in zip(lens, n_decode)]
    want = [plain_logits(folder, r) for r in reqs]
    engine = Engine(model, max_tokens=64 * (sum((len(r) + 63) // 64 for r in reqs) + 2))
    for round_ in range(2):
        slots = [engine.alloc_slot() for _ in reqs]
        shared = Rows(dtype, f"seed {seed} round {round_}")     # bfloat16 rows of a round are judged together
        rows = [shared for _ in reqs]
        cut = lens[0] // 2 if lens[0] > 40 and round_ == 1 else 0
        if cut:
            engine.step(slots[:1], [reqs[0][:cut]], [[]])
        out = engine.step(slots, [r[(cut if b == 0 else 0):n] for b, (r, n) in enumerate(zip(reqs, lens))],
                          [[n - 1 - (cut if b == 0 else 0)] for b, n in enumerate(lens)])
        for b in range(len(reqs)):
            rows[b].add(out[b], want[b][lens[b] - 1], "prompt")
        for step in range(max(n_decode)):
            live = [b for b in range(len(reqs)) if step < n_decode[b]]
            out = engine.step([slots[b] for b in live], [[reqs[b][lens[b] + step]] for b in live])
            for i, b in enumerate(live):
                rows[b].add(out[i], want[b][lens[b] + step], f"decoded token {step}")
            for b in live:
                if step + 1 == n_decode[b]:
                    engine.free_slot(slots[b])
        for b in range(len(reqs)):
            if n_decode[b] == 0:
                engine.free_slot(slots[b])
        shared.done()
    engine.cache.check()
    model.rt.check_status()
