"""The Vuvalorn design against its plain statement (``plain_vuvalorn``): every mechanism alone, then the model through
``Engine.step`` cut in every way (whole prompts, token by token, portions down to one and two tokens, unequal batches, slots,
pages and state rows used again), and greedy generation through ``Session.generate``, the command line and the trace
replay.  Configurations and weights are made here; where random weights would hide a fault (a key far back, the first
tokens of a sequence, a cap that never binds, a correction that never decides) the weights or inputs are made so that it
shows."""
import json

import numpy as np
import pytest
import torch

import plain_vuvalorn as P
from gpu_util import DEV, TOL, check
from nncpu_b200 import Engine, GenerateParams, Model, SamplerParams, Session, SessionParams
from nncpu_b200.cache import PAGE
from nncpu_b200.config import config_from_dict
from nncpu_b200.config.specs import NormSpec
from nncpu_b200.engine.model import parameter_list
from nncpu_b200.kernels import ops
from nncpu_b200.parts import Runtime, build
from nncpu_b200.parts.base import SublayerClosing
from nncpu_b200.weights import random_tensors, write_safetensors

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
STORE = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, identity, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}


def rot(base, dims):
    return {"base": base, "dims": dims}


def att(heads, kv, dim, conv, scale, cap=None, r=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "conv": conv, "scale": scale, "softcap": cap, "rot": r}
    return {"type": "attention", "mixer": m, "mlp": mlp}


CONFIGS = {
    # odd sizes everywhere and a width that is no multiple of 8 (no tensor-core product takes it); a loop that begins with
    # the first layer; taps of 2, 4 and 5; more identity experts than experts; a layer without a feed-forward
    "A": {"architecture": "Vuvalorn", "vocab": 211, "width": 76, "norm": {"eps": 3e-6}, "embedding": {"scale": 6.5},
          "logit_scale": 0.3, "loop": {"start": 0, "stop": 2, "times": 3},
          "layers": [att(6, 2, 24, 4, 0.3, 7.0, rot(1e4, 16), dense(20, 0.7)),
                     att(4, 4, 15, 2, 0.25, 30.0, rot(300.0, 6), moe(5, 6, 3, 12)),
                     att(3, 1, 10, 5, 0.4, 11.0, rot(2e3, 10), None),
                     att(2, 2, 16, 3, 0.3, 5.0, rot(5e5, 2), dense(36, 3.0))]},
    # sizes the tensor-core paths take: heads that fill rows of 64 and of 128 lanes and heads that do not, taps from 2 to 7,
    # a loop in the middle, experts in both forms (few tokens, grouped).  Only the last layer's experts are a choice, all
    # other routers give everything: a choice that bfloat16 rounding turns round then stays with its own token
    "B": {"architecture": "Vuvalorn", "vocab": 640, "width": 256, "norm": {"eps": 1e-5}, "embedding": {"scale": 11.0},
          "logit_scale": 0.25, "loop": {"start": 1, "stop": 3, "times": 2},
          "layers": [att(8, 2, 128, 4, 0.09, 15.0, rot(1e6, 128), moe(3, 1, 4, 64)),
                     att(8, 4, 64, 3, 0.125, 25.0, rot(1e4, 48), dense(128, 2.5)),
                     att(6, 3, 96, 2, 0.1, 9.0, rot(4e5, 64), moe(4, 2, 6, 136)),
                     att(4, 2, 128, 3, 0.08, 50.0, rot(1e5, 16), None),
                     att(4, 1, 48, 7, 0.14, 40.0, rot(1e4, 32), moe(12, 4, 3, 64))]},
    # values at the edges: one tap, nine taps, more query heads on a key/value head than one block serves, a head of one
    # pair, heads of 144 lanes, no cap, a cap too large for the fast form, no rotation, one expert, no identity experts, one
    # pass, a loop that ends with the last layer, no scales
    "C": {"architecture": "Vuvalorn", "vocab": 97, "width": 104, "norm": {"eps": 1e-5}, "loop": {"start": 2, "stop": 4, "times": 1},
          "layers": [att(34, 1, 64, 1, 0.15, 12.0, rot(100.0, 2), moe(1, 1, 1, 8)),
                     att(3, 3, 2, 9, 0.5, None, rot(100.0, 2), moe(4, 0, 4, 12)),
                     att(2, 1, 144, 4, 0.1, 20.0, rot(1e4, 144), dense(24, 0.4)),
                     att(4, 2, 64, 2, 0.1, 5000.0, None, moe(3, 5, 4, 8))]},
}


def write_folder(path, cfg_dict, seed, store, sharpen=None):
    """A model folder with random weights, scaled so that every part of a layer moves the stream: the query and key norms'
    weights are scaled up so that attention is not close to uniform and a wrong key changes the logits (less so for a
    bfloat16 run, whose rounding a sharp softmax and the choice of experts make larger in every layer); the routers' scores are
    of the size of the corrections, so that those decide about many choices."""
    sharpen = sharpen or (4.0 if store == torch.float32 else 2.0)
    config = config_from_dict(cfg_dict)
    tensors = random_tensors(parameter_list(config.model_spec()), seed, store)
    for name in list(tensors):
        t = tensors[name].float()
        if name.endswith((".q.norm", ".k.norm")):
            t = t * sharpen ** 0.5
        elif name.endswith(".router"):
            t = t * 4.0 / t.shape[1] ** 0.5
        elif name.endswith(".correction"):
            t = t * 2.5
        elif name.endswith(".mix.g"):
            t = t * 10.0
        elif t.dim() == 2 and not name.endswith((".conv", "loop.step")):
            t = t * 3.0
        tensors[name] = t.to(store)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(config.to_dict()))
    write_safetensors(path / "model.safetensors", tensors, {"format": "pt"})
    return path


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("vuvalorn")
    return {(name, dtype): write_folder(root / f"{name}_{dtype}", cfg, 41 + i, STORE[dtype])
            for i, (name, cfg) in enumerate(CONFIGS.items()) for dtype in DTYPES}


def toks(cfg, n, seed):
    return np.random.RandomState(seed).randint(0, cfg["vocab"], size=n).tolist()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def f32(x):
    return torch.tensor(np.asarray(x), dtype=torch.float32, device=DEV)


# -- attention alone ------------------------------------------------------------------------------

def pages_of(lens, n_kv, hd, row, seed):
    """Random keys and values in shuffled bfloat16 pages whose rows are longer than the heads (zeros behind)."""
    g = torch.Generator().manual_seed(seed)
    n_pages = sum((n + PAGE - 1) // PAGE for n in lens) + 2
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((len(lens), max((n + PAGE - 1) // PAGE for n in lens)), -1, dtype=torch.int32)
    kp, vp = (torch.zeros(n_pages, n_kv, PAGE, row, dtype=torch.bfloat16) for _ in range(2))
    ks, vs = [], []
    for b, n in enumerate(lens):
        k, v = (torch.randn(n, n_kv, hd, generator=g).bfloat16() for _ in range(2))
        for p in range((n + PAGE - 1) // PAGE):
            page = table[b, p] = order.pop()
            a, z = p * PAGE, min(n, (p + 1) * PAGE)
            kp[page, :, :z - a, :hd] = k[a:z].transpose(0, 1)
            vp[page, :, :z - a, :hd] = v[a:z].transpose(0, 1)
        ks.append(k.double().numpy())
        vs.append(v.double().numpy())
    return kp.to(DEV), vp.to(DEV), table.to(DEV), ks, vs


def plain_rows(q, k, v, positions, scale, cap, gate=None):
    """Attention of queries at the given positions over keys 0 .. position; gate [n, heads] logits or None."""
    group = q.shape[1] // k.shape[1]
    out = np.zeros((len(positions), q.shape[1], v.shape[2]))
    for i, p in enumerate(positions):
        for h in range(q.shape[1]):
            s = P.capped((k[:p + 1, h // group] @ q[i, h]) * scale, cap)
            out[i, h] = P.softmax(s) @ v[:p + 1, h // group]
    return out if gate is None else out * P.sigmoid(gate)[:, :, None]


@pytest.mark.parametrize("nh,nkv,hd,scale,cap", [(4, 2, 64, 0.3, 6.0), (8, 2, 128, 0.2, 20.0), (2, 2, 40, 1.0, 3.0), (6, 2, 96, 0.02, 50.0),
                                                 (34, 1, 64, 0.4, 11.0), (16, 1, 128, 0.1, 0.5), (3, 1, 112, 0.3, 0.0), (5, 5, 24, 2.0, 1000.0)])
def test_capped_scores_and_gates_per_head_in_every_kernel(nh, nkv, hd, scale, cap):
    """The 32-bit kernel and the three bfloat16 kernels: a portion of 9 tokens, a whole prompt of 67, a portion of 130, then
    one token each with the keys in one split, in several that a cluster merges, and in several through scratch."""
    lens, new = [150, 67, 420], [9, 67, 130]
    row = ops.attention_rows(hd, hd)[0]
    g = torch.Generator().manual_seed(nh + hd)
    kp, vp, table, ks, vs = pages_of(lens, nkv, hd, row, 3)
    q = [torch.randn(n, nh, hd, generator=g).bfloat16() for n in new]
    n = sum(new)
    logits = torch.randn(n, nh + 5, generator=g) * 2
    qp = torch.zeros(n, nh, row, dtype=torch.bfloat16)
    qp[:, :, :hd] = torch.cat(q)
    qp = qp.view(n, -1).to(DEV)
    cu = i32(np.cumsum([0] + new).tolist())
    tok_pos = i32([p for b in range(3) for p in range(lens[b] - new[b], lens[b])])
    tok_seq = i32([b for b in range(3) for _ in range(new[b])])
    want = np.concatenate([plain_rows(q[b].double().numpy(), ks[b], vs[b], range(lens[b] - new[b], lens[b]), scale, cap)
                           for b in range(3)])
    gated = (want * P.sigmoid(logits[:, 5:].double().numpy())[:, :, None]).reshape(n, -1)
    want = want.reshape(n, -1)
    if 0.0 < cap < 6.0 * scale * hd ** 0.5:        # the cap binds
        free = plain_rows(q[1].double().numpy(), ks[1], vs[1], range(67), scale, 0.0).reshape(67, -1)
        assert np.abs(free - want[9:76]).max() > 0.03 * np.abs(want).max()
    logits = logits.to(DEV)
    last = [int(cu[b + 1]) - 1 for b in range(3)]
    for gate, ref in ((None, want), ((logits, 5), gated)):
        kw = {"v_lanes": hd, "cap": cap, "head_gate": gate}
        out = torch.full((n, nh * hd), float("nan"), dtype=torch.float32, device=DEV)
        ops.attention(qp.float(), kp.float(), vp.float(), table, tok_seq, tok_pos, out, nh, nkv, row, scale, 0, row, **kw)
        check(out, ref, 2e-5, "32-bit kernel")
        out = torch.full((n, nh * hd), float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.attention_prefill_mma(qp, kp, vp, table, cu, tok_pos, out, 3, nh, nkv, row, scale, 0, **kw)
        check(out, ref, 2e-2, "portion kernel")
        out = torch.full((n, nh * hd), float("nan"), dtype=torch.bfloat16, device=DEV)
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        ops.attention_prefill_tc(qp, kp, vp, table, cu, tok_pos, out, status, 3, nh, nkv, row, scale, 0, **kw)
        assert int(status.item()) == 0
        check(out, ref, 2e-2, "tcgen05 prompt kernel")
        if gate is not None:
            kw["head_gate"] = (logits[last].contiguous(), 5)
        for n_splits, scratched in ((1, False), (2, False), (5, False), (3, True)):
            scratch = torch.empty(ops.attention_decode_scratch_floats(3, nh, nkv, row, n_splits), device=DEV) if scratched else None
            got = torch.full((3, nh * hd), float("nan"), dtype=torch.bfloat16, device=DEV)
            ops.attention_decode_mma(qp[last].contiguous(), kp, vp, table, i32([0, 1, 2]), i32([l - 1 for l in lens]), got, scratch,
                                     nh, nkv, row, scale, 0, n_splits, **kw)
            check(got, ref[last], 2e-2, f"decode, {n_splits} splits")


def test_scores_far_beyond_their_cap():
    """Scores of thousands in both directions: every key with a large positive one weighs the same, and nothing overflows."""
    hd = 64
    kp, vp, table, ks, vs = pages_of([200], 1, hd, hd, 4)
    q = torch.sign(torch.tensor(ks[0][7, 0])).bfloat16().view(1, 1, hd) * 100
    for cap in (2.0, 60.0):
        want = plain_rows(q.double().numpy(), ks[0], vs[0], [199], 1.0, cap).reshape(1, -1)
        qd, args = q.view(1, -1).to(DEV), (table, i32([0]), i32([199]))
        out = torch.empty(1, hd, dtype=torch.float32, device=DEV)
        ops.attention(qd.float(), kp.float(), vp.float(), *args, out, 1, 1, hd, 1.0, 0, cap=cap)
        check(out, want, 1e-4, "32-bit")
        out = torch.empty(1, hd, dtype=torch.bfloat16, device=DEV)
        ops.attention_decode_mma(qd, kp, vp, *args, out, None, 1, 1, hd, 1.0, 0, 2, cap=cap)
        check(out, want, 2e-2, "decode")
        ops.attention_prefill_mma(qd, kp, vp, table, i32([0, 1]), args[2], out, 1, 1, 1, hd, 1.0, 0, cap=cap)
        check(out, want, 2e-2, "portion")
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        ops.attention_prefill_tc(qd, kp, vp, table, i32([0, 1]), args[2], out, status, 1, 1, 1, hd, 1.0, 0, cap=cap)
        check(out, want, 2e-2, "prompt")


class Projected:
    """The short convolutions, norms, rotation and append of one layer, driven by hand: a cache of pages in order, state rows,
    and the plain statement of whole sequences beside it."""

    def __init__(self, nh, nkv, hd, taps, dims, dtype, seed, n_slots=3):
        g = np.random.RandomState(seed)
        self.nh, self.nkv, self.hd, self.taps, self.dims, self.dtype = nh, nkv, hd, taps, dims, dtype
        self.C = (nh + nkv) * hd
        self.w = g.randn(self.C, taps) * 0.5
        self.qg, self.kg = g.randn(hd) * 0.3 + 1.0, g.randn(hd) * 0.3 + 1.0
        self.row = hd if dtype == torch.float32 else ops.attention_rows(hd, hd)[0]
        self.width = 5                                  # pages a sequence may have
        shape = (n_slots * self.width + 1, nkv, PAGE, self.row)
        self.kp, self.vp = (torch.full(shape, 9.0, dtype=dtype, device=DEV) for _ in range(2))
        self.state = torch.full((n_slots + 1, ops.conv_state_floats(taps, self.C)), 7.0, device=DEV)
        self.wd = f32(self.w.T.copy())

    def table(self, slots):
        return i32([[max(s, 0) * self.width + j for j in range(self.width)] for s in slots])

    def cos_sin(self, pos):
        if not self.dims:
            return None
        f = 300.0 ** (-np.arange(0, self.dims, 2) / self.dims)
        a = np.outer(pos, f)
        return f32(np.stack([np.cos(a), np.sin(a)], axis=-1))

    def run(self, parts):
        """[(slot, start, rows [n, ld])] -> the queries [n, heads, row]; a negative slot is a padding sequence."""
        proj = f32(np.concatenate([rows for *_, rows in parts]))
        pos = [st + j for _, st, rows in parts for j in range(len(rows))]
        seq = i32([i if s >= 0 else -1 for i, (s, _, rows) in enumerate(parts) for _ in rows])
        cu = i32(np.cumsum([0] + [len(rows) for *_, rows in parts]).tolist())
        for s, st, _ in parts:
            if st == 0 and s >= 0:
                self.state[s].zero_()
        q = torch.full((len(pos), self.nh * self.row), float("nan"), dtype=self.dtype, device=DEV)
        ops.qk_conv_norm_append(proj, self.wd, self.state, i32([s for s, *_ in parts]), cu, f32(self.qg), f32(self.kg), 1e-5,
                                self.cos_sin(pos), seq, i32(pos), self.table([s for s, *_ in parts]), self.kp, self.vp, q, self.nh,
                                self.nkv, self.hd)
        return q.view(len(pos), self.nh, self.row)

    def plain(self, rows):
        """(queries, keys, values) [T, heads, hd] of a whole sequence."""
        y = P.short_conv(rows[:, :self.C], self.w).reshape(len(rows), -1, self.hd)
        q, v = y[:, :self.nh], y[:, self.nh:]
        q, k = P.norm(q, self.qg, 1e-5), P.norm(v, self.kg, 1e-5)
        if self.dims:
            q, k = (P.rotate_pairs(z, np.arange(len(rows)), rot(300.0, self.dims)) for z in (q, k))
        return q, k, v

    def kept(self, slot, n):
        """Keys and values [n, kv heads, row] of a slot's first n positions."""
        a = slot * self.width
        return tuple(p[a:a + self.width].transpose(1, 2).reshape(-1, self.nkv, self.row)[:n] for p in (self.kp, self.vp))


CONV_SIZES = [(4, 2, 64, 3, 32), (6, 2, 24, 4, 16), (8, 2, 128, 4, 128), (3, 1, 7, 2, 2), (2, 2, 144, 3, 10), (5, 5, 96, 5, 0), (2, 1, 64, 1, 64),
              (2, 1, 10, 9, 6), (4, 4, 128, 2, 40), (3, 1, 42, 3, 2)]


@pytest.mark.parametrize("nh,nkv,hd,taps,dims", CONV_SIZES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_convolution_norm_rotation_and_append(nh, nkv, hd, taps, dims, dtype):
    """Whole; then in portions of 1, 2, 3, ... tokens (shorter than the taps among them) beside another sequence that goes on and
    a padding sequence: the same bits.  The value is the key before norm and rotation."""
    if dtype == torch.bfloat16 and ops.attention_rows(hd, hd) is None:
        return
    m = Projected(nh, nkv, hd, taps, dims, dtype, hd + taps)
    g = np.random.RandomState(hd)
    tol = 1e-5 if dtype == torch.float32 else 8e-3
    seqs = [g.randn(150, m.C + 3), g.randn(90, m.C + 3)]
    want = [m.plain(s) for s in seqs]
    whole = m.run([(0, 0, seqs[0])]).clone()
    check(whole[..., :hd], want[0][0], tol, "queries")
    keys, values = (t.clone() for t in m.kept(0, 150))
    check(keys[..., :hd], want[0][1], tol, "keys")
    check(values[..., :hd], want[0][2], tol, "values")
    for t in (whole, keys, values):
        assert t.shape[-1] == hd or float(t[..., hd:].float().abs().max()) == 0.0, "zeros behind a head"
    pad, rows, at = g.randn(3, m.C + 3), [], 0
    for i, k in enumerate((1, 2, 1, 3, 2, 64, 8, 1, 68)):
        other = [(2, 0, seqs[1][:41])] if i == 0 else [(2, 41, seqs[1][41:43])] if i == 2 else [(2, 43, seqs[1][43:])] if i == 4 else []
        q = m.run([(1, at, seqs[0][at:at + k]), (-1, 0, pad)] + other)
        rows.append(q[:k].clone())
        at += k
    assert torch.equal(torch.cat(rows), whole), "portions beside others are not the same bits"
    assert all(torch.equal(a, b) for a, b in zip(m.kept(1, 150), (keys, values)))
    k2, v2 = m.kept(2, 90)
    check(k2[..., :hd], want[1][1], tol, "keys of the other sequence")
    check(v2[..., :hd], want[1][2], tol, "values of the other sequence")
    assert float(m.kp[-1].float().min()) == 9.0, "a page of nobody was written"
    assert float(m.state[-1].min()) == 7.0, "a state row of nobody was written"
    if taps > 1:        # one input less or more shows
        short = P.short_conv(seqs[0][:, :m.C], np.concatenate([np.zeros((m.C, 1)), m.w[:, 1:]], axis=1))
        assert np.abs(short[:, nh * hd:].reshape(150, nkv, hd) - want[0][2]).max() > 0.05


@pytest.mark.parametrize("nh,nkv,hd,taps,dims", [s for s in CONV_SIZES if s[2] <= 128])
def test_a_decode_step_from_the_projections(nh, nkv, hd, taps, dims):
    """Three sequences of 1, 65 and 200 tokens, then ten steps of one token each through the attention kernel that starts from
    the projections (in one split, in a cluster of three, through scratch): outputs, appended keys and values, and the state,
    which the append kernel must be able to go on from."""
    cap, scale = 9.0, 0.3
    m = Projected(nh, nkv, hd, taps, dims, torch.bfloat16, hd * taps)
    other = Projected(nh, nkv, hd, taps, dims, torch.bfloat16, hd * taps)
    g = np.random.RandomState(taps)
    lens = [1, 65, 200]
    seqs = [g.randn(n + 12, m.C + nh) for n in lens]
    full = [m.plain(s) for s in seqs]
    for x in (m, other):
        x.run([(b, 0, seqs[b][:n]) for b, n in enumerate(lens)])
    for step in range(10):
        pos = [n + step for n in lens]
        qkv = f32(np.stack([seqs[b][p] for b, p in enumerate(pos)]))
        n_splits, scratched = ((1, False), (3, False), (4, True))[step % 3]
        scratch = torch.empty(ops.attention_decode_scratch_floats(3, nh, nkv, m.row, n_splits), device=DEV) if scratched else None
        got = torch.full((3, nh * hd), float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.attention_decode_mma_from_qkv(qkv, f32(m.qg), f32(m.kg), 1e-5, m.cos_sin(pos), m.kp, m.vp, True, m.table([0, 1, 2]),
                                          i32([0, 1, 2]), i32(pos), got, scratch, nh, nkv, hd, scale, 0, n_splits,
                                          values_are_keys=True, v_head_dim=hd, rot_pairs=True, cap=cap, head_gated=True,
                                          conv=(m.wd, m.state, i32([0, 1, 2])))
        want = []
        for b, p in enumerate(pos):
            q, k, v = full[b]
            k, v = (torch.tensor(z[:p + 1]).bfloat16().double().numpy() for z in (k, v))
            q = torch.tensor(q[p:p + 1]).bfloat16().double().numpy()
            want.append(plain_rows(q, k, v, [p], scale, cap, seqs[b][p:p + 1, m.C:]).reshape(-1))
        check(got, np.stack(want), 2.5e-2, f"step {step}, {n_splits} splits")
        other.run([(b, p, seqs[b][p:p + 1]) for b, p in enumerate(pos)])
    for b, n in enumerate(lens):
        for a, z, what in zip(m.kept(b, n + 10), other.kept(b, n + 10), ("keys", "values")):
            check(a, z, 8e-3, f"{what} of sequence {b} against the append kernel's")
    q = [x.run([(b, n + 10, seqs[b][n + 10:n + 12]) for b, n in enumerate(lens)]) for x in (m, other)]
    assert torch.equal(q[0], q[1]), "the states the steps left differ from the append kernel's"


def test_a_step_that_is_done_over_finds_the_same_inputs():
    """A step reads one copy of the kept inputs and leaves the other: done again from the same position it gives the same."""
    m = Projected(2, 1, 64, 4, 32, torch.bfloat16, 5)
    g = np.random.RandomState(1)
    s = g.randn(40, m.C)
    m.run([(0, 0, s[:20])])
    first = m.run([(0, 20, s[20:23])]).clone()
    assert torch.equal(m.run([(0, 20, s[20:23])]), first)
    m.run([(0, 20, s[20:30])])                      # longer this time
    rest = m.run([(0, 30, s[30:])])
    check(rest[..., :64], m.plain(s)[0][30:], 8e-3, "what follows")


# -- the feed-forward alone -----------------------------------------------------------------------

@pytest.mark.parametrize("n_outputs,top,corrected", [(5, 2, True), (12, 3, True), (4, 4, True), (1, 1, True), (70, 6, True), (300, 1, True),
                                                     (9, 3, False)])
def test_router_with_corrected_choice_and_plain_scores(n_outputs, top, corrected):
    g = torch.Generator().manual_seed(n_outputs)
    n, width = 37, 72
    z = torch.randn(n, n_outputs, generator=g) * 2
    corr = torch.randn(n_outputs, generator=g) * 0.4 if corrected else None
    plain = corr.double().numpy() if corrected else np.zeros(n_outputs)
    for one_launch in (False, True):
        ids, ws = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
        scoring = ("plain", corr.to(DEV) if corrected else None, 1.0)
        if one_launch:
            x, w = torch.randn(n, width, generator=g), torch.randn(n_outputs, width, generator=g) * 0.2
            s = P.softmax(x.double().numpy() @ w.double().numpy().T)
            ops.moe_router(x.to(DEV), w.to(DEV), None, top, ids, ws, scoring)
        else:
            s = P.softmax(z.double().numpy())
            ops.moe_route(z.to(DEV), top, ids, ws, scoring)
        chosen = [P.route(s[t], plain, top) for t in range(n)]
        assert ids.cpu().numpy().tolist() == [c.tolist() for c, _ in chosen]
        check(ws, np.stack([v for _, v in chosen]), 1e-5, "weights: the scores without correction, not renormalised")
        if corrected and n_outputs > 4:
            assert any(c.tolist() != np.argsort(-s[t], kind="stable")[:top].tolist() for t, (c, _) in enumerate(chosen)), \
                "the correction decides nowhere"


class Ctx:
    branch_is_fresh, out_scale, next_norm, n_tokens, closing = False, 1.0, None, 0, None

    def __init__(self):
        self.memo = {}


def ff_part(rt, width, f, seed, store):
    """The framework's part with random weights, and the same weights for the plain statement."""
    cfg = {"architecture": "Vuvalorn", "vocab": 8, "width": width, "norm": {"eps": 1e-5}, "layers": [att(1, 1, 8, 1, 1.0, mlp=f)]}
    part = build("feed_forward", config_from_dict(cfg).model_spec().layers[0].feed_forward)
    tensors = random_tensors(part.params(), seed, store)
    scale = {"router": 4.0 / width ** 0.5, "correction": 2.0}
    tensors = {k: (v.float() * scale.get(k.split(".")[-1], 4.0)).to(store) for k, v in tensors.items()}
    plain = {k: v.double().numpy() for k, v in tensors.items()}
    part.bind({k: v.to(DEV) for k, v in tensors.items()}, rt)
    return part, plain


def clear_rows(x, f, w):
    """The tokens whose choice is not close: the last chosen and the first not chosen lie apart."""
    return P.margins(P.softmax(x @ w["l0.mlp.router"].T), w["l0.mlp.correction"], f["router"]["top"]) > 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 3, 9, 70, 300])
@pytest.mark.parametrize("width,f", [(256, moe(8, 3, 2, 64)), (88, moe(5, 6, 1, 40)), (100, moe(6, 2, 3, 20)), (128, moe(4, 0, 2, 64)),
                                     (136, moe(8, 8, 16, 72)), (136, moe(1, 9, 4, 9))])
def test_experts_some_of_which_hand_the_input_on(dtype, n, width, f):
    """Few tokens (a block per slot) and many (sorted, grouped products): added into a stream, written into a branch of its own,
    and closed with the sublayer's norm and the one that follows."""
    rt = Runtime(DEV, STORE[dtype])
    part, w = ff_part(rt, width, f, n + width, STORE[dtype])
    g = torch.Generator().manual_seed(n)
    x = torch.randn(n, width, generator=g).to(STORE[dtype])
    xn = x.double().numpy()
    rows = clear_rows(xn, f, w)
    want = P.routed_experts(xn, f, w, "l0.mlp")[rows]
    tol = 3e-5 if dtype == "float32" else 3e-2
    before = torch.randn(n, width, generator=g)
    out = before.clone().to(DEV)
    part.forward(Ctx(), x.to(DEV), out)
    check(out.cpu()[rows], before.double().numpy()[rows] + want, tol, "added into the stream")
    ctx = Ctx()
    ctx.branch_is_fresh = True
    branch = torch.full((n, width), float("nan"), device=DEV)
    part.forward(ctx, x.to(DEV), branch)
    check(branch.cpu()[rows], want, tol, "a branch of its own")
    if f["router"]["identity"] and n > 8:
        gone = P.routed_experts(xn, {**f, "router": {**f["router"], "experts": 99}}, {**w, **{f"l0.mlp.e{e}.{k}": w[f"l0.mlp.e0.{k}"] * 0
                                for e in range(f["router"]["experts"], 20) for k in ("gate", "up", "down")}}, "l0.mlp")[rows]
        assert np.abs(gone - want).max() > 0.05 * np.abs(want).max(), "the identity experts do not show"
    norms = []
    for name in ("post", "then"):
        norm = build("norm", NormSpec("rmsnorm", width, 1e-5, name, suffix=""))
        norm.bind({name: (torch.randn(width, generator=g) * 0.2 + 1.0).to(STORE[dtype]).to(DEV)}, rt)
        norms.append(norm)
    for then in (True, False):
        stream = before.clone().to(DEV)
        normed = torch.full((n, width), float("nan"), dtype=STORE[dtype], device=DEV)
        ctx.closing = SublayerClosing(stream, norms[0], norms[1] if then else None, normed if then else None)
        branch = torch.full((n, width), float("nan"), device=DEV)
        part.forward(ctx, x.to(DEV), branch)
        if not ctx.closing.done:
            assert n * f["router"]["top"] < 8 or dtype == "float32" or not part.grouped
            continue
        gammas = [m.gamma.double().cpu().numpy() for m in norms]
        after = before.double().numpy()[rows] + P.norm(want, gammas[0], 1e-5)
        check(stream.cpu()[rows], after, tol, "the stream after the closing norm")
        if then:
            check(normed.cpu()[rows], P.norm(after, gammas[1], 1e-5), tol, "the norm that follows")
    rt.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 40, 300])
@pytest.mark.parametrize("width,f", [(256, dense(128, 0.5)), (76, dense(20, 1.2)), (128, dense(36, 1.5))])
def test_clamped_gated_feed_forward(dtype, n, width, f):
    rt = Runtime(DEV, STORE[dtype])
    part, w = ff_part(rt, width, f, n + width, STORE[dtype])
    g = torch.Generator().manual_seed(n)
    x = (torch.randn(n, width, generator=g) * 2).to(STORE[dtype])
    want = P.feed_forward(x.double().numpy(), f, w, "l0.mlp")
    ctx = Ctx()
    ctx.branch_is_fresh = True
    out = torch.full((n, width), float("nan"), device=DEV)
    part.forward(ctx, x.to(DEV), out)
    check(out, want, 3e-5 if dtype == "float32" else 2e-2, "feed-forward")
    loose = P.feed_forward(x.double().numpy(), {**f, "limit": 50.0}, w, "l0.mlp")
    assert np.abs(loose - want).max() > 0.02 * np.abs(want).max(), "the limit does not bind"
    rt.check_status()


def test_a_factor_on_a_norms_output():
    rt = Runtime(DEV, torch.bfloat16)
    g = np.random.RandomState(3)
    x, w = g.randn(9, 72), torch.tensor(g.randn(72)).bfloat16()
    for offset in (0.0, 1.0):
        norm = build("norm", NormSpec("rmsnorm", 72, 1e-5, "n", suffix="", offset=offset, gain=0.37))
        norm.bind({"n": w.to(DEV)}, rt)

        class C:
            memo = {}
        check(norm.forward(C(), f32(x)), 0.37 * P.norm(x, w.double().numpy() + offset, 1e-5), 8e-3, f"offset {offset}")


# -- the model ------------------------------------------------------------------------------------

def close(got, want, dtype, what):
    """Logits against the plain model's.  float32: the largest difference within 1e-4 of the largest logit.
    bfloat16: rounding of the activations to 8 bits of mantissa is the design's own noise, so the measure is the root mean
    square of the differences over all the rows given, held to 5 % of the logits' own; rows of tokens whose choice of experts
    is closer than that noise are NaN in ``want`` and not judged.  A fault of the cache or the state moves far more than that
    with these weights, and the float32 runs hold the same code to 1e-4."""
    if dtype == "float32":
        return check(got, want, TOL[dtype], what)
    g = got.detach().double().cpu().numpy()
    g = g.reshape(-1, g.shape[-1])
    w = np.asarray(want, dtype=np.float64).reshape(g.shape)
    assert np.isfinite(g).all(), f"{what}: NaN or infinity"
    rows = np.isfinite(w).all(axis=1)
    if not rows.any():
        return
    rms = float(np.sqrt(np.mean((g - w)[rows] ** 2)) / np.sqrt(np.mean(w[rows] ** 2)))
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


CLOSE_CALL = 0.015       # scores (with their corrections) a bfloat16 run may take the other way round


def blank_close_calls(rows, note):
    for m in note:
        rows[m < CLOSE_CALL] = np.nan
    assert np.isfinite(rows[:, 0]).mean() > 0.3 or len(rows) < 20, "hardly a row is left to judge"


def plain_logits(folder, tokens):
    """The plain model's logits; for a bfloat16 folder those of tokens with a close choice of experts are NaN."""
    cfg, w = P.load(folder)
    note = []
    logits = P.forward(cfg, w, tokens, note=note)
    if "bfloat16" in folder.name:
        blank_close_calls(logits, note)
    return logits


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_every_position_and_layer(folders, name, dtype):
    cfg = CONFIGS[name]
    t = toks(cfg, 150, 1)
    pcfg, w = P.load(folders[name, dtype])
    note = []
    want, streams = P.forward(pcfg, w, t, True, note)
    if dtype == "bfloat16":
        for a in [want] + streams:
            blank_close_calls(a, note)
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
    assert info["config"]["architecture"] == "Vuvalorn" and info["parameters"] > 0
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_across_pages(folders, dtype):
    """420 decoded tokens after a prompt of 150: pages pass by, and the kept inputs have been handed on 420 times."""
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
    engine.cache.check()


def test_long_prompt_on_the_tensor_core_paths(folders):
    """600 tokens in one step through sizes that the tensor-core kernels take, then ten tokens one by one: bfloat16 and
    float32 against the plain model."""
    cfg = CONFIGS["B"]
    t = toks(cfg, 610, 3)
    rows = list(range(0, 600, 7)) + [1, 2, 3, 63, 64, 65, 127, 128, 129, 255, 256, 511, 512, 599]
    for dtype in ("bfloat16", "float32"):
        want = plain_logits(folders["B", dtype], t)
        model = Model.load(folders["B", dtype], dtype=dtype)
        engine = Engine(model, max_tokens=64 * 11)
        s = engine.alloc_slot()
        close(engine.step([s], [t[:600]], [rows]), want[rows], dtype, f"{dtype}: a prompt of 600 tokens")
        out = torch.cat([engine.step([s], [[t[i]]]).clone() for i in range(600, 610)])
        close(out, want[600:], dtype, f"{dtype}: ten tokens after it")
        model.rt.check_status()


FAR = {"architecture": "Vuvalorn", "vocab": 64, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 20.0}, "logit_scale": 1.5,
       "layers": [att(2, 1, 16, 3, 1.0, 25.0, rot(1e4, 8)), att(4, 2, 80, 2, 0.4, 30.0, rot(1e4, 32), moe(3, 1, 2, 32))]}


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_far_back(tmp_path, dtype):
    """Sharp queries and keys, 560 positions: rows that look far back and across pages.  The same tokens with one token near
    the start exchanged answer otherwise far behind it."""
    folder = write_folder(tmp_path / dtype, FAR, 3, STORE[dtype], sharpen=3.0 if dtype == "float32" else 1.5)
    t = toks(FAR, 560, 8)
    want = plain_logits(folder, t)
    changes = []
    for at in (5, 62, 63, 64, 130):
        u = list(t)
        u[at] = (u[at] + 7) % 64
        changes.append(np.nan_to_num(np.abs(plain_logits(folder, u) - want)[300:]).max(axis=1))
    rows = sorted({0, 1, 2, 63, 64, 499, 559} | {300 + int(c.argmax()) for c in changes})
    assert max(c.max() for c in changes) > 0.02 * np.nanmax(np.abs(want)), "nothing far back shows"
    model = Model.load(folder, dtype=dtype)
    engine = Engine(model, max_tokens=1280)
    s = engine.alloc_slot()
    close(engine.step([s], [t], [rows]), want[rows], dtype, "a prompt with far keys")
    s2 = engine.alloc_slot()
    engine.step([s2], [t[:500]], [[]])
    out = torch.cat([engine.step([s2], [[t[i]]]).clone() for i in range(500, 535)])
    close(out, want[500:535], dtype, "decoded past far keys")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_of_a_sequence(folders, dtype):
    """Token by token from the first (the convolutions find zeros before it), on a slot whose last owner left its inputs."""
    for name in CONFIGS:
        cfg = CONFIGS[name]
        model = Model.load(folders[name, dtype], dtype=dtype)
        engine = Engine(model, max_tokens=PAGE, n_slots=1)
        rows = Rows(dtype, f"{name}: first tokens")
        for seed in (1, 2, 3):
            t = toks(cfg, 14, seed)
            want = plain_logits(folders[name, dtype], t)
            s = engine.alloc_slot()
            for i in range(14):
                rows.add(engine.step([s], [[t[i]]])[0], want[i], f"sequence {seed}, token {i}")
            engine.free_slot(s)
        rows.done()


def test_passes_keep_caches_of_their_own_and_their_vectors_differ(folders):
    """The plain model with the passes' vectors exchanged, and with one pass less, answers otherwise; the library's cache has a
    user per layer run."""
    pcfg, w = P.load(folders["A", "float32"])
    t = toks(CONFIGS["A"], 30, 4)
    want = P.forward(pcfg, w, t)
    other = P.forward(pcfg, {**w, "loop.step": w["loop.step"][::-1]}, t)
    fewer = P.forward({**pcfg, "loop": {**pcfg["loop"], "times": 2}}, w, t)
    for x in (other, fewer):
        assert np.abs(x - want).max() > 0.02 * np.abs(want).max()
    model = Model.load(folders["A", "float32"], dtype="float32")
    requests, _ = model.cache_requests()
    assert len(requests) == 8 and all(kv is not None and st is not None for kv, st in requests)
    engine = Engine(model, max_tokens=64)
    assert len({engine.cache.kv(i)[0].data_ptr() for i in range(8)}) == 8


def random_vuvalorn(rs):
    """A random configuration: head sizes in and out of what the tensor-core kernels take, any grouping of heads, taps from 1 to
    6, any feed-forward, a loop anywhere or nowhere."""
    width = int(rs.choice([72, 100, 136, 200, 256]))
    layers = []
    for i in range(int(rs.randint(1, 5))):
        mlp, u = None, rs.rand()
        if u < 0.4:
            mlp = dense(int(rs.choice([20, 64, 136])), float(rs.choice([0.5, 2.0, 7.0])))
        elif u < 0.9:
            E, I = int(rs.choice([1, 2, 4, 6, 12])), int(rs.choice([0, 1, 3, 8]))
            mlp = moe(E, I, int(rs.randint(1, E + I + 1)), int(rs.choice([16, 20, 64, 80])))
        kv, group, dim = int(rs.choice([1, 2, 3])), int(rs.choice([1, 2, 4, 8])), int(rs.choice([10, 16, 40, 64, 80, 128]))
        layers.append(att(kv * group, kv, dim, int(rs.randint(1, 7)), float(rs.choice([dim ** -0.5, 0.2])),
                          float(rs.choice([3.0, 15.0, 50.0])) if rs.rand() < 0.9 else None,
                          rot(float(rs.choice([1e4, 4e5, 300.0])), int(rs.choice([dim, dim // 2 // 2 * 2, 2]))) if rs.rand() < 0.9 else None, mlp))
    cfg = {"architecture": "Vuvalorn", "vocab": int(rs.randint(100, 600)), "width": width,
           "norm": {"eps": float(rs.choice([1e-6, 1e-5]))}, "embedding": {"scale": float(rs.choice([1.0, 8.0, 31.0]))},
           "logit_scale": float(rs.choice([1.0, 0.2, 3.0])), "layers": layers}
    if rs.rand() < 0.8:
        a = int(rs.randint(0, len(layers)))
        cfg["loop"] = {"start": a, "stop": int(rs.randint(a + 1, len(layers) + 1)), "times": int(rs.randint(1, 4))}
    return cfg


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", range(10))
def test_random_configuration_and_trace(tmp_path, seed, dtype):
    """Random configurations, each with a batch of unequal prompts (the first one cut in two steps the second time
    round), decoding with early leavers, then the same again on the slots, pages and state rows given back."""
    rs = np.random.RandomState(9000 + seed)
    cfg = random_vuvalorn(rs)
    folder = write_folder(tmp_path / dtype, cfg, seed, STORE[dtype])
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
