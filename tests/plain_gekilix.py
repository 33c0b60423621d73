"""A plain, slow statement of the Gekilix decoder: one function per mechanism, float64 NumPy on the CPU, one masked
matrix per head for attention and one token at a time in the recurrence.  It shares no code with the library: it has
its own file reader, reads ``config.json`` itself and knows nothing of pages, slots, steps or state rows.  The tests
hold the library to it.

Notation: x is the residual stream [T, W], h a sublayer's input, p a position (from 0), H heads, G groups (of B and C,
or of keys and values), N the rows and P the columns of a head's recurrent state.

The design in short.  x = embed[token]; per layer x <- x + mixer(norm1(x)), then, if the layer has a feed-forward,
x <- x + ff(norm2(x)); logits = head norm(x).  Norms multiply by one plus their weight.  Mixers: ``mamba2`` (a state
space with one decay per head and token) and ``attention`` (softmax over a sliding window and the sequence's first
tokens).  Feed-forward: routed experts with sigmoid scores that weigh the experts' INPUT, and a gated shared expert.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np


# -- files ----------------------------------------------------------------------------

def read_safetensors(path) -> dict:
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    data = raw[8 + n:]
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        buf, dt = data[lo:hi], info["dtype"]
        if dt == "BF16":
            a = (np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif dt == "F32":
            a = np.frombuffer(buf, dtype="<f4").astype(np.float64)
        else:
            raise ValueError(f"{name}: element type {dt}")
        out[name] = a.reshape(info["shape"])
    return out


def load(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


# -- small functions --------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms(x, eps):
    """x over the root of its mean square along the last axis, eps inside the root; no weight."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """A norm of the stream: the weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


# -- attention ----------------------------------------------------------------------------

def frequencies(rot):
    """Radians a position for every pair of lanes.  With ``scaling`` a pair whose wavelength is longer than
    original / low turns ``factor`` times slower, one shorter than original / high as it is, and one between the two
    is blended."""
    dims = rot["dims"]
    f = np.array([rot["base"] ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)
    sc = rot.get("scaling")
    if not sc:
        return f
    out = []
    for v in f:
        wave = 2.0 * math.pi / v
        if wave < sc["original"] / sc["high"]:
            out.append(v)
        elif wave > sc["original"] / sc["low"]:
            out.append(v / sc["factor"])
        else:
            s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * v / sc["factor"] + s * v)
    return np.array(out)


def rotate_pairs(x, positions, rot):
    """x [T, H, d]: lanes 2i and 2i + 1 of a head's first ``dims`` turn by position * f_i; the rest pass."""
    f = frequencies(rot)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    y = x.copy()
    n = 2 * len(f)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2] = u * c - v * s
    y[..., 1:n:2] = v * c + u * s
    return y


def visible(i, j, mask):
    """Whether the query at position i sees the key at position j."""
    if j > i:
        return False
    if not mask:
        return True
    return i - j < mask["size"] or j < mask.get("keep_first", 0)


def attention_core(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]."""
    T, H = q.shape[:2]
    group = H // k.shape[1]
    see = np.array([[visible(i, j, mask) for j in range(T)] for i in range(T)])
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T) * scale
        s = np.where(see, s, -np.inf)
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (w / w.sum(axis=1, keepdims=True)) @ v[:, h // group]
    return out


def attention(h, m, w, name, eps):
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    # one norm over all the heads' lanes at once, before the split and before the rotation
    q = rms(h @ w[f"{name}.q"].T, eps) * w[f"{name}.q.norm"]
    k = rms(h @ w[f"{name}.k"].T, eps) * w[f"{name}.k.norm"]
    q, k = q.reshape(T, H, d), k.reshape(T, G, d)
    v = (h @ w[f"{name}.v"].T).reshape(T, G, e)
    if m.get("rot"):
        q, k = (rotate_pairs(t, np.arange(T), m["rot"]) for t in (q, k))
    o = attention_core(q, k, v, m["scale"], m.get("mask"))
    return o.reshape(T, H * e) @ w[f"{name}.o"].T


# -- the state space ----------------------------------------------------------------------

def short_conv(x, w, b):
    """x [T, channels], w [channels, taps]: y_t = sum_j w[:, j] x_(t - taps + 1 + j) + b, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            at = t - (taps - 1) + j
            if at >= 0:
                y[t] += w[:, j] * x[at]
    return y + b


def state_space(x, B, C, dt, log_decay_rate, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (after softplus): per head
    S <- exp(-exp(rate) dt) S + dt B x^T,  y = S^T C + D x.  -> y [T, H, P]."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P))
    y = np.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(log_decay_rate[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y


def gated_group_norm(y, z, w, n_groups, eps):
    """The gate first, then every one of n_groups equal parts over its own root mean square, then the weight."""
    T, inner = y.shape
    u = (y * silu(z)).reshape(T, n_groups, inner // n_groups)
    return rms(u, eps).reshape(T, inner) * w


def mamba2(h, m, w, name, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    p = h @ w[f"{name}.in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, w[f"{name}.conv"], w[f"{name}.conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[f"{name}.dt_bias"])
    y = state_space(x, B, C, dt, w[f"{name}.A_log"], w[f"{name}.D"]).reshape(T, inner)
    return gated_group_norm(y, z, w[f"{name}.norm"], m["norm_groups"], eps) @ w[f"{name}.o"].T


# -- feed-forward ---------------------------------------------------------------------------

def gated_expert(h, w, name):
    return (silu(h @ w[f"{name}.gate"].T) * (h @ w[f"{name}.up"].T)) @ w[f"{name}.down"].T


def route(scores, top):
    """The ``top`` largest scores of one token (the lower index wins a tie)."""
    return np.argsort(-scores, kind="stable")[:top]


def routed_experts(h, f, w, name):
    out = np.zeros_like(h)
    s = sigmoid(h @ w[f"{name}.router"].T)
    for t in range(h.shape[0]):
        for e in route(s[t], f["router"]["top"]):
            out[t] += gated_expert(s[t, e] * h[t:t + 1], w, f"{name}.e{e}")[0]
    if f.get("shared"):
        out += sigmoid(h @ w[f"{name}.shared.sg"].T) * gated_expert(h, w, f"{name}.shared")
    return out


# -- the model ------------------------------------------------------------------------------

MIXERS = {"mamba2": mamba2, "attention": attention}


def forward(cfg, w, tokens, with_streams=False):
    """Logits [T, vocab] of a whole sequence (and the stream after every layer)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        x = x + MIXERS[layer["type"]](norm(x, w[f"l{i}.norm1"], eps), layer["mixer"], w, f"l{i}.mix", eps)
        if layer.get("mlp"):
            x = x + routed_experts(norm(x, w[f"l{i}.norm2"], eps), layer["mlp"], w, f"l{i}.mlp")
        streams.append(x.copy())
    logits = norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, streams) if with_streams else logits


def greedy(cfg, w, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(np.argmax(forward(cfg, w, t)[-1])))
    return t[len(prompt):]
