"""A plain, slow statement of the Vuvalorn decoder: one function per mechanism, float64 NumPy on the CPU, one masked
matrix per head.  It shares no code with the library: it has its own file reader, reads ``config.json`` itself and
knows nothing of pages, slots, steps or state rows.  The tests hold the library to it.

Notation: x is the residual stream [T, W], h a sublayer's input, p a position (from 0), H query heads, G key/value
heads, d the lanes of a head.

The design in short.  x = scale * embed[token].  A layer norms the input AND the output of both sublayers:
x <- x + n1b(attention(n1(x))), x <- x + n2b(ff(n2(x))).  A range of layers runs several times in a row with the same
weights, and row t of ``loop.step`` is added to x before pass t.  Attention has no value projection (a value is its key
between the short convolution and the key norm), caps its scores with a tanh and weighs every head's output with one
sigmoid.  The feed-forward is one clamped gated layer, or routed experts some of which are the identity.  The logits are
the final norm times the embedding table, times a constant.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np

SWISH = 1.702            # the dense feed-forward's gate is g * sigmoid(SWISH * g)


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


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def norm(x, w, eps):
    """x over the root of its mean square along the last axis (eps inside the root), times the weight."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


# -- attention ----------------------------------------------------------------------------

def short_conv(u, w):
    """u [T, channels], w [channels, taps]: every channel by itself, y_t = sum_j w[:, j] u_(t - taps + 1 + j), with zeros
    before the sequence's start."""
    T, taps = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            if t - (taps - 1) + j >= 0:
                y[t] += w[:, j] * u[t - (taps - 1) + j]
    return y


def rotate_pairs(x, positions, rot):
    """x [T, heads, d]: lanes 2i and 2i + 1 of a head's first ``dims`` turn by p * base^(-2i / dims); the rest pass."""
    dims = rot["dims"]
    f = float(rot["base"]) ** (-np.arange(0, dims, 2, dtype=np.float64) / dims)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    y = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * c - v * s
    y[..., 1:dims:2] = v * c + u * s
    return y


def capped(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def attention_core(q, k, v, scale, cap):
    """q [T, H, d], k and v [T, G, d] -> [T, H, d]: causal softmax over the capped scores."""
    T, H = q.shape[:2]
    group = H // k.shape[1]
    see = np.tril(np.ones((T, T), dtype=bool))
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        s = capped((q[:, h] @ k[:, h // group].T) * scale, cap)
        out[:, h] = softmax(np.where(see, s, -np.inf)) @ v[:, h // group]
    return out


def attention(h, m, w, name, eps):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w[f"{name}.q"].T, h @ w[f"{name}.k"].T
    if f"{name}.q.conv" in w:
        q, k = short_conv(q, w[f"{name}.q.conv"]), short_conv(k, w[f"{name}.k.conv"])
    q, k = q.reshape(T, H, d), k.reshape(T, G, d)
    v = k                                                   # before norm and rotation
    q, k = norm(q, w[f"{name}.q.norm"], eps), norm(k, w[f"{name}.k.norm"], eps)
    if m.get("rot"):
        q, k = (rotate_pairs(z, np.arange(T), m["rot"]) for z in (q, k))
    o = attention_core(q, k, v, m["scale"], m.get("softcap"))
    o = o * sigmoid(h @ w[f"{name}.g"].T)[:, :, None]       # one number per head
    return o.reshape(T, H * d) @ w[f"{name}.o"].T


# -- feed-forward ---------------------------------------------------------------------------

def clamped_gated(h, w, name, limit):
    g = np.minimum(h @ w[f"{name}.gate"].T, limit)
    u = np.clip(h @ w[f"{name}.up"].T, -limit, limit)
    return (g * sigmoid(SWISH * g) * (u + 1.0)) @ w[f"{name}.down"].T


def expert(h, w, name):
    return (silu(h @ w[f"{name}.gate"].T) * (h @ w[f"{name}.up"].T)) @ w[f"{name}.down"].T


def route(scores, correction, top):
    """One token's choice: the ``top`` largest of score + correction (the lower index wins a tie); weights are the scores
    themselves."""
    ids = np.argsort(-(scores + correction), kind="stable")[:top]
    return ids, scores[ids]


def margins(scores, correction, top):
    """How far apart the last chosen and the first not chosen lie, per token (infinity where everything is chosen)."""
    if top == scores.shape[1]:
        return np.full(len(scores), np.inf)
    key = np.sort(scores + correction, axis=1)[:, ::-1]
    return key[:, top - 1] - key[:, top]


def routed_experts(h, f, w, name, note=None):
    """The first ``experts`` outputs of the router are experts with tensors, the last ``identity`` hand the input on.
    ``note``: a list that receives the choices' margins."""
    n = f["router"]["experts"]
    s = softmax(h @ w[f"{name}.router"].T)
    if note is not None:
        note.append(margins(s, w[f"{name}.correction"], f["router"]["top"]))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(*route(s[t], w[f"{name}.correction"], f["router"]["top"])):
            out[t] += weight * (h[t] if e >= n else expert(h[t:t + 1], w, f"{name}.e{e}")[0])
    return out


def feed_forward(h, f, w, name, note=None):
    return clamped_gated(h, w, name, f["limit"]) if f["kind"] == "dense" else routed_experts(h, f, w, name, note)


# -- the model ------------------------------------------------------------------------------

def runs(cfg):
    """(layer, pass or None) in running order; the pass's number stands at its first layer."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + body + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, with_streams=False, note=None):
    """Logits [T, vocab] of a whole sequence (and the stream after every layer run); ``note``: see ``routed_experts``."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    streams = []
    for i, step in runs(cfg):
        layer = cfg["layers"][i]
        if step is not None:
            x = x + w["loop.step"][step]
        y = attention(norm(x, w[f"l{i}.norm1"], eps), layer["mixer"], w, f"l{i}.mix", eps)
        x = x + norm(y, w[f"l{i}.norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(norm(x, w[f"l{i}.norm2"], eps), layer["mlp"], w, f"l{i}.mlp", note)
            x = x + norm(y, w[f"l{i}.norm2b"], eps)
        streams.append(x.copy())
    logits = norm(x, w["final.norm"], eps) @ w["embed"].T * cfg.get("logit_scale", 1.0)
    return (logits, streams) if with_streams else logits


def greedy(cfg, w, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(np.argmax(forward(cfg, w, t)[-1])))
    return t[len(prompt):]
