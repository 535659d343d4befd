"""Mamusun, slowly: numpy in float64, one function per mechanism, whole sequences, no cache.

It shares no code with the library: it reads config.json as a plain dict and model.safetensors with
a reader of its own, and walks the recurrence token by token.  The tests compare the library's
kernels, its step function and its generation loop with these functions.
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


# ------------------------------------------------------------------------------------------ files
def read_safetensors(path):
    """name -> float64 array (integer tables as int64)."""
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw, shape = data[lo:hi], tuple(info["shape"])
        kind = info["dtype"]
        if kind == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif kind == "F32":
            a = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif kind == "I32":
            a = np.frombuffer(raw, dtype="<i4").astype(np.int64)
        else:
            raise ValueError(f"{name}: element type {kind}")
        out[name] = a.reshape(shape)
    return out


def load_folder(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# ------------------------------------------------------------------------------------------ small functions
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    """Rows divided by their root mean square, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return unit_rms(x, eps) * w


def short_conv(u, w, b):
    """Causal convolution over time, a filter a channel, zeros before the start: u [T, C], w [C, taps], b [C]."""
    T, taps = u.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    y = np.tile(b, (T, 1)).astype(np.float64)
    for j in range(taps):
        y += padded[j:j + T] * w[:, j]
    return y


# ------------------------------------------------------------------------------------------ rotations
def base_freqs(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_freqs(dims, rot):
    """Frequencies scaled by bands of wavelengths: short waves stay, long ones are slowed by `factor`, a linear
    blend between the two bounds."""
    out, s = [], rot.get("scaling")
    for f in base_freqs(dims, rot["base"]):
        if s:
            wave = 2 * math.pi / f
            if wave < s["original"] / s["high"]:
                pass
            elif wave > s["original"] / s["low"]:
                f = f / s["factor"]
            else:
                part = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - part) * f / s["factor"] + part * f
        out.append(f)
    return np.array(out)


def ramp_freqs(dims, rot):
    """Frequencies blended by a ramp over the pair index, and the factor on cos and sin (YaRN)."""
    freqs, s = base_freqs(dims, rot["base"]), rot.get("scaling")
    if not s:
        return np.array(freqs), 1.0

    def index_of(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))
    lo = max(math.floor(index_of(s["fast"])), 0)
    hi = min(math.ceil(index_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1.0 - r))
    return np.array(out), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, freqs, magnitude, interleaved):
    """x [T, heads, dim]: the first 2 * len(freqs) dimensions of every head rotated; pair i is dimensions (2i, 2i + 1)
    where `interleaved`, else (i, i + len(freqs))."""
    n = len(freqs)
    out = x.copy()
    ang = positions[:, None].astype(np.float64) * freqs
    c, s = np.cos(ang)[:, None, :] * magnitude, np.sin(ang)[:, None, :] * magnitude
    iu, iv = (np.arange(n) * 2, np.arange(n) * 2 + 1) if interleaved else (np.arange(n), np.arange(n) + n)
    a, b = x[..., iu], x[..., iv]
    out[..., iu] = a * c - b * s
    out[..., iv] = b * c + a * s
    return out


# ------------------------------------------------------------------------------------------ attention
def attend(q, k, v, scale, window=0, sinks=None):
    """q [T, H, D]; k [T, G, D]; v [T, G, V]; a query at i sees the keys j <= i (with a window: the last `window` of
    them); sinks [H]: exp(sink) joins the softmax's denominator."""
    T, H, D = q.shape
    G = k.shape[1]
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = (j <= i) & ((i - j < window) if window else True)
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        top = s.max(axis=1, keepdims=True)
        if sinks is not None:
            top = np.maximum(top, sinks[h])
        e = np.exp(s - top)
        den = e.sum(axis=1, keepdims=True) + (np.exp(sinks[h] - top) if sinks is not None else 0.0)
        out[:, h] = (e / den) @ v[:, g]
    return out


def window_mixer(h, W, p, m, eps, kept):
    """The windowed attention with a norm a head and no rotation; with `kv_from` the keys and values are another
    layer's (`kept`: layer -> (k, v)).  Returns the output and this layer's keys and values."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = norm_plain((h @ W[p + "q"].T).reshape(T, H, D), W[p + "q.norm"], eps)
    if m.get("kv_from") is not None:
        k, v = kept[m["kv_from"]]
    else:
        k = norm_plain((h @ W[p + "k"].T).reshape(T, G, D), W[p + "k.norm"], eps)
        v = (h @ W[p + "v"].T).reshape(T, G, V)
    o = attend(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(T, H * V) @ W[p + "o"].T, (k, v)


def left_mixer(h, W, p, m, eps, positions):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    freqs = banded_freqs(m["rot"]["dims"], m["rot"])
    q = unit_rms(rotate((h @ W[p + "q"].T).reshape(T, H, D), positions, freqs, 1.0, True), eps)
    k = unit_rms(rotate((h @ W[p + "k"].T).reshape(T, G, D), positions, freqs, 1.0, True), eps)
    v = (h @ W[p + "v"].T).reshape(T, G, V)
    return attend(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, H * V) @ W[p + "o"].T


def key_value_mixer(h, W, p, m, eps, positions):
    """Attention whose values are its keys as projected; norms over whole rows, before the rotation; a learned sink."""
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    T = h.shape[0]
    q, k = h @ W[p + "q"].T + W[p + "q.b"], h @ W[p + "k"].T + W[p + "k.b"]
    v = k.reshape(T, G, D)
    freqs, mag = ramp_freqs(m["rot"]["dims"], m["rot"])
    q = rotate(norm_plain(q, W[p + "q.norm"], eps).reshape(T, H, D), positions, freqs, mag, False)
    k = rotate(norm_plain(k, W[p + "k.norm"], eps).reshape(T, G, D), positions, freqs, mag, False)
    return attend(q, k, v, m["scale"], 0, W[p + "sink"]).reshape(T, H * D) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ the recurrence
def block_gates(u, w, b):
    """sigmoid of a product per part: u [T, C] in w.shape[0] equal parts, w [parts, n, n] ([out, in]), b [parts, n]."""
    T, C = u.shape
    parts, n = w.shape[0], w.shape[1]
    z = np.einsum("tbi,boi->tbo", u.reshape(T, parts, n), w) + b
    return sigmoid(z).reshape(T, C)


def gated_recurrence(u, r, i, lam, S=None):
    """log a = -8 r softplus(lam);  S <- a S + sqrt(1 - a^2) i u.  Returns S after every token [T, C]."""
    S = np.zeros(u.shape[1]) if S is None else S.copy()
    out = np.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = np.exp(log_a) * S + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def right_mixer(h, W, p):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = short_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r, i = block_gates(u, W[p + "ra"], W[p + "ra.b"]), block_gates(u, W[p + "ri"], W[p + "ri.b"])
    return (gated_recurrence(u, r, i, W[p + "lam"]) * y) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forward
def poly_norm(z, four, eps):
    a, b, c, e = four
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def dense_ff(h, W, p, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(z, top):
    """The `top` largest logits of every row (the lower index first among equals) and the softmax over them."""
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    picked = np.take_along_axis(z, chosen, axis=1)
    e = np.exp(picked - picked.max(axis=1, keepdims=True))
    return chosen, e / e.sum(axis=1, keepdims=True)


def experts_ff(h, W, p, mlp):
    chosen, weights = route(h @ W[p + "router"].T + W[p + "router.b"], mlp["router"]["top"])
    out = np.zeros((h.shape[0], W[p + "e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, wt in zip(chosen[t], weights[t]):
            q = f"{p}e{e}."
            out[t] += wt * clamped_expert(h[t:t + 1], W[q + "gate"], W[q + "up"], W[q + "down"], mlp["expert"]["limit"])[0]
    return out


# ------------------------------------------------------------------------------------------ the model
def forward(cfg, W, tokens, per_layer=False):
    """Logits [T, vocab] of one sequence from its first token; with `per_layer` also the stream after every layer."""
    tokens = np.asarray(tokens, dtype=np.int64)
    positions = np.arange(len(tokens))
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = W["embed"][tokens]
    results, kept, streams = [x], {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            y, kept[i] = window_mixer(x, W, p + "mix.", m, eps, kept)
        elif layer["type"] == "attention_2":
            y = key_value_mixer(x, W, p + "mix.", m, eps, positions)
        else:
            y = 0.5 * norm_plain(left_mixer(x, W, p + "mix.left.", m["left"], eps, positions), W[p + "mix.left.out"], eps) \
                + 0.5 * norm_plain(right_mixer(x, W, p + "mix.right."), W[p + "mix.right.out"], eps)
        x = norm_around_zero(alpha * x + y, W[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            f = dense_ff(x, W, p + "mlp.", eps) if mlp["kind"] == "dense" else experts_ff(x, W, p + "mlp.", mlp)
            x = norm_around_zero(alpha * x + f, W[p + "norm2"], eps)
        results.append(x)
        x = sum(w * r for w, r in zip(W[p + "dwa"], results))
        streams.append(x.copy())
    logits = norm_around_zero(x, W["final.norm"], eps) @ W["head"].T
    return (logits, np.stack(streams)) if per_layer else logits


def generate(cfg, W, prompt, steps):
    """Greedy continuation: the first of the largest logits, `steps` times."""
    ids = list(prompt)
    for _ in range(steps):
        ids.append(int(np.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]
