"""Podenex, slowly: numpy in float64, one function per mechanism, whole sequences, no cache.

It shares no code with the library: it reads config.json as a plain dict and model.safetensors with a
reader of its own, expands every latent row to keys and values, and runs each token's experts one by one.
The tests compare the library's kernels, its step function and its generation loop with these functions.
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


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def layer_norm(x, w, eps):
    """Mean taken off, divided by the root of the mean squared deviation; a gain, no bias."""
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def short_conv(u, w):
    """Causal convolution over time, a filter a channel, the last tap on the current token; u [T, C], w [C, taps]."""
    T, taps = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            at = t - taps + 1 + j
            if at >= 0:
                y[t] += w[:, j] * u[at]
    return y


def distance_bucket(n, rows, far):
    """Which of `rows` buckets the distance n falls in: single distances below rows / 2, then `rows - rows / 2` buckets
    that grow by a constant factor up to `far`, which the last one holds with everything beyond."""
    half = rows // 2
    if n < half:
        return n
    steps = math.log(n / half) / math.log(far / half) * (rows - half)
    near = round(steps)
    if abs(steps - near) < 1e-9:      # on a border: decided in whole numbers, (n / half)^(rows - half) against (far / half)^near
        m = rows - half
        steps = near if n ** m * half ** near >= far ** near * half ** m else near - 1
    return min(rows - 1, half + math.floor(steps))


def rotate_neighbours(x, positions, dims, base):
    """x [T, heads, dim]: the first `dims` of every head rotated, (2i, 2i + 1) as a pair."""
    out = x.copy()
    i = np.arange(dims // 2)
    ang = positions[:, None].astype(np.float64) * base ** (-2.0 * i / dims)
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def softmax_rows(s, seen, sink=None):
    """Weights over the keys that `seen` names; with `sink` the denominator holds exp(sink) as well."""
    s = np.where(seen, s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    total = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - top)
    return e / total


def attend(q, k, v, scale, seen, bias=None, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, V], seen [T, T], bias [H, T, T] or None; returns [T, H, V]."""
    H, G = q.shape[1], k.shape[1]
    out = np.zeros((q.shape[0], H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[h]
        out[:, h] = softmax_rows(s, seen, sink) @ v[:, g]
    return out


def window_sight(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def chunk_sight(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def distance_bias(table, far, T):
    """[heads, T, T]: the table's row for the bucket of i - j (0 above the diagonal)."""
    of = np.array([distance_bucket(n, table.shape[0], far) for n in range(T)], dtype=np.int64)
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return np.where(j <= i, table[of[np.maximum(i - j, 0)]].transpose(2, 0, 1), 0.0)


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


# ------------------------------------------------------------------------------------------ mixers
def _mixed(v, W, p, m, carry):
    """The layer's values: blended with the first such layer's where the layer mixes; `carry` keeps the first's."""
    if not m.get("v_mix"):
        return v
    if "v_first" not in carry:
        carry["v_first"] = v
        return v
    return mix_values(v, carry["v_first"].reshape(v.shape), float(W[p + "vmix"].reshape(())))


def chunked_mixer(h, W, p, m, carry):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in ("q", "k", "v"))
    v = _mixed(v, W, p, m, carry)
    o = attend(q.reshape(T, H, D), k.reshape(T, G, D), v.reshape(T, G, V), m["scale"], chunk_sight(T, m["mask"]["size"]),
               bias=distance_bias(W[p + "rel"], m["bias_max"], T))
    o = o * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ W[p + "o"].T


def windowed_mixer(h, W, p, m, eps, carry):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (h @ W[p + n].T + W[p + n + ".b"] for n in ("q", "k", "v"))
    q = rms_norm(q.reshape(T, H, D), W[p + "q.norm"], eps)
    k = rms_norm(k.reshape(T, G, D), W[p + "k.norm"], eps)
    v = _mixed(v, W, p, m, carry)
    o = attend(q, k, v.reshape(T, G, V), m["scale"], window_sight(T, m["mask"]["size"]), sink=0.0)
    return o.reshape(T, H * V) @ W[p + "o"].T + W[p + "o.b"]


def latent_mixer(h, W, p, m, positions, eps):
    H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).reshape(T, H, D + R)
    down = h @ W[p + "dkv"].T
    c = rms_norm(down[:, :C], W[p + "dkv.norm"], eps)
    shared = rotate_neighbours(down[:, None, C:], positions, m["rot"]["dims"], m["rot"]["base"])
    q_rot = rotate_neighbours(q[:, :, D:], positions, m["rot"]["dims"], m["rot"]["base"])
    k = (c @ W[p + "uk"].T).reshape(T, H, D)
    v = (c @ W[p + "uv"].T).reshape(T, H, V)
    q = np.concatenate([q[:, :, :D], q_rot], axis=2)
    k = np.concatenate([k, np.repeat(shared, H, axis=1)], axis=2)
    o = attend(q, k, v, m["scale"], window_sight(T, m["mask"]["size"]))
    return (o.reshape(T, H * V) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forward
def route(z, r):
    """Chosen experts [T, top] and their weights from the router's logits."""
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    choice = s
    groups = r.get("groups")
    if groups:
        best = s.reshape(len(s), groups["count"], -1).max(axis=-1)
        kept = np.argsort(-best, axis=-1, kind="stable")[:, :groups["keep"]]
        allowed = np.zeros(best.shape, dtype=bool)
        np.put_along_axis(allowed, kept, True, axis=1)
        choice = np.where(np.repeat(allowed, s.shape[1] // groups["count"], axis=1), s, -np.inf)
    chosen = np.argsort(-choice, axis=-1, kind="stable")[:, :r["top"]]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def expert(h, up, down):
    return relu_squared(h @ up.T) @ down.T


def experts_ff(h, W, p, mlp):
    chosen, weights = route(h @ W[p + "router"].T, mlp["router"])
    out = np.zeros((h.shape[0], W[p + "e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weights[t]):
            out[t] += w * expert(h[t:t + 1], W[f"{p}e{e}.up"], W[f"{p}e{e}.down"])[0]
    if mlp.get("shared"):
        out += expert(h, W[p + "shared.up"], W[p + "shared.down"])
    return out


def side_input(x, tokens, W, p, layer, dim, eps):
    e = W["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    return rms_norm((gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T, W[p + "side.norm"], eps)


# ------------------------------------------------------------------------------------------ the model
def forward(cfg, W, tokens, per_layer=False):
    """Logits [T, vocab] of one sequence from its first token; with `per_layer` also the stream after every layer."""
    tokens = np.asarray(tokens, dtype=np.int64)
    positions = np.arange(len(tokens))
    eps = cfg["norm"]["eps"]
    x = W["embed"][tokens]
    streams, carry = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = layer_norm(x, W[p + "norm1"], eps)
        if layer["type"] == "attention":
            x = x + chunked_mixer(h, W, p + "mix.", m, carry)
        elif layer["type"] == "attention_2":
            x = x + windowed_mixer(h, W, p + "mix.", m, eps, carry)
        else:
            x = x + latent_mixer(h, W, p + "mix.", m, positions, eps)
        if layer.get("mlp") is not None:
            x = x + experts_ff(layer_norm(x, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"])
        if cfg.get("token_side"):
            x = x + side_input(x, tokens, W, p, i, cfg["token_side"]["dim"], eps)
        streams.append(x.copy())
    logits = layer_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, np.stack(streams)) if per_layer else logits


def generate(cfg, W, prompt, steps):
    """Greedy continuation: the first of the largest logits, `steps` times."""
    ids = list(prompt)
    for _ in range(steps):
        ids.append(int(np.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]
