"""Small Podenex configurations and helpers shared by the CPU and GPU tests.

The configurations differ from one another in every size and option: chunks and windows shorter than a page, longer
than a page (and no multiple of it), very short, and of one position; plain and grouped heads, values of the keys'
size, narrower and wider; convolutions of 4, 2 and 1 taps (the last carries no state); distance tables of few and
many rows that saturate inside the chunk and beyond it; values that are carried from the first layer into layers of
the same kind and of the other, whose head counts differ, and layers that do not take part, the first to take part
being of either kind and not always the model's first; cached rows whose rotated part is turned whole or in part;
experts with and without groups, with and without a shared expert, all chosen or one; layers without a feed-forward; with
and without the per-layer input from the token ids; a third model whose sizes are no multiples of 8 anywhere; a
fourth with head sizes of the tensor-core kernels.
"""
import copy
import json
import os

import numpy as np


def _moe(experts, top, ff, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router, **({"shared": {"ff": shared}} if shared else {})}


def _mixed(v_mix):
    return {} if v_mix is None else {"v_mix": v_mix}


def _chunked(dim, vdim, heads, kv, chunk, conv, rows, far, scale, mlp, v_mix=True):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "dim": dim, "vdim": vdim, "heads": heads, "kv_heads": kv, "scale": scale, "conv": conv, "bias_max": far, "bias_rows": rows,
        "mask": {"size": chunk}, **_mixed(v_mix)}}


def _windowed(dim, vdim, heads, kv, window, scale, mlp, v_mix=True):
    return {"type": "attention_2", "mlp": mlp, "mixer": {
        "dim": dim, "vdim": vdim, "heads": heads, "kv_heads": kv, "scale": scale, "mask": {"size": window}, **_mixed(v_mix)}}


def _latent(heads, dim, rot_dim, rot, base, vdim, q_rank, kv_rank, window, scale, mlp):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "rot": {"dims": rot, "base": base}, "vdim": vdim, "q_rank": q_rank,
        "kv_rank": kv_rank, "scale": scale, "mask": {"size": window}}}


CONFIGS = {
    "pod_a": {"architecture": "Podenex", "vocab": 300, "width": 64, "norm": {"eps": 1e-5}, "token_side": {"dim": 8}, "layers": [
        _chunked(16, 32, 4, 2, 40, 4, 12, 25, 0.3, _moe(8, 2, 24, groups=(4, 2), shared=40)),
        _latent(3, 16, 8, 8, 500.0, 24, 20, 32, 33, 0.25, _moe(8, 3, 24)),
        _windowed(32, 16, 8, 4, 20, 0.2, _moe(4, 1, 16, groups=(2, 1), shared=8)),
        _chunked(32, 32, 2, 2, 90, 2, 8, 200, 0.25, None, v_mix=None)]},
    "pod_b": {"architecture": "Podenex", "vocab": 200, "width": 96, "norm": {"eps": 1e-6}, "layers": [
        _windowed(48, 48, 3, 3, 70, 0.2, _moe(6, 6, 32), v_mix=False),
        _windowed(16, 48, 6, 2, 130, 0.3, None),
        _latent(2, 32, 48, 32, 10000.0, 16, 48, 96, 100, 0.15, _moe(6, 2, 32, groups=(3, 3), shared=16)),
        _chunked(48, 32, 6, 3, 70, 1, 32, 64.5, 0.2, _moe(9, 2, 16, groups=(9, 4)))]},
    "pod_c": {"architecture": "Podenex", "vocab": 101, "width": 60, "norm": {"eps": 1e-5}, "token_side": {"dim": 5}, "layers": [
        _latent(3, 10, 6, 4, 50.0, 7, 9, 14, 11, 0.3, _moe(5, 1, 14, shared=6)),
        _chunked(12, 10, 3, 1, 9, 3, 5, 7, 0.35, _moe(5, 2, 14)),
        _windowed(6, 5, 4, 2, 1, 0.4, _moe(3, 3, 10, groups=(3, 3))),
        _windowed(10, 10, 3, 1, 7, 0.4, None)]},
    "pod_d": {"architecture": "Podenex", "vocab": 160, "width": 128, "norm": {"eps": 1e-6}, "token_side": {"dim": 16}, "layers": [
        _windowed(64, 64, 4, 1, 65, 0.12, _moe(8, 2, 40, groups=(2, 1), shared=48)),
        _chunked(128, 64, 2, 1, 128, 4, 16, 100, 0.1, _moe(4, 2, 40, shared=24)),
        _latent(4, 64, 32, 32, 1e6, 64, 64, 64, 128, 0.1, _moe(4, 2, 40))]},
}
SEEDS = {"pod_a": 3, "pod_b": 4, "pod_c": 5, "pod_d": 6}
TOL = {"float32": 1e-4, "bfloat16": 8e-2}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name])


def write_model(folder: str, cfg: dict, seed: int, scale_up: float = 6.0) -> str:
    """A model folder with random weights through the library's own random-weights mode, the matrices scaled up so that
    the mixers and the experts matter in the logits; a table of distances' rows that are well apart."""
    import torch

    import ember_cpp_b200 as E
    from ember_cpp_b200.weights import read_folder, write_file
    E.write_random_model(folder, E.config.config_from_dict(cfg), seed)
    tensors = {name: t.clone() for name, t in read_folder(folder).items()}     # (the file is mapped: copies, then rewrite)
    for name, t in tensors.items():
        if name.endswith(".rel"):
            tensors[name] = (t.float() * 2.0).to(torch.bfloat16)
        elif name in ("embed", "head"):
            tensors[name] = (t.float() * 2.0).to(torch.bfloat16)
        elif t.dim() == 2 and not name.endswith((".conv", ".router", "side.embed")):
            tensors[name] = (t.float() * scale_up).to(torch.bfloat16)
    write_file(os.path.join(folder, "model.safetensors"), tensors, {"format": "pt"})
    stored = copy.deepcopy(cfg)
    for layer in stored["layers"]:                       # (what only random-weights mode reads: the table's shape says it)
        layer["mixer"].pop("bias_rows", None)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(stored, f)
    return folder


def ids(seed: int, vocab: int, n: int) -> list:
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def row_error(got, ref) -> float:
    """Worst row of rms(delta - mean(delta)) / rms(ref - mean(ref))."""
    return float(row_errors(got, ref).max())


def row_errors(got, ref):
    got, ref = np.atleast_2d(np.asarray(got, dtype=np.float64)), np.atleast_2d(np.asarray(ref, dtype=np.float64))
    d, r = got - ref, ref - ref.mean(-1, keepdims=True)
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean(-1))


def rows_agree(got, ref, dtype: str) -> bool:
    """`got` against the plain model's `ref` (lists of [rows, vocab] arrays).  In 32-bit every row is within TOL.  In
    bfloat16 a rounding can turn a near tie of the router's choice the other way, and the token then runs another expert
    than the plain model's: some rows may differ by more (at most one in five), the typical row must not."""
    errors = np.concatenate([row_errors(g, r) for g, r in zip(got, ref)])
    if dtype == "float32":
        return bool(errors.max() < TOL[dtype])
    return bool((errors >= TOL[dtype]).mean() <= 0.2 and np.median(errors) < TOL[dtype] / 2)
