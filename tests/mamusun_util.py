"""Small Mamusun configurations and helpers shared by the CPU and GPU tests.

The configurations differ from one another in every size and option: windows shorter than a page, longer than a page (and
no multiple of it) and very short; plain and grouped heads, values of the keys' size and of another; a part of every head
rotated or all of it, with and without the frequencies' scaling; layers that read another layer's keys through a narrower
and through a wider window, two of them reading the same one, one beside a norm; recurrences of one block and of several,
convolutions of 4, 2 and 1 taps (the last carries no state); dense and expert feed-forwards and layers without one;
all experts chosen or one; a factor of one and of more on the stream; a third model whose sizes are no multiples of 8
anywhere; a fourth with the head sizes that take the tensor-core kernels of plain attention.
"""
import copy
import json
import os

import numpy as np

BANDS = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}
YARN = {"factor": 8.0, "original": 96, "fast": 8.0, "slow": 0.5}
DENSE = lambda ff: {"kind": "dense", "ff": ff}  # noqa: E731


def _moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _window(dim, vdim, heads, kv, window, scale, mlp, **more):
    return {"type": "attention", "mixer": {"dim": dim, "vdim": vdim, "heads": heads, "kv_heads": kv, "scale": scale,
                                           "mask": {"size": window}, **more}, "mlp": mlp}


def _keyvalue(dim, heads, kv, rot_dims, base, scaling, scale, mlp):
    rot = {"dims": rot_dims, "base": base, **({"scaling": scaling} if scaling else {})}
    return {"type": "attention_2", "mixer": {"dim": dim, "vdim": dim, "heads": heads, "kv_heads": kv, "scale": scale, "rot": rot}, "mlp": mlp}


def _parallel(dim, vdim, heads, kv, window, rot_dims, base, scaling, scale, width, blocks, conv, mlp):
    rot = {"dims": rot_dims, "base": base, **({"scaling": scaling} if scaling else {})}
    left = {"dim": dim, "vdim": vdim, "heads": heads, "kv_heads": kv, "scale": scale, "mask": {"size": window}, "rot": rot}
    return {"type": "parallel", "mixer": {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv}}, "mlp": mlp}


CONFIGS = {
    "mam_a": {"architecture": "Mamusun", "vocab": 300, "width": 64, "norm": {"eps": 1e-5}, "postln_alpha": 1.7, "layers": [
        _window(32, 32, 4, 2, 20, 0.2, DENSE(72)),
        _parallel(32, 16, 4, 2, 33, 16, 100.0, BANDS, 0.3, 48, 3, 4, _moe(8, 2, 24, 1.5)),
        _window(32, 32, 8, 2, 50, 0.3, None, kv_from=0),
        _keyvalue(16, 4, 2, 8, 200.0, YARN, 0.3, DENSE(40)),
        _window(32, 32, 4, 2, 9, 0.25, _moe(5, 3, 16, 2.0), kv_from=0)]},
    "mam_b": {"architecture": "Mamusun", "vocab": 200, "width": 96, "norm": {"eps": 1e-6}, "postln_alpha": 1.0, "layers": [
        _keyvalue(48, 3, 3, 48, 5000.0, None, 0.15, None),
        _parallel(16, 48, 3, 3, 70, 16, 1000.0, None, 0.25, 80, 1, 2, DENSE(104)),
        _window(16, 40, 6, 3, 130, 0.3, _moe(6, 6, 32, 0.8))]},
    "mam_c": {"architecture": "Mamusun", "vocab": 101, "width": 60, "norm": {"eps": 1e-5}, "postln_alpha": 2.2, "layers": [
        _parallel(12, 10, 3, 1, 9, 4, 50.0, {"factor": 3.0, "low": 2.0, "high": 5.0, "original": 40}, 0.35, 45, 5, 1, _moe(5, 1, 14, 2.0)),
        _window(12, 10, 3, 1, 7, 0.3, DENSE(50)),
        _keyvalue(10, 3, 1, 6, 30.0, {"factor": 2.0, "original": 30, "fast": 4.0, "slow": 1.0}, 0.3, DENSE(26)),
        _window(12, 10, 2, 1, 12, 0.3, None, kv_from=1)]},
    "mam_d": {"architecture": "Mamusun", "vocab": 160, "width": 128, "norm": {"eps": 1e-6}, "postln_alpha": 1.3, "layers": [
        _parallel(64, 64, 4, 1, 100, 64, 10000.0, BANDS, 0.12, 128, 4, 3, DENSE(96)),
        _window(128, 128, 2, 1, 65, 0.1, _moe(4, 2, 40, 3.0)),
        _keyvalue(128, 2, 2, 32, 500.0, YARN, 0.1, DENSE(64)),
        _window(128, 128, 3, 1, 90, 0.09, None, kv_from=1)]},
}
SEEDS = {"mam_a": 3, "mam_b": 4, "mam_c": 5, "mam_d": 6}
TOL = {"float32": 3e-5, "bfloat16": 8e-2}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name])


def write_model(folder: str, cfg: dict, seed: int, scale_up: float = 8.0) -> str:
    """A model folder with random weights through the library's own random-weights mode, the matrices
    scaled up so that the mixers and the feed-forwards matter in the logits."""
    import torch

    import ember_cpp_b200 as E
    from ember_cpp_b200.weights import read_folder, write_file
    E.write_random_model(folder, E.config.config_from_dict(cfg), seed)
    tensors = {name: t.clone() for name, t in read_folder(folder).items()}     # (the file is mapped: copies, then rewrite)
    for name, t in tensors.items():
        if t.dim() == 2 and not name.endswith((".conv", ".ra.b", ".ri.b", ".router")):
            tensors[name] = (t.float() * (20.0 if name == "embed" else scale_up)).to(torch.bfloat16)
        elif name.endswith((".ra", ".ri")):
            tensors[name] = (t.float() * 4.0).to(torch.bfloat16)
        elif name.endswith(".lam"):        # decays from a token or two to hundreds
            tensors[name] = torch.linspace(-7.0, 0.0, t.numel()).to(torch.bfloat16)
    write_file(os.path.join(folder, "model.safetensors"), tensors, {"format": "pt"})
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    return folder


def ids(seed: int, vocab: int, n: int) -> list:
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def row_errors(got, ref) -> np.ndarray:
    """Per row: rms(delta - mean(delta)) / rms(ref - mean(ref))."""
    got, ref = np.atleast_2d(np.asarray(got, dtype=np.float64)), np.atleast_2d(np.asarray(ref, dtype=np.float64))
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    r = ref - ref.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean(-1))


def rows_agree(got, ref, dtype: str) -> bool:
    """`got` against the plain model's `ref` (lists of [rows, vocab] arrays).  In 32-bit every row is within TOL.  In
    bfloat16 a rounding can turn a near tie of the router's choice the other way, and the token then runs another expert
    than the plain model's: some rows may differ by more (at most one in eight), the typical row must not."""
    errors = np.concatenate([row_errors(g, r) for g, r in zip(got, ref)])
    if dtype == "float32":
        return bool(errors.max() < TOL[dtype])
    return bool((errors >= TOL[dtype]).mean() <= 0.125 and np.median(errors) < TOL[dtype] / 2)
