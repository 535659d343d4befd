"""Mamusun on the host side: configuration, spec, random weights, the cache a layer shares with the layers that read it,
the plain implementation's own mechanisms, and the step function, batching and generation loop over the CPU double of
the kernels, against the plain implementation."""
import json
import math

import numpy as np
import pytest

import ember_cpp_b200 as E
from ember_cpp_b200.config import ConfigError, MamusunConfig, config_from_dict
from ember_cpp_b200.parts import CacheNeed, DecoderModel
from ember_cpp_b200.parts.position import Rotary
from ember_cpp_b200.weights import read_folder

import mamusun_util as U
import plain_mamusun as P
from conftest import run_batch
from cpu_ops import CpuOps


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: U.write_model(str(tmp_path_factory.mktemp(name)), U.config(name), U.SEEDS[name]) for name in U.CONFIGS}


@pytest.fixture(scope="module")
def plains(folders):
    return {name: P.load_folder(folder) for name, folder in folders.items()}


def cpu_engine(folder, max_tokens=1024, dtype="float32"):
    return E.Engine.from_folder(folder, dtype=dtype, max_tokens=max_tokens, device="cpu", ops=CpuOps())


# ------------------------------------------------------------------------------ configuration
def test_the_architecture_is_registered_and_reads_its_own_keys():
    cfg = config_from_dict(U.config("mam_a"))
    assert isinstance(cfg, MamusunConfig) and "Mamusun" in E.config.architectures()
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.alpha, len(cfg.layers)) == (300, 64, 1e-5, 1.7, 5)
    assert config_from_dict(cfg.to_dict()) == cfg


@pytest.mark.parametrize("path, value, word", [
    (("width",), None, "width"), (("norm", "eps"), 0, "norm.eps"), (("postln_alpha",), None, "postln_alpha"),
    (("layers", 0, "type"), "serial", "type"), (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"), (("layers", 0, "mixer", "scale"), None, "scale"),
    (("layers", 1, "mixer", "left", "mask"), None, "mask.size"), (("layers", 1, "mixer", "left", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 34, "rot.dims"), (("layers", 1, "mixer", "left", "rot", "scaling", "low"), None, "scaling.low"),
    (("layers", 1, "mixer", "right", "blocks"), 5, "blocks"), (("layers", 1, "mixer", "right", "conv"), 0, "right.conv"),
    (("layers", 1, "mixer", "left"), None, "left"), (("layers", 1, "mlp", "router", "top"), 9, "top"),
    (("layers", 1, "mlp", "expert", "limit"), -1.0, "expert.limit"), (("layers", 0, "mlp", "kind"), "gated", "kind"),
    (("layers", 0, "mlp", "ff"), 1.5, "ff"), (("layers", 2, "mixer", "kv_from"), 2, "kv_from"), (("layers", 2, "mixer", "kv_from"), 1, "kv_from"),
    (("layers", 4, "mixer", "kv_from"), 2, "kv_from"), (("layers", 2, "mixer", "dim"), 16, "dim"), (("layers", 3, "mixer", "vdim"), 8, "vdim"),
    (("layers", 3, "mixer", "rot", "scaling", "fast"), 0, "scaling.fast"), (("layers", 3, "mixer", "rot", "base"), None, "rot.base")])
def test_a_bad_value_is_refused_by_its_key(path, value, word):
    d = U.config("mam_a")
    at = d
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        config_from_dict(d)


def test_the_spec_names_the_designs_parts_and_tensors(folders):
    spec = E.config.get_architecture("Mamusun").build_spec(config_from_dict(U.config("mam_a")))
    assert [l.mixer.kind for l in spec.layers] == ["causal_attention", "parallel", "causal_attention", "causal_attention", "causal_attention"]
    assert [a.cache_of for a in spec.schedule] == [None, None, 0, None, 0]
    assert {l.block for l in spec.layers} == {"post_norm"} and spec.layers[2].ffn is None and spec.layers[2].norm2 is None
    assert [l.addons[0].params["layers"] for l in spec.layers] == [1, 2, 3, 4, 5]
    model = DecoderModel(spec)
    needs = model.application_needs()
    # layer 0's cache must hold what its readers see: the wider of the three windows
    assert needs[0][0] == CacheNeed("window", 2, 32, 50, 0, 0) and needs[2][0] is None and needs[4][0] is None
    assert needs[1][0] == CacheNeed("window", 2, 32, 33, 0, 16) and needs[3][0] == CacheNeed("full", 2, 16, 0, 0, 0)
    assert sorted(needs[1][1]) == ["right.S", "right.conv"] and needs[1][1]["right.conv"].shape == (3, 48)
    t = read_folder(folders["mam_a"])
    assert "l2.mix.k" not in t and "l2.mix.k.norm" not in t and "l2.mix.v" not in t and t["l2.mix.q"].shape == (256, 64)
    assert "l3.mix.v" not in t and t["l3.mix.k.b"].shape == (32,) and t["l3.mix.sink"].shape == (4,) and t["l3.mix.k.norm"].shape == (32,)
    assert t["l0.mix.q.norm"].shape == (32,) and t["l1.mix.right.ra"].shape == (3, 16, 16) and t["l1.mix.right.ri.b"].shape == (3, 16)
    assert t["l1.mlp.router.b"].shape == (8,) and t["l0.mlp.act"].shape == (4,) and t["l4.dwa"].shape == (6,)
    assert "l2.norm2" not in t and "l1.mix.left.q.norm" not in t and "l0.mix.q.b" not in t


def test_cache_needs_join():
    w = lambda n, **m: CacheNeed("window", 2, 16, n, **m)  # noqa: E731
    assert w(20).joined(w(50)) == w(50) and w(50).joined(w(20)) == w(50) and w(9, keep_first=3).joined(w(5)) == w(9, keep_first=3)
    assert w(20).joined(CacheNeed("full", 2, 16)).kind == "full" and CacheNeed("full", 2, 16).joined(CacheNeed("full", 2, 16)).kind == "full"
    assert CacheNeed("chunk", 2, 16, 30).joined(w(20)) == CacheNeed("full", 2, 16)
    with pytest.raises(ValueError, match="read as"):
        w(20).joined(CacheNeed("window", 1, 16, 20))


@pytest.mark.parametrize("dims, base, scaling", [(16, 100.0, U.BANDS), (64, 10000.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 300}),
                                                 (8, 50.0, {"factor": 3.0, "low": 2.0, "high": 5.0, "original": 40}), (16, 100.0, None)])
def test_frequencies_scaled_by_bands(dims, base, scaling):
    rot = Rotary("", dims=dims, base=base, interleaved=True, scaling=None if scaling is None else {"kind": "bands", **scaling})
    want = P.banded_freqs(dims, {"base": base, "scaling": scaling})
    assert np.allclose(rot.freqs_host, want, rtol=1e-14) and rot.magnitude == 1.0
    if scaling:
        plain = np.array(P.base_freqs(dims, base))
        ratio = want / plain          # some stay, some are slowed by the whole factor, none by more
        assert np.isclose(ratio.max(), 1.0) and np.isclose(ratio.min(), 1 / scaling["factor"]) and (np.diff(ratio) <= 1e-12).all()


@pytest.mark.parametrize("dims, base, scaling", [(8, 200.0, U.YARN), (48, 5000.0, {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0})])
def test_frequencies_scaled_by_a_ramp(dims, base, scaling):
    rot = Rotary("", dims=dims, base=base, scaling=scaling)
    want, mag = P.ramp_freqs(dims, {"base": base, "scaling": scaling})
    assert np.allclose(rot.freqs_host, want, rtol=1e-14) and math.isclose(rot.magnitude, mag) and mag > 1.0


def test_the_plain_models_window_sink_and_routing():
    k = np.zeros((6, 1, 2))
    v = np.arange(6.0)[:, None, None] * np.ones((1, 1, 2))
    o = P.attend(np.zeros((6, 1, 2)), k, v, 1.0, window=2)
    assert np.allclose(o[:, 0, 0], [0, 0.5, 1.5, 2.5, 3.5, 4.5])                   # the token itself and the one before
    o = P.attend(np.zeros((6, 1, 2)), k, v, 1.0, sinks=np.array([math.log(2.0)]))
    assert np.allclose(o[:, 0, 0], [np.arange(i + 1).sum() / (i + 3) for i in range(6)])
    chosen, weights = P.route(np.array([[0.0, 3.0, 1.0, 3.0 + math.log(3.0)]]), 2)
    assert chosen.tolist() == [[3, 1]] and np.allclose(weights, [[0.75, 0.25]])
    z = np.array([[1.0, -2.0]])
    rms = lambda t: t / np.sqrt((t * t).mean())  # noqa: E731
    assert np.allclose(P.poly_norm(z, (1.0, 0.5, 2.0, 0.25), 0.0), rms(z) + 0.5 * rms(z ** 2) + 2.0 * rms(z ** 3) + 0.25)
    u, one = np.array([[1.0], [0.0], [0.0]]), np.ones((3, 1))
    S = P.gated_recurrence(u, one, one, np.array([0.0]))                          # log a = -8 ln 2
    assert np.allclose(S[:, 0], np.sqrt(1 - 2.0 ** -16) * 2.0 ** (-8.0 * np.arange(3)))


# ------------------------------------------------------------------------------ the step function over the double
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_prompts_decoding_portions_and_batches_equal_the_plain_model(folders, plains, name):
    eng, (cfg, W) = cpu_engine(folders[name]), plains[name]
    seqs = [U.ids(10 + i, cfg["vocab"], n) for i, n in enumerate((75, 1, 23, 2))]
    refs = [P.forward(cfg, W, s) for s in seqs]
    for prompts in ([len(s) for s in seqs], [40, 1, 1, 1]):
        got, _ = run_batch(eng, seqs, prompts)
        assert U.rows_agree(got, refs, "float32")
    slot, at, rows = eng.open(), 0, []
    for n in (2, 5, 30, 3, 2, 33):                                                 # portions of one sequence
        rows.append(eng.step([(slot, seqs[0][at:at + n], list(range(n)))]).numpy())
        at += n
    eng.close(slot)
    assert U.rows_agree([np.concatenate(rows)], refs[:1], "float32")
    eng.cache.check()
    assert eng.cache.slots.held == 0 and all(g.pages.held == 0 for g in eng.cache.groups)


def test_the_stream_after_every_layer(folders, plains):
    cfg, W = plains["mam_a"]
    eng = cpu_engine(folders["mam_a"])
    seq = U.ids(77, cfg["vocab"], 31)
    _, streams = P.forward(cfg, W, seq, per_layer=True)
    seen = []
    for block in eng.model.blocks:
        inner = block.forward
        block.forward = lambda ctx, x, app, inner=inner: (lambda y: seen.append(y.clone()) or y)(inner(ctx, x, app))
    slot = eng.open()
    eng.step([(slot, seq, [30])])
    assert len(seen) == len(streams) == 5
    for got, want in zip(seen, streams):
        assert np.abs(got.numpy() - want).max() < 1e-4 * np.abs(want).max()


def test_every_mechanism_shows_in_the_logits(folders, plains):
    """The comparisons above see a mechanism only if it matters: each change moves the plain model's logits by far more than
    the tolerance."""
    cfg, W = plains["mam_a"]
    seq = U.ids(5, cfg["vocab"], 70)
    ref = P.forward(cfg, W, seq)

    def moved(c, w):
        return float(np.median(U.row_errors(P.forward(c, w, seq), ref)[55:]))
    changes = []
    for path, value in ((("postln_alpha",), 1.5), (("layers", 0, "mixer", "mask", "size"), 19), (("layers", 2, "mixer", "mask", "size"), 49),
                        (("layers", 4, "mixer", "mask", "size"), 10), (("layers", 1, "mixer", "left", "mask", "size"), 32),
                        (("layers", 1, "mixer", "left", "rot", "scaling", "factor"), 2.0), (("layers", 3, "mixer", "rot", "scaling", "factor"), 2.0),
                        (("layers", 1, "mlp", "expert", "limit"), 0.5)):
        c = U.config("mam_a")
        at = c
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        changes.append(moved(c, W))
    for name in ("l3.mix.sink", "l1.mix.right.lam", "l1.mix.right.conv.b", "l1.mlp.router.b", "l2.dwa", "l1.mix.left.out", "l0.mlp.act"):
        changes.append(moved(U.config("mam_a"), {**W, name: W[name] * 0.5}))
    assert min(changes) > 10 * U.TOL["float32"], changes


def test_state_rows_and_pages_are_used_again(folders, plains):
    """A small cache: the next batch gets the slots, state rows and pages that the batch before it left
    (filled with NaN in between); a sequence that begins must not read them."""
    eng, (cfg, W) = cpu_engine(folders["mam_a"], max_tokens=256), plains["mam_a"]
    for round_ in range(2):
        seqs = [U.ids(200 * round_ + i, 300, n) for i, n in enumerate((100, 30))]
        got, slots = run_batch(eng, seqs, [3, 25])
        assert sorted(slots) == [0, 1]
        assert U.rows_agree(got, [P.forward(cfg, W, s) for s in seqs], "float32")
        for g in eng.cache.groups:
            for t in g.k + g.v:
                t.fill_(float("nan"))
        for state in eng.cache.states:
            for t in (state or {}).values():
                t.fill_(float("nan"))


def test_greedy_generation_through_the_session(folders, plains):
    for name in ("mam_a", "mam_c"):
        cfg, W = plains[name]
        session = E.Session(folders[name], None, max_batch_size=3, dtype="float32", max_tokens=1024, ops=CpuOps(), device="cpu")
        prompts = [U.ids(50 + i, cfg["vocab"], n) for i, n in enumerate((5, 23, 1, 9))]
        assert session.generate_batch(prompts, steps=6, temperature=0.0) == [P.generate(cfg, W, p, 6) for p in prompts]


def test_a_sum_over_depth_behind_an_arrangement_that_adds_into_the_stream():
    """`depth_average` behind a pre-norm layer: the results in front must be copies, not the stream that later layers add to."""
    import torch
    from ember_cpp_b200.parts import Application, LayerSpec, ModelSpec, PartSpec
    d = 8
    norm = lambda n: PartSpec("rmsnorm", n, {"width": d, "eps": 1e-6, "weight": ""})  # noqa: E731
    mixer = lambda i: PartSpec("rglru", f"m{i}.", {"width": d, "inner": 6, "blocks": 2, "conv": 2, "factor": 8.0})  # noqa: E731
    layers = tuple(LayerSpec("pre_norm", norm(f"n{i}"), mixer(i), None, None, addons=(PartSpec("depth_average", f"d{i}.", {"layers": i + 1}),))
                   for i in range(3))
    spec = ModelSpec(width=d, vocab_size=11, token_table="t", position=PartSpec("none"), layers=layers,
                     schedule=tuple(Application(i) for i in range(3)), final_norm=norm("f"), head="h")
    gen = torch.Generator().manual_seed(1)
    tensors = {w.name: torch.randn(w.shape, generator=gen) * 0.5 for w in DecoderModel(spec).weight_specs()}
    eng = E.Engine.from_spec(spec, tensors, dtype="float32", max_tokens=64, device="cpu", ops=CpuOps())
    ids = [3, 1, 4, 1, 5]
    got = eng.step([(eng.open(), ids, list(range(5)))]).numpy()
    W = {k: t.double().numpy() for k, t in tensors.items()}
    x = W["t"][ids]
    results = [x]
    for i in range(3):
        x = x + P.right_mixer(P.norm_plain(x, W[f"n{i}"], 1e-6), W, f"m{i}.")
        results.append(x)
        x = sum(c * r for c, r in zip(W[f"d{i}.dwa"], results))
    want = P.norm_plain(x, W["f"], 1e-6) @ W["h"].T
    assert np.abs(got - want).max() < 1e-4 * np.abs(want).max()


def test_the_command_line_writes_a_random_model_of_this_design(tmp_path):
    from ember_cpp_b200 import cli
    cfg_file = tmp_path / "cfg.json"
    cfg_file.write_text(json.dumps(U.config("mam_b")))
    out = tmp_path / "model"
    assert cli.main([str(out), "-", "1", "random-weights", "--config", str(cfg_file), "--seed", "5"]) == 0
    cfg = E.load_config(str(out))
    assert isinstance(cfg, MamusunConfig) and cfg.width == 96
