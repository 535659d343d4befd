"""Podenex on the host side: configuration, spec, random weights, distance buckets, and the step function, batching and
generation loop over the CPU double of the kernels, against the plain implementation."""
import json
import math

import numpy as np
import pytest
import torch

import ember_cpp_b200 as E
from ember_cpp_b200.config import ConfigError, PodenexConfig, config_from_dict
from ember_cpp_b200.parts import CacheNeed, DecoderModel
from ember_cpp_b200.parts.position import distance_buckets
from ember_cpp_b200.weights import read_folder

import plain_podenex as P
import podenex_util as U
from conftest import run_batch
from cpu_ops import CpuOps


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: U.write_model(str(tmp_path_factory.mktemp(name)), U.config(name), U.SEEDS[name]) for name in U.CONFIGS}


@pytest.fixture(scope="module")
def plains(folders):
    return {name: P.load_folder(folder) for name, folder in folders.items()}


def cpu_engine(folder, max_tokens=1024):
    return E.Engine.from_folder(folder, dtype="float32", max_tokens=max_tokens, device="cpu", ops=CpuOps())


# ------------------------------------------------------------------------------ configuration
def test_the_architecture_is_registered_and_reads_its_own_keys():
    cfg = config_from_dict(U.config("pod_a"))
    assert isinstance(cfg, PodenexConfig) and "Podenex" in E.config.architectures()
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.side_dim, len(cfg.layers)) == (300, 64, 1e-5, 8, 4)
    assert config_from_dict(cfg.to_dict()) == cfg
    assert config_from_dict(U.config("pod_b")).side_dim == 0


@pytest.mark.parametrize("path, value, word", [
    (("width",), None, "width"), (("vocab",), 0, "vocab"), (("norm", "eps"), 0, "norm.eps"), (("layers", 0, "type"), "gla", "type"),
    (("token_side", "dim"), 0, "token_side.dim"), (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"), (("layers", 0, "mixer", "conv"), None, "conv"),
    (("layers", 0, "mixer", "bias_max"), 0, "bias_max"), (("layers", 0, "mixer", "bias_rows"), 1, "bias_rows"),
    (("layers", 0, "mixer", "v_mix"), "yes", "v_mix"), (("layers", 2, "mixer", "vdim"), 24, "v_mix"),
    (("layers", 2, "mixer", "scale"), 0, "scale"), (("layers", 1, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 10, "rot.dims"), (("layers", 1, "mixer", "q_rank"), None, "q_rank"),
    (("layers", 1, "mixer", "v_mix"), True, "v_mix"), (("layers", 1, "mixer", "mask"), None, "mask.size"),
    (("layers", 0, "mlp", "kind"), "dense", "kind"), (("layers", 0, "mlp", "router", "top"), 9, "top"),
    (("layers", 0, "mlp", "router", "groups", "count"), 3, "groups"), (("layers", 0, "mlp", "router", "groups", "keep"), 5, "groups"),
    (("layers", 0, "mlp", "shared", "ff"), None, "shared.ff"), (("layers", 0, "mlp", "expert", "ff"), -1, "expert.ff")])
def test_a_bad_value_is_refused_by_its_key(path, value, word):
    d = U.config("pod_a")
    at = d
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        config_from_dict(d)


def test_the_spec_names_the_designs_tensors_and_states_and_caches(folders):
    spec = E.config.get_architecture("Podenex").build_spec(config_from_dict(U.config("pod_a")))
    assert [l.mixer.kind for l in spec.layers] == ["causal_attention", "latent_attention", "causal_attention", "causal_attention"]
    assert [l.mixer.params.get("value_mix") for l in spec.layers] == ["keep", None, "vmix", None]
    assert spec.layers[3].ffn is None and spec.layers[3].norm2 is None and [len(l.addons) for l in spec.layers] == [1] * 4
    needs = DecoderModel(spec).application_needs()
    assert [n for n, _ in needs] == [CacheNeed("chunk", 2, 16, 40, 0, 32), CacheNeed("window", 1, 32, 33, 0, 8),
                                     CacheNeed("window", 4, 32, 20, 0, 16), CacheNeed("chunk", 2, 32, 90, 0, 0)]
    assert needs[0][1]["conv"].shape == (3, 4 * 16 + 2 * 16 + 2 * 32) and needs[1][1] is None and needs[2][1] is None
    t = read_folder(folders["pod_a"])
    assert t["l0.norm1"].shape == (64,) and "l0.norm1.bias" not in t and "l3.norm2" not in t and t["side.embed"].shape == (300, 32)
    assert t["l0.mix.q.conv"].shape == (64, 4) and t["l0.mix.rel"].shape == (12, 4) and t["l0.mix.g"].shape == (4, 64)
    assert t["l2.mix.q.b"].shape == (256,) and t["l2.mix.o.b"].shape == (64,) and t["l2.mix.k.norm"].shape == (32,)
    assert t["l2.mix.vmix"].shape == () and "l0.mix.vmix" not in t and "l3.mix.vmix" not in t
    assert t["l1.mix.g"].shape == (72, 64) and t["l1.mix.dkv.norm"].shape == (32,) and t["l1.mix.dkv"].shape == (40, 64)
    assert t["l0.mlp.e7.up"].shape == (24, 64) and "l0.mlp.e0.gate" not in t and t["l0.mlp.shared.down"].shape == (64, 40)
    # the first mixing layer's number is there in some checkpoints and read by nothing
    more = dict(t, **{"l0.mix.vmix": torch.tensor(0.3, dtype=torch.bfloat16)})
    E.Engine.from_spec(spec, more, dtype="float32", max_tokens=128, device="cpu", ops=CpuOps())


# ------------------------------------------------------------------------------ distances in buckets
@pytest.mark.parametrize("rows, far", [(2, 5), (4, 3), (8, 64), (12, 25), (16, 128), (16, 27.5), (32, 128), (32, 4096), (7, 40), (64, 33)])
def test_distance_buckets_follow_their_equation(rows, far):
    got = distance_buckets(rows, far)
    want = [P.distance_bucket(n, rows, far) for n in range(len(got) + 50)]
    assert got == want[:len(got)] and set(want[len(got):]) == {rows - 1}
    assert got[-1] == rows - 1 and (len(got) < 2 or got[-2] < rows - 1)


def test_a_distance_on_a_buckets_border_begins_that_bucket():
    # 8 single distances, then 8 buckets that grow by sqrt(2) up to 128: every second border is a whole distance
    got = distance_buckets(16, 128)
    assert [got[n] for n in (7, 8, 15, 16, 31, 32, 63, 64)] == [7, 8, 9, 10, 11, 12, 13, 14]
    assert len(got) - 1 == math.ceil(8 * 2 ** 3.5)
    with pytest.raises(ValueError, match="buckets"):
        distance_buckets(16, 8)
    with pytest.raises(ValueError, match="buckets"):
        distance_buckets(1, 8)


# ------------------------------------------------------------------------------ the plain model's own mechanisms
def test_the_router_of_the_plain_model_keeps_to_the_groups_of_the_largest_scores():
    z = np.array([[3.0, -9, 2.9, 2.8, 1.0, 1.1, 0.0, 2.0]])
    s = np.exp(z[0]) / np.exp(z[0]).sum()
    # groups of two; their largest: 3.0, 2.9, 1.1, 2.0: the sum of two would have put the second in front of the first
    chosen, weights = P.route(z, {"top": 2, "groups": {"count": 4, "keep": 1}})
    assert chosen[0].tolist() == [0, 1] and np.allclose(weights[0], s[[0, 1]])
    chosen, weights = P.route(z, {"top": 3, "groups": {"count": 4, "keep": 2}})
    assert chosen[0].tolist() == [0, 2, 3] and np.allclose(weights[0], s[[0, 2, 3]]) and weights.sum() < 1
    assert P.route(z, {"top": 3})[0][0].tolist() == [0, 2, 3]


def test_sinks_windows_and_chunks_of_the_plain_model():
    assert np.allclose(P.softmax_rows(np.zeros((1, 1)), np.ones((1, 1), bool), sink=0.0), 0.5)
    assert P.window_sight(5, 2).sum(1).tolist() == [1, 2, 2, 2, 2] and P.chunk_sight(5, 2).sum(1).tolist() == [1, 2, 1, 2, 1]
    table = np.arange(8.0)[:, None] * np.ones((1, 2))
    b = P.distance_bias(table, 20, 30)
    assert b.shape == (2, 30, 30) and b[0, 10, 10] == 0 and b[1, 10, 7] == 3 and b[0, 29, 0] == 7 and b[0, 3, 9] == 0


@pytest.mark.parametrize("name, tensor, layer", [
    ("pod_a", "l0.mix.rel", 0), ("pod_a", "l0.mix.g", 0), ("pod_a", "l2.mix.vmix", 2), ("pod_a", "l1.mix.g", 1), ("pod_b", "l3.mix.vmix", 3),
    ("pod_a", "l0.mix.v.conv", 0), ("pod_a", "l2.mix.o.b", 2), ("pod_a", "l2.mix.k.norm", 2), ("pod_a", "l1.side.norm", 1),
    ("pod_a", "l0.mlp.router", 0), ("pod_a", "l0.mlp.shared.up", 0), ("pod_c", "l3.mix.vmix", 3), ("pod_d", "l2.mix.dkv.norm", 2)])
def test_every_mechanism_moves_the_logits_by_far_more_than_the_tolerance(plains, name, tensor, layer):
    cfg, W = plains[name]
    seq = U.ids(3, cfg["vocab"], 60)
    other = dict(W)
    rng = np.random.default_rng(1)
    other[tensor] = W[tensor] + (0.3 if W[tensor].ndim == 0 else rng.standard_normal(W[tensor].shape) * max(W[tensor].std(), 0.2))
    err = U.row_errors(P.forward(cfg, other, seq), P.forward(cfg, W, seq))
    assert np.median(err) > 20 * U.TOL["float32"], np.median(err)


# ------------------------------------------------------------------------------ the step function over the double
@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_prompts_decoding_portions_and_batches_equal_the_plain_model(folders, plains, name):
    eng, (cfg, W) = cpu_engine(folders[name]), plains[name]
    seqs = [U.ids(10 + i, cfg["vocab"], n) for i, n in enumerate((100, 1, 23, 2))]
    refs = [P.forward(cfg, W, s) for s in seqs]
    for prompts in ([len(s) for s in seqs], [60, 1, 1, 1]):
        got, _ = run_batch(eng, seqs, prompts)
        assert max(U.row_error(g, r) for g, r in zip(got, refs)) < U.TOL["float32"]
    slot, at, rows = eng.open(), 0, []
    for n in (2, 5, 30, 3, 2, 33, 25):                                             # portions of one sequence
        rows.append(eng.step([(slot, seqs[0][at:at + n], list(range(n)))]).numpy())
        at += n
    eng.close(slot)
    assert U.row_error(np.concatenate(rows), refs[0]) < U.TOL["float32"]
    eng.cache.check()
    assert eng.cache.slots.held == 0 and all(g.pages.held == 0 for g in eng.cache.groups)


@pytest.mark.parametrize("name", ["pod_a", "pod_c"])
def test_the_stream_after_every_layer(folders, plains, name):
    cfg, W = plains[name]
    eng = cpu_engine(folders[name])
    seq = U.ids(77, cfg["vocab"], 31)
    _, streams = P.forward(cfg, W, seq, per_layer=True)
    seen = []
    for block in eng.model.blocks:
        inner = block.forward
        # (a copy: the next layer may add into the stream in place)
        block.forward = lambda ctx, x, app, inner=inner: (lambda y: seen.append(y.clone()) or y)(inner(ctx, x, app))
    slot = eng.open()
    eng.step([(slot, seq, [30])])
    assert len(seen) == len(streams)
    for got, want in zip(seen, streams):
        assert np.abs(got.numpy() - want).max() < 1e-4 * np.abs(want).max()


def test_state_rows_and_pages_are_used_again(folders, plains):
    """A small cache: the next batch gets the slots, state rows and pages that the batch before it left
    (filled with NaN in between); a sequence that begins must not read them."""
    eng, (cfg, W) = cpu_engine(folders["pod_a"], max_tokens=256), plains["pod_a"]
    for round_ in range(2):
        seqs = [U.ids(200 * round_ + i, 300, n) for i, n in enumerate((100, 30))]
        got, slots = run_batch(eng, seqs, [3, 25])
        assert sorted(slots) == [0, 1]
        assert max(U.row_error(g, P.forward(cfg, W, s)) for g, s in zip(got, seqs)) < U.TOL["float32"]
        for g in eng.cache.groups:
            for t in g.k + g.v:
                t.fill_(float("nan"))
        for state in eng.cache.states:
            for t in (state or {}).values():
                t.fill_(float("nan"))


def test_windows_and_chunks_hold_few_pages_of_a_long_sequence(folders):
    eng = cpu_engine(folders["pod_a"], max_tokens=512)
    slot = eng.open()
    eng.step([(slot, U.ids(1, 300, 130), [])])
    eng.step([(slot, U.ids(2, 300, 1), [0])])
    assert [[p >= 0 for p in g.held[slot]] for g in eng.cache.groups] == [
        [False, True, True],        # 131 lies in the chunk from 120 on
        [False, True, True],        # a window of 33 reaches back to 99
        [False, True, True],        # of 20 to 112
        [False, True, True]]        # and the chunk of 90 begins at 90


def test_greedy_generation_through_the_session(folders, plains):
    for name in ("pod_a", "pod_c"):
        cfg, W = plains[name]
        session = E.Session(folders[name], None, max_batch_size=3, dtype="float32", max_tokens=1024, ops=CpuOps(), device="cpu")
        prompts = [U.ids(50 + i, cfg["vocab"], n) for i, n in enumerate((5, 23, 1, 9))]
        assert session.generate_batch(prompts, steps=6, temperature=0.0) == [P.generate(cfg, W, p, 6) for p in prompts]


def test_the_command_line_writes_a_random_model_of_this_design(tmp_path):
    from ember_cpp_b200 import cli
    cfg_file = tmp_path / "cfg.json"
    cfg_file.write_text(json.dumps(U.config("pod_b")))
    out = tmp_path / "model"
    assert cli.main([str(out), "-", "1", "random-weights", "--config", str(cfg_file), "--seed", "5"]) == 0
    cfg = E.load_config(str(out))
    assert isinstance(cfg, PodenexConfig) and cfg.width == 96 and read_folder(str(out))["l3.mix.rel"].shape == (32, 6)
