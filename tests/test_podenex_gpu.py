"""Podenex on the GPU: every mechanism's kernels against the plain implementation, then whole models through the
engine (prompts, token-by-token decoding, portions, unequal batches, slots, state rows and pages used again, long
decoding, graph replay), greedy generation through the session and the command line, and a trace replay."""
import math

import numpy as np
import pytest
import torch

import ember_cpp_b200 as E
from ember_cpp_b200.cache.sequence_cache import SequenceCache
from ember_cpp_b200.engine.plan import StepPlan, build_step
from ember_cpp_b200.parts import CacheNeed
from ember_cpp_b200.parts.position import Rotary, distance_buckets

import plain_podenex as P
import podenex_util as U
from conftest import run_batch

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def ops():
    from ember_cpp_b200.csrc.ops import CudaOps
    return CudaOps()


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: U.write_model(str(tmp_path_factory.mktemp(name)), U.config(name), U.SEEDS[name]) for name in U.CONFIGS}


@pytest.fixture(scope="module")
def plains(folders):
    return {name: P.load_folder(folder) for name, folder in folders.items()}


def rnd(seed, *shape, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def f64(t):
    return t.detach().double().cpu().numpy()


def close(got, want, tol):
    got, want = f64(got) if torch.is_tensor(got) else got, np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape
    assert np.abs(got - want).max() <= tol * max(np.abs(want).max(), 1e-9), np.abs(got - want).max() / np.abs(want).max()


# ------------------------------------------------------------------------------ norm, gates
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, width", [(3, 60), (700, 384), (5, 2051), (40, 4096)])
def test_layer_norm_with_a_gain_alone(ops, dtype, rows, width):
    x, w = rnd(1, rows, width, scale=3.0) + 5.0, rnd(2, width)
    got = ops.layernorm(x.cuda(), w.cuda(), None, 1e-5, DT[dtype])
    close(got, P.layer_norm(f64(x), f64(w), 1e-5), 1e-5 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("proj_dtype", DTYPES)
@pytest.mark.parametrize("heads, vd, span, col", [(4, 32, 32, 8), (3, 10, 10, 5), (6, 24, 1, 16), (5, 7, 1, 3), (2, 48, 6, 4)])
def test_output_gates_a_value_and_a_head(ops, dtype, proj_dtype, heads, vd, span, col):
    if dtype == "float32" and proj_dtype == "bfloat16":
        pytest.skip("a gate narrower than the rows it multiplies")
    T, n = 9, heads * vd
    a, proj = rnd(1, T, n).to(DT[dtype]), rnd(2, T, col + n // span + 4, scale=2.0).to(DT[proj_dtype])
    got = ops.gate_mul(a.cuda(), proj.cuda(), col, "sigmoid", span=span)
    close(got, f64(a) * np.repeat(P.sigmoid(f64(proj)[:, col:col + n // span]), span, axis=1), 1e-6 if dtype == "float32" else 8e-3)


# ------------------------------------------------------------------------------ attention in windows and chunks
class Feed:
    """Sequences fed step by step through a paged cache whose pages are taken in a scrambled order, with NaN in every page
    before: `step(plan, view, rows)` gets each step's rows and returns its output rows."""

    def __init__(self, ops, need, dtype):
        self.ops = ops
        self.cache = SequenceCache([(need, None)], [None], 4096, None, DT[dtype], "cuda")
        self.cache.groups[0].pages._free = np.random.default_rng(0).permutation(self.cache.n_pages).tolist()
        self.view = self.cache.views[0]
        self.view.k.fill_(float("nan"))
        self.view.v.fill_(float("nan"))

    def run(self, steps, data, step):
        cache, n_seq = self.cache, len(steps[0])
        slots = [cache.open() for _ in range(n_seq)]
        outs, at = [[] for _ in range(n_seq)], [0] * n_seq
        for news in steps:
            live = [(i, n) for i, n in enumerate(news) if n > 0]
            entries = [(slots[i], n) for i, n in live]
            tails = cache.reserve(entries)
            host = build_step([(s, [0] * n, []) for s, n in entries], cache.lengths, [cache.groups[0].table], cache.max_blocks, tails=tails)
            plan = StepPlan(host, torch.from_numpy(host.packed).cuda())
            if plan.has_tails:
                self.ops.clear_tails(cache.groups[0], plan.tails[0])
            out = step(plan, self.view, torch.cat([data[i][at[i]:at[i] + n] for i, n in live]).contiguous().cuda())
            cache.commit(entries)
            row = 0
            for i, n in live:
                outs[i].append(out[row:row + n])
                at[i] += n
                row += n
        cache.check()
        for s in slots:
            cache.close(s)
        return [torch.cat(o) for o in outs]


def attend(ops, dtype, shape, steps, data, scale, window=0, chunk=0, table=None, far=0.0, sink=None):
    heads, kv, hd, vd = shape
    need = CacheNeed("chunk" if chunk else "window", kv, hd, chunk or window, 0, 0 if vd == hd else vd)
    more = {}
    if table is not None:
        of = distance_buckets(table.shape[0], far)[:chunk or window]
        more["dist_bias"] = table[torch.tensor(of)].t().contiguous().cuda()
    if sink is not None:
        more["sinks"] = torch.full((heads,), sink, device="cuda")
    return Feed(ops, need, dtype).run(steps, [d.to(DT[dtype]) for d in data], lambda plan, view, rows: ops.attention(
        rows, view, plan, heads, kv, hd, scale, window, DT[dtype], store=True, keep_first=0, value_dim=vd, chunk=chunk, **more))


def plain_attend(qkv, shape, scale, window=0, chunk=0, table=None, far=0.0, sink=None):
    heads, kv, hd, vd = shape
    x = f64(qkv)
    n = x.shape[0]
    q, k = x[:, :heads * hd].reshape(n, heads, hd), x[:, heads * hd:(heads + kv) * hd].reshape(n, kv, hd)
    v = x[:, (heads + kv) * hd:].reshape(n, kv, vd)
    seen = P.chunk_sight(n, chunk) if chunk else P.window_sight(n, window)
    bias = None if table is None else P.distance_bias(f64(table), far, n)
    return P.attend(q, k, v, scale, seen, bias=bias, sink=sink).reshape(n, heads * vd)


SHAPES = [((8, 2, 64, 32), 44), ((4, 2, 96, 48), 100), ((2, 1, 128, 128), 130), ((4, 4, 32, 80), 64), ((6, 3, 24, 40), 33),
          ((3, 1, 12, 10), 9), ((4, 1, 64, 64), 128), ((2, 2, 128, 16), 65), ((3, 3, 64, 112), 20), ((16, 1, 16, 32), 70)]
STEPS = [[190, 1, 50], [2, 40, 1], [64, 0, 5]] + [[1, 1, 1]] * 35 + [[8, 0, 48]]       # prompts, portions, one token each
FED = [299, 76, 139]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape, size", SHAPES)
def test_attention_inside_chunks_with_a_bias_by_distance(ops, dtype, shape, size):
    heads, kv, hd, vd = shape
    data = [rnd(10 + i, n, (heads + kv) * hd + kv * vd).to(DT[dtype]).float() for i, n in enumerate(FED)]
    table, far, scale = rnd(3, 12, heads, scale=2.0), 0.4 * size + 7, 1.5 / math.sqrt(hd)
    got = attend(ops, dtype, shape, STEPS, data, scale, chunk=size, table=table, far=far)
    for g, d in zip(got, data):
        close(g, plain_attend(d, shape, scale, chunk=size, table=table, far=far), 3e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape, size", SHAPES + [((4, 2, 64, 32), 1)])
def test_attention_over_a_window_with_a_sink(ops, dtype, shape, size):
    heads, kv, hd, vd = shape
    data = [rnd(20 + i, n, (heads + kv) * hd + kv * vd).to(DT[dtype]).float() for i, n in enumerate(FED)]
    scale = 1.5 / math.sqrt(hd)
    got = attend(ops, dtype, shape, STEPS, data, scale, window=size, sink=0.0)
    for g, d in zip(got, data):
        close(g, plain_attend(d, shape, scale, window=size, sink=0.0), 3e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [True, False])
@pytest.mark.parametrize("kind, size", [("chunk", 64), ("chunk", 100), ("chunk", 20), ("window", 64), ("window", 65), ("window", 100), ("window", 20)])
def test_one_marked_key_is_seen_exactly_inside_its_chunk_or_window(ops, dtype, prompt, kind, size):
    """Among 300 keys of which one carries a marked value and a large score: exactly the queries whose chunk or window
    holds it see it; at chunk, window and page borders, in prompts and in decoded rows.  The others share a score of zero,
    the window's with a sink beside them."""
    shape, n = (2, 1, 32, 16), 300
    heads, kv, hd, vd = shape
    opts = {"chunk": size} if kind == "chunk" else {"window": size, "sink": 0.0}
    for marked in ((0, size * 2, size * 3 - 1, 128, 191) if prompt else (size * 3 - 1, 128)):
        qkv = torch.zeros(n, (heads + kv) * hd + kv * vd)
        qkv[:, :heads * hd] = 1.0
        qkv[marked, heads * hd:(heads + kv) * hd] = 1.0                  # its score is hd * scale, every other key's is 0
        qkv[marked, (heads + kv) * hd:] = 5.0
        if marked >= n:
            continue
        steps = [[n]] if prompt else [[max(marked - 3, 1)]] + [[1]] * (n - max(marked - 3, 1))
        got = f64(attend(ops, dtype, shape, steps, [qkv], 0.5, **opts)[0])
        p = np.arange(n)
        lo = p // size * size if kind == "chunk" else np.maximum(p - size + 1, 0)
        seen = (marked <= p) & (marked >= lo)
        assert (np.abs(got[~seen]) < 1e-6).all() and seen.any() and not seen.all()
        want = 5.0 * math.exp(16.0) / (math.exp(16.0) + (p - lo)[seen] + (kind == "window"))
        assert np.abs(got[seen] - want[:, None]).max() < (1e-4 if dtype == "float32" else 5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [True, False])
@pytest.mark.parametrize("hd, vd", [(64, 32), (32, 32), (12, 10)])
def test_the_bias_of_every_distance_alone_decides(ops, dtype, prompt, hd, vd):
    """Keys and queries of zero: the weights are the softmax of the biases, which lie far apart from bucket to bucket;
    distances far beyond the last bucket take its entry."""
    heads, kv, n, rows, far = 2, 1, 300, 16, 100
    qkv = torch.zeros(n, (heads + kv) * hd + kv * vd)
    qkv[:, (heads + kv) * hd:] = rnd(5, n, vd)
    table = rnd(6, rows, heads, scale=3.0)
    table[rows - 1] += 4.0                                   # the far keys count
    got = attend(ops, dtype, (heads, kv, hd, vd), [[n]] if prompt else [[200]] + [[1]] * 100, [qkv], 0.7, chunk=280, table=table, far=far)[0]
    qkv[:, (heads + kv) * hd:] = qkv[:, (heads + kv) * hd:].to(DT[dtype]).float()
    close(got, plain_attend(qkv, (heads, kv, hd, vd), 0.7, chunk=280, table=table, far=far), 3e-5 if dtype == "float32" else 1e-2)


def test_a_sink_of_score_zero_halves_a_lone_keys_weight(ops):
    qkv = torch.zeros(1, 2 * 16 + 8)
    qkv[0, 2 * 16:] = 4.0
    for dtype in DTYPES:
        got = attend(ops, dtype, (1, 1, 16, 8), [[1]], [qkv], 1.0, window=8, sink=0.0)[0]
        assert torch.allclose(got.float().cpu(), torch.full((1, 8), 2.0))


# ------------------------------------------------------------------------------ norms a head, values carried from the first layer
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("other_dtype", DTYPES)
@pytest.mark.parametrize("heads, kv, hd, vd", [(4, 2, 64, 32), (3, 3, 12, 10), (2, 1, 160, 96), (6, 2, 32, 48)])
def test_norms_a_head_and_blended_values_go_into_the_cache(ops, dtype, other_dtype, heads, kv, hd, vd):
    dt, eps, lam = DT[dtype], 1e-5, 0.375
    width, vw, k0 = (heads + kv) * hd + kv * vd, kv * vd, heads * hd
    news = [[70, 1, 3], [1, 1, 1], [2, 64, 5]]
    total = [sum(s[i] for s in news) for i in range(3)]
    # rows: the projection | columns no one reads | the other layer's values
    data = [rnd(i, n, width + 4 + vw) for i, n in enumerate(total)]
    qg, kg = rnd(7, hd, scale=0.3) + 1, rnd(8, hd, scale=0.3) + 1
    need = CacheNeed("window", kv, hd, 4096, 0, 0 if vd == hd else vd)
    feed = Feed(ops, need, dtype)
    slots_pages = []

    def step(plan, view, rows):
        proj, other = rows[:, :width + 4], rows[:, width + 4:].to(DT[other_dtype])
        out = ops.qkv_prepare(proj, plan, view, heads, kv, hd, vd, dt, store=True, norm="head", q_gain=qg.cuda(), k_gain=kg.cuda(),
                              eps=eps, mix=(other, lam))
        slots_pages.append(plan.pages[0].clone().cpu())
        return torch.cat([out[:, :k0].float(), rows[:, width + 4:].to(DT[other_dtype]).float()], 1)
    got = feed.run(news, data, step)
    pages = {i: slots_pages[-1][i] for i in range(3)}
    for i, d in enumerate(data):
        x = f64(d)
        q = P.rms_norm(x[:, :k0].reshape(-1, heads, hd), f64(qg), eps).reshape(-1, k0)
        close(got[i][:, :k0], q, 1e-5 if dtype == "float32" else 5e-3)
        p = torch.arange(total[i])
        at = pages[i][p // 64].long()
        k = feed.view.k[at.cuda(), :, (p % 64).cuda(), :].reshape(total[i], -1)
        v = feed.view.v[at.cuda(), :, (p % 64).cuda(), :].reshape(total[i], -1)
        close(k, P.rms_norm(x[:, k0:k0 + kv * hd].reshape(-1, kv, hd), f64(kg), eps).reshape(-1, kv * hd), 1e-5 if dtype == "float32" else 5e-3)
        close(v, P.mix_values(x[:, width - vw:width], f64(got[i][:, k0:]), lam), 1e-5 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv, hd, vd", [(4, 2, 64, 32), (3, 1, 12, 10)])
def test_keys_and_blended_values_alone(ops, dtype, heads, kv, hd, vd):
    """The queries stay where the convolution left them: only the pages are written."""
    dt = DT[dtype]
    width, vw, k0, n = (heads + kv) * hd + kv * vd, kv * vd, heads * hd, 80
    x, other = rnd(1, n, width).to(dt), rnd(2, n, vw)
    for lam in (None, 0.25):
        feed = Feed(ops, CacheNeed("chunk", kv, hd, 4096, 0, 0 if vd == hd else vd), dtype)
        pages = []

        def step(plan, view, rows):
            pages.append(plan.pages[0].clone())
            mix = {} if lam is None else {"mix": (other.cuda(), lam)}
            assert ops.qkv_prepare(rows, plan, view, heads, kv, hd, vd, dt, store=True, queries=False, **mix) is None
            return rows
        got = feed.run([[n]], [x], step)[0]
        assert torch.equal(got.cpu(), x)
        p = torch.arange(n)
        at = pages[0][0].cpu()[p // 64].long()
        k = feed.view.k[at.cuda(), :, (p % 64).cuda(), :].reshape(n, -1)
        v = feed.view.v[at.cuda(), :, (p % 64).cuda(), :].reshape(n, -1)
        assert torch.equal(k.cpu(), x[:, k0:k0 + kv * hd])
        own = f64(x[:, width - vw:])
        close(v, own if lam is None else P.mix_values(own, f64(other), lam), 1e-6 if dtype == "float32" else 5e-3)


# ------------------------------------------------------------------------------ attention over cached rows in a window
def latent(ops, dtype, heads, rank, rot, window, steps, data, q_rank, scale, gains, rotary):
    """`data`: rows of q_rank | rank | rot | others' columns | the heads' queries (already in the row's space)."""
    need = CacheNeed("window" if window else "full", 1, rank, window, 0, rot)
    down_w = q_rank + rank + rot + 5

    def step(plan, view, rows):
        c_q = ops.latent_rows(rows[:, :down_w].contiguous(), plan, q_rank, gains[0].cuda(), gains[1].cuda(), rank, rot, 1e-5, rotary, view, DT[dtype])
        q = rows[:, down_w:].to(DT[dtype]).contiguous()
        o = ops.latent_attention(q, view, plan, heads, rank, rot, scale, DT[dtype], window=window)
        return torch.cat([c_q.float(), o.float()], 1)
    return Feed(ops, need, dtype).run(steps, data, step)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("heads, q_rank, rank, rot, dims, window", [(4, 48, 96, 32, 32, 96), (3, 20, 32, 16, 8, 33), (2, 9, 14, 6, 4, 11),
                                                                    (16, 64, 512, 64, 64, 130), (20, 16, 64, 16, 16, 0), (2, 8, 32, 16, 16, 1)])
def test_windowed_attention_over_cached_rows(ops, dtype, interleaved, heads, q_rank, rank, rot, dims, window):
    base, scale, down_w = 700.0, 2.0 / math.sqrt(rank + rot), q_rank + rank + rot + 5
    rotary = Rotary("", dims=dims, base=base, interleaved=interleaved)
    rotary.load(None, type("R", (), {"device": "cuda"}))
    gains = rnd(1, q_rank, scale=0.2) + 1, rnd(2, rank, scale=0.2) + 1
    data = [rnd(10 + i, n, down_w + heads * (rank + rot)) for i, n in enumerate(FED)]
    for d in data:                                       # (what a bfloat16 query holds)
        d[:, down_w:] = d[:, down_w:].to(DT[dtype]).float()
    got = latent(ops, dtype, heads, rank, rot, window, STEPS, data, q_rank, scale, gains, rotary)
    for g, d in zip(got, data):
        x = f64(d)
        n = x.shape[0]
        close(g[:, :q_rank], P.rms_norm(x[:, :q_rank], f64(gains[0]), 1e-5), 1e-5 if dtype == "float32" else 5e-3)
        c = P.rms_norm(x[:, q_rank:q_rank + rank], f64(gains[1]), 1e-5)
        k_r = x[:, q_rank + rank:q_rank + rank + rot].copy()
        if interleaved:
            k_r = P.rotate_neighbours(k_r[:, None], np.arange(n), dims, base)[:, 0]
        else:
            order = np.arange(dims).reshape(2, dims // 2).T.reshape(-1)      # halves apart, as neighbours
            k_r[:, order] = P.rotate_neighbours(k_r[:, None, order], np.arange(n), dims, base)[:, 0]
        q = x[:, down_w:].reshape(n, heads, rank + rot)
        want = P.attend(q, np.concatenate([c, k_r], 1)[:, None], c[:, None], scale, P.window_sight(n, window or n))
        close(g[:, q_rank:], want.reshape(n, heads * rank), 5e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [True, False])
@pytest.mark.parametrize("window", [64, 65, 20])
def test_one_marked_row_is_seen_exactly_inside_the_window(ops, dtype, prompt, window):
    heads, q_rank, rank, rot, n = 2, 8, 32, 16, 300
    rotary = Rotary("", dims=rot, base=1e30)
    rotary.freqs = torch.zeros(rot // 2, device="cuda")
    gains = torch.ones(q_rank), torch.ones(rank)
    down_w = q_rank + rank + rot + 5
    for marked in ((0, 127, 128, 191, 200) if prompt else (127, 192)):
        x = torch.zeros(n, down_w + heads * (rank + rot))
        x[:, q_rank] = 1.0                                               # every row is a lone value in its first column ...
        x[marked, q_rank], x[marked, q_rank + 1] = 0.0, 1.0              # ... the marked one in its second
        x[marked, q_rank + rank] = 1.0
        q = torch.zeros(heads, rank + rot)
        q[:, rank] = 20.0                                                # and only its key part has a score
        x[:, down_w:] = q.reshape(-1)
        steps = [[n]] if prompt else [[marked - 3]] + [[1]] * (n - marked + 3)
        got = f64(latent(ops, dtype, heads, rank, rot, window, steps, [x], q_rank, 1.0, gains, rotary)[0])[:, q_rank:].reshape(n, heads, rank)
        p = np.arange(n)
        seen = (p >= marked) & (p - marked < window)
        assert (np.abs(got[~seen][:, :, 1]) < 1e-6).all()
        assert (got[seen][:, :, 1] > 0.99 * math.sqrt(rank)).all() and seen.sum() == min(window, n - marked)


# ------------------------------------------------------------------------------ the router, the experts
@pytest.mark.parametrize("experts, top, groups, keep", [(8, 2, 4, 2), (12, 4, 2, 1), (6, 6, 1, 1), (5, 1, 1, 1), (64, 8, 8, 3), (9, 3, 9, 4), (160, 6, 8, 3)])
def test_the_routers_choice_by_a_softmax_over_all(ops, experts, top, groups, keep):
    T = 300
    logits = rnd(1, T, experts + 3, scale=2.0)               # columns behind the router's own are not read
    logits[:, experts:] = 50.0
    chosen, weights = ops.moe_pick(logits.cuda(), torch.zeros(experts).cuda(), experts, top, groups, keep, 1.0, scores="softmax_all", group_top=1)
    conf = {"top": top, **({"groups": {"count": groups, "keep": keep}} if groups > 1 else {})}
    want_e, want_w = P.route(f64(logits[:, :experts]), conf)
    assert np.array_equal(chosen.cpu().numpy(), want_e)
    close(weights, want_w, 1e-5)


@pytest.mark.parametrize("scores, groups, keep, group_top", [("softmax_all", 4, 2, 1), ("sigmoid", 8, 3, 2), ("softmax", 1, 1, 2)])
@pytest.mark.parametrize("T, experts, top", [(1, 8, 2), (8, 32, 2), (64, 16, 6), (33, 160, 6), (5, 1024, 8)])
def test_choice_and_sort_in_one_launch_equal_the_two(ops, scores, groups, keep, group_top, T, experts, top):
    logits, corr = rnd(1, T, experts + 3, scale=2.0).cuda(), rnd(2, experts, scale=0.1).cuda()
    args = (corr, experts, top, groups, keep, 1.5, scores, group_top)
    if top > keep * (experts // groups):
        pytest.skip("the kept groups hold fewer experts")
    chosen, want = ops.moe_pick(logits, *args)
    weights, (pair_expert, offsets, order, *_) = ops.moe_pick_route(logits, *args)
    assert torch.equal(weights, want) and torch.equal(pair_expert.view(T, top), chosen)
    counts = torch.bincount(chosen.view(-1).long(), minlength=experts).cumsum(0)
    assert offsets[0] == 0 and torch.equal(offsets[1:].long(), counts) and sorted(order.tolist()) == list(range(T * top))
    assert torch.equal(chosen.view(-1)[order.long()], chosen.view(-1).sort().values)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, width, inner, experts, top", [(3, 64, 24, 6, 3), (70, 64, 24, 6, 3), (200, 96, 130, 4, 2), (40, 60, 14, 5, 2)])
def test_experts_without_a_gate_and_their_weighted_sum(ops, dtype, T, width, inner, experts, top):
    dt = DT[dtype]
    h = rnd(1, T, width).to(dt)
    up, down = rnd(2, experts, inner, width, scale=0.3).to(dt), rnd(3, experts, width, inner, scale=0.3).to(dt)
    logits, shared, x = rnd(4, T, experts, scale=2.0), rnd(5, T, width), rnd(6, T, width)
    chosen, weights = ops.moe_pick(logits.cuda(), torch.zeros(experts).cuda(), experts, top, 1, 1, 1.0, scores="softmax_all", group_top=1)
    routing = ops.moe_route(None, T, chosen, experts, top)
    y = ops.moe_down(ops.moe_up(h.cuda(), up.cuda(), routing, dt, "relu2"), down.cuda(), routing)
    got, rows = ops.moe_combine(x.cuda(), y, weights, shared.cuda(), None, experts, rows_dtype=dt)
    want = f64(x) + f64(shared)
    for t in range(T):
        for e, wt in zip(chosen[t].tolist(), f64(weights[t])):
            want[t] += wt * P.expert(f64(h[t:t + 1]), f64(up[e]), f64(down[e]))[0]
    close(got, want, 3e-5 if dtype == "float32" else 1e-2)
    assert torch.equal(rows, got.to(dt)) and torch.equal(ops.moe_combine(x.cuda(), y, weights, shared.cuda(), None, experts), got)


# ------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def engines(folders):
    return {(name, dtype): E.Engine.from_folder(folders[name], dtype=dtype, max_tokens=2048) for name in U.CONFIGS for dtype in DT}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_prompts_decoding_portions_and_batches_equal_the_plain_model(engines, plains, name, dtype):
    eng, (cfg, W) = engines[(name, dtype)], plains[name]
    seqs = [U.ids(10 + i, cfg["vocab"], n) for i, n in enumerate((200, 1, 40, 97, 2))]
    refs = [P.forward(cfg, W, s) for s in seqs]
    for prompts in ([len(s) for s in seqs], [150, 1, 1, 30, 1]):
        got, _ = run_batch(eng, seqs, prompts)
        assert U.rows_agree(got, refs, dtype)
    each_alone = [run_batch(eng, [s], [min(len(s), 33)])[0][0] for s in seqs]          # alone: no neighbour changes a row
    assert U.rows_agree(each_alone, refs, dtype)
    from_the_first = run_batch(eng, [seqs[2]], [1])[0][0]                              # one token at a time from the first
    assert U.rows_agree([from_the_first], [refs[2]], dtype)
    slot, at, rows = eng.open(), 0, []
    for n in (2, 5, 64, 3, 2, 30, 94):                                                 # portions of one sequence
        rows.append(eng.step([(slot, seqs[0][at:at + n], list(range(n)))]).cpu().numpy())
        at += n
    eng.close(slot)
    assert U.rows_agree([np.concatenate(rows)], [refs[0]], dtype)
    eng.ops.check()
    eng.cache.check()
    assert eng.cache.slots.held == 0 and all(g.pages.held == 0 for g in eng.cache.groups)


@pytest.mark.parametrize("name", ["pod_a", "pod_d"])
def test_the_stream_after_every_layer_in_32_bit(engines, plains, name):
    eng, (cfg, W) = engines[(name, "float32")], plains[name]
    seq = U.ids(77, cfg["vocab"], 50)
    _, streams = P.forward(cfg, W, seq, per_layer=True)
    seen = []
    forwards = [b.forward for b in eng.model.blocks]
    try:
        for block, inner in zip(eng.model.blocks, forwards):
            # (a copy: the next layer's products add into the stream in place)
            block.forward = lambda ctx, x, app, inner=inner: (lambda y: seen.append(y.clone()) or y)(inner(ctx, x, app))
        slot = eng.open()
        eng.step([(slot, seq, [49])])
        eng.close(slot)
    finally:
        for block, inner in zip(eng.model.blocks, forwards):
            block.forward = inner
    assert len(seen) == len(streams)
    for got, want in zip(seen, streams):
        assert np.abs(got.cpu().numpy() - want).max() < 1e-4 * np.abs(want).max()


@pytest.mark.parametrize("name", ["pod_a", "pod_b"])
def test_in_32_bit_a_row_does_not_depend_on_the_batch_or_the_cut(engines, plains, name):
    eng, vocab = engines[(name, "float32")], plains[name][0]["vocab"]
    seqs = [U.ids(70 + i, vocab, n) for i, n in enumerate((90, 31, 64))]
    together, _ = run_batch(eng, seqs, [60, 31, 1])
    for i, s in enumerate(seqs):
        alone, _ = run_batch(eng, [s], [len(s)])
        assert np.array_equal(alone[0], together[i])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_past_many_chunks_with_slots_used_again(folders, plains, dtype):
    """A small cache: sequences decoded through many chunks and windows hold few pages, and the next batch gets the
    slots, state rows and pages that the batch before it left (filled with NaN in between)."""
    eng, (cfg, W) = E.Engine.from_folder(folders["pod_a"], dtype=dtype, max_tokens=384), plains["pod_a"]
    for round_ in range(2):
        seqs = [U.ids(200 * round_ + i, 300, n) for i, n in enumerate((330, 90))]
        got, slots = run_batch(eng, seqs, [3, 70])
        assert sorted(slots) == [0, 1]
        assert U.rows_agree(got, [P.forward(cfg, W, s) for s in seqs], dtype)
        for g in eng.cache.groups:
            for t in g.k + g.v:
                t.fill_(float("nan"))
        for state in eng.cache.states:
            for t in (state or {}).values():
                t.fill_(float("nan"))
    assert max(g.pages.size for g in eng.cache.groups) == 6


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_and_portions_take_the_tensor_core_kernels(folders, plains, dtype):
    for name in ("pod_a", "pod_d"):
        eng, (cfg, W) = E.Engine.from_folder(folders[name], dtype=dtype, max_tokens=1024), plains[name]
        seq = U.ids(77, cfg["vocab"], 400)
        ref = P.forward(cfg, W, seq)
        got, _ = run_batch(eng, [seq], [399])
        assert U.rows_agree(got, [ref], dtype)
        slot, at, rows = eng.open(), 0, []
        for n in (100, 188, 112):
            rows.append(eng.step([(slot, seq[at:at + n], list(range(n)))]).cpu().numpy())
            at += n
        eng.close(slot)
        assert U.rows_agree([np.concatenate(rows)], [ref], dtype)


def test_graph_replay_equals_launch_by_launch(folders):
    seqs = [U.ids(300 + i, 300, n) for i, n in enumerate((40, 75, 9))]
    outs = []
    for graphs in (True, False):
        eng = E.Engine.from_folder(folders["pod_a"], dtype="float32", max_tokens=1024, cuda_graphs=graphs)
        assert eng.cuda_graphs == graphs
        outs.append(run_batch(eng, seqs, [20, 60, 1])[0])
    for a, b in zip(*outs):
        assert np.array_equal(a, b)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_session(folders, plains, dtype):
    for name in ("pod_a", "pod_b"):
        cfg, W = plains[name]
        session = E.Session(folders[name], None, max_batch_size=3, dtype=dtype, max_tokens=2048)
        prompts = [U.ids(50 + i, cfg["vocab"], n) for i, n in enumerate((5, 23, 1, 9))]
        got = session.generate_batch(prompts, steps=8, temperature=0.0)
        want = [P.generate(cfg, W, p, 8) for p in prompts]
        if dtype == "float32":
            assert got == want
        else:       # a near tie may fall the other way in bfloat16: a first token is the plain model's best or within a tenth of
            for p, g in zip(prompts, got):     # the logits' spread of it; and many of the tokens are the same
                row = P.forward(cfg, W, p)[-1]
                assert row[g[0]] >= row.max() - 0.1 * row.std()
            assert sum(a == b for g, w in zip(got, want) for a, b in zip(g, w)) >= 12


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_of_a_model_folder(folders, plains, tmp_path, dtype):
    """bin/trace_run picks the model by config.json: each request whole, then unequal requests together and decoded
    together, their slots given back at their ends."""
    from test_replay_gpu import Replay
    cfg, W = plains["pod_b"]
    vocab = cfg["vocab"]
    seqs = {f"q{i}": U.ids(400 + i, vocab, n) for i, n in enumerate((130, 1, 47))}
    refs = {k: P.forward(cfg, W, s) for k, s in seqs.items()}
    rp = Replay(folders["pod_b"], dtype, tmp_path, sum(len(s) for s in seqs.values()))
    for k, s in seqs.items():
        got = rp.step([(k + "w", s, list(range(len(s))))], end=[k + "w"]).reshape(len(s), vocab)
        assert U.rows_agree([got], [refs[k]], dtype)
    fed = {k: max(1, len(s) - 20) for k, s in seqs.items()}
    rows = {k: [] for k in seqs}
    out = rp.step([(k, s[:fed[k]], list(range(fed[k]))) for k, s in seqs.items()], end=[k for k, s in seqs.items() if fed[k] == len(s)])
    at = 0
    for k in seqs:
        rows[k].append(out.reshape(-1, vocab)[at:at + fed[k]])
        at += fed[k]
    while any(fed[k] < len(s) for k, s in seqs.items()):
        live = [k for k, s in seqs.items() if fed[k] < len(s)]
        out = rp.step([(k, [seqs[k][fed[k]]], [0]) for k in live], end=[k for k in live if fed[k] + 1 == len(seqs[k])]).reshape(-1, vocab)
        for r, k in enumerate(live):
            rows[k].append(out[r:r + 1])
            fed[k] += 1
    rp.close()
    assert U.rows_agree([np.concatenate(rows[k]) for k in seqs], [refs[k] for k in seqs], dtype)


def test_the_command_line_generates_greedily(folders, plains):
    """bin/ember picks the model by config.json: a prompt's greedy tokens in 32-bit."""
    import os
    import subprocess
    import sys
    cfg, W = plains["pod_a"]
    prompt = U.ids(900, cfg["vocab"], 7)
    cli = [sys.executable, os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "ember")]
    r = subprocess.run(cli + [folders["pod_a"], "-", "1", "prompt", " ".join(map(str, prompt)), "-mt", "5", "-t", "0", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == P.generate(cfg, W, prompt, 5)
