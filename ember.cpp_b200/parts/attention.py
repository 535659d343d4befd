"""Causal multi-head attention over the cache, with a fused q|k|v projection.

ember.cpp's GPT-2 block: `qkv = h W^T + b`, split into q | k | v by columns
(sizes [H*hd, KV*hd, KV*hd], graph_ir.cpp:733-735), write k and v at their positions, then for
each query the scaled scores over the keys up to its own position, softmax, weighted sum of the
values (graph_ir.cpp:2539-2620; cpu_attention.cpp:92-211), and the output projection whose result
is added to the residual stream (graph_ir.cpp:742, 754).  Query head h reads key/value head
h // (H / KV) (cpu_attention.cpp:127).  With `window` > 0 a query at position p sees positions
p-window+1 .. p (cpu_attention.cpp, swa_visible_ranges).  The scale is a parameter: the
architecture computes it (GPT-2: 1/sqrt(hd), optionally divided by layer+1).

Beyond GPT-2's shape, all as parameters: the first `keep_first` positions of a sequence stay
visible beside the window (query p sees key j <= p if p - j < window or j < keep_first; the cache
keeps their pages); values may have a row size of their own (`value_dim`); q, k and v may be
stored as three matrices (`qkv` a tuple of three names: they are laid end to end at load, so the
step still makes one product); tensor names may carry no `.weight` suffix (`suffix`).

Further options, each off by default and each a parameter (`parts/attention.py::CausalAttention`):
`qk_norm` = (name of q's gain, name of k's gain): q and k are each divided by their root mean square over
the whole projection, before they are cut into heads, and multiplied by a gain of that size; `value_norm`:
every value head is divided by its own root mean square before it is cached; `q_temp` = (coef, every): q at
position p is multiplied by 1 + coef * ln(floor((p + 1) / every) + 1); `distance_slope_base` = b: the score of
key j for query i of head h loses 2^(-b (h + 1) / heads) * (i - j); `sink`: the name of one learned number per
head whose exponential is added to the softmax's denominator (it has no key and no value); `gate`: the name of a
matrix W_g, the heads laid end to end are multiplied by sigmoid(W_g h) before the output projection.  With a norm
on q or k or v, or a gate, the projection q | k | v (| g) is left in float32 (the norms read it unrounded) and
the normed rows are rounded to the compute type once.

And, again each a parameter: `qkv_bias` = suffix: q, k and v (stored as three matrices) have biases of that
suffix, added in the projection, and the output projection has none; `conv` = (taps, suffix): a short causal
convolution over time on every channel of q, k and v (a filter [channels, taps] a tensor, the last tap on the
current token, zeros before the sequence's start, no bias, no activation) directly after the projection; the
last taps - 1 projected rows of a sequence are its state ("conv"); `rotary` = (dims, base, interleaved): the
mixer rotates the first `dims` dimensions of every q and k head itself, neighbours (2i, 2i + 1) paired where
`interleaved`; `head_scale`: the name of one learned factor a query head on its scores; `chunk` = size: query i
sees key j <= i only if floor(i / size) = floor(j / size), counted from the sequence's position 0 (the cache
then keeps the pages of the query's own run alone); `fixed_sink` = s: a sink whose score is the constant s.

And: `qk_norm_scope` = "head": the norms of `qk_norm` are a head at a time, with one gain of the head's size for all
heads; `unit_qk`: after the rotation every q and k head is divided by its own root mean square (no gain); `rotary` may
carry a fourth entry, the frequencies' scaling (parts/position.py); `values_are_keys`: the values are the keys as
projected (biases included), before norm and rotation, and there is no value matrix; `shares_cache`: the layer has no
tensors of keys and values and reads the keys and values that another entry of the schedule cached.  With any of these,
or with both norms and a rotation, the projection stays in float32 and one launch makes norms and rotation of q and
k, rounds once, and puts keys and values straight into the cache's pages (`ops.qkv_prepare`).

And: `out_bias` = suffix: the output projection has a bias of that suffix; `gate_scope` = "head": the gate's matrix has one
row a head and the whole head's output is multiplied by its sigmoid (also beside convolutions); `distance_bias` = (name,
far, rows): a table [rows, heads] whose entry for the bucket of the distance to the key (`position.distance_buckets`) is
added to a score after the scale (`rows` is what random-weights mode draws; a checkpoint's table has its own number);
`value_mix`: "keep" leaves the layer's values (after the convolution, before the cache) for later layers of the step, any
other name is that of a stored number lambda, and the values become (1 - lambda) * own + lambda * those kept, before they are
cached (values carried from the first layer: Zhou et al., "Value Residual Learning").
"""
from __future__ import annotations

from .base import CacheNeed, Mixer, StateNeed, WeightSpec, register_part


def slope_base_or_sink(slope_base, sink) -> bool:
    return slope_base is not None or sink is not None


class CausalAttention(Mixer):

    def __init__(self, prefix: str, width: int, n_heads: int, kv_heads: int, head_dim: int, scale: float,
                 window: int = 0, qkv="c_attn", out: str = "c_proj", stored: str = "in_out",
                 bias: bool = True, init_std: float = 0.02, out_init_std: float = 0.02, bias_init_std: float = 0.01,
                 keep_first: int = 0, value_dim: int | None = None, suffix: str = ".weight", qk_norm=None,
                 value_norm: bool = False, norm_eps: float = 0.0, q_temp=None, distance_slope_base: float | None = None,
                 sink: str | None = None, gate: str | None = None, qkv_bias: str | None = None, conv=None, rotary=None,
                 head_scale: str | None = None, chunk: int = 0, fixed_sink: float | None = None, qk_norm_scope: str = "row",
                 unit_qk: bool = False, values_are_keys: bool = False, shares_cache: bool = False, out_bias: str | None = None,
                 gate_scope: str = "value", distance_bias=None, value_mix: str | None = None):
        super().__init__(prefix)
        if n_heads % kv_heads:
            raise ValueError(f"attention {prefix!r}: {n_heads} heads are not a multiple of {kv_heads} key/value heads")
        if not 1 <= head_dim <= 256:
            raise ValueError(f"attention {prefix!r}: head size {head_dim} is not in [1, 256]")
        if stored not in ("in_out", "out_in"):
            raise ValueError(f"attention {prefix!r}: stored = {stored!r}")
        self.width, self.n_heads, self.kv_heads, self.head_dim = int(width), int(n_heads), int(kv_heads), int(head_dim)
        self.scale, self.window, self.keep_first = float(scale), int(window), int(keep_first)
        # keep_first or an explicit value size take the kernels that know both (and every head size, also in bfloat16)
        self.qk_norm_names = None if qk_norm is None else tuple(prefix + n for n in qk_norm)
        self.value_norm, self.norm_eps = bool(value_norm), float(norm_eps)
        self.q_temp = None if q_temp is None else (float(q_temp[0]), int(q_temp[1]))
        if self.q_temp is not None and self.q_temp[1] <= 0:
            raise ValueError(f"attention {prefix!r}: a temperature that grows every {self.q_temp[1]} positions")
        self.slope_base = None if distance_slope_base is None else float(distance_slope_base)
        self.sink_name = None if sink is None else prefix + sink
        self.gate_name = None if gate is None else prefix + gate
        if gate_scope not in ("value", "head"):
            raise ValueError(f"attention {prefix!r}: gate_scope = {gate_scope!r}")
        self.gate_scope = gate_scope
        # rows that pass a norm, a temperature or a gate between the projection and the attention
        self.prepared = (self.qk_norm_names is not None or self.value_norm or self.q_temp is not None
                         or (self.gate_name is not None and conv is None))
        self.out_bias_name = None if out_bias is None else prefix + out + out_bias
        if out_bias is not None and bias:
            raise ValueError(f"attention {prefix!r}: an output bias by its suffix comes without the fused projection's biases")
        self.distance_bias = None
        if distance_bias is not None:
            self.distance_bias = (prefix + distance_bias[0], float(distance_bias[1]), int(distance_bias[2]))
        self.value_mix = value_mix
        self.value_lambda_name = None if value_mix in (None, "keep") else prefix + value_mix
        self.value_lambda = 0.0
        self.fixed_sink = None if fixed_sink is None else float(fixed_sink)
        self.chunk = int(chunk)
        self.head_scale_name = None if head_scale is None else prefix + head_scale
        self.conv = None if conv is None else (int(conv[0]), str(conv[1]))
        self.qkv_bias_suffix = qkv_bias
        self.rotary = None
        if rotary is not None:
            from .position import Rotary
            self.rotary = Rotary(prefix, dims=int(rotary[0]), base=float(rotary[1]), interleaved=bool(rotary[2]),
                                 scaling=rotary[3] if len(rotary) > 3 else None)
            if self.rotary.dims > head_dim:
                raise ValueError(f"attention {prefix!r}: {self.rotary.dims} rotated dimensions of a head of {head_dim}")
        if self.chunk < 0 or (self.chunk and window):
            raise ValueError(f"attention {prefix!r}: chunk {self.chunk} (not negative, and not beside a window)")
        if self.fixed_sink is not None and sink is not None:
            raise ValueError(f"attention {prefix!r}: a learned sink or a fixed one")
        if self.conv is not None and not 1 <= self.conv[0] <= 16:
            raise ValueError(f"attention {prefix!r}: a convolution of {self.conv[0]} taps is not in [1, 16]")
        if (qkv_bias is not None or self.conv is not None) and (isinstance(qkv, str) or bias):
            raise ValueError(f"attention {prefix!r}: biases on q, k and v alone and convolutions come with q, k and v "
                             "stored as three matrices, without the fused projection's biases")
        if qk_norm_scope not in ("row", "head"):
            raise ValueError(f"attention {prefix!r}: qk_norm_scope = {qk_norm_scope!r}")
        self.qk_norm_scope, self.unit_qk = qk_norm_scope, bool(unit_qk)
        self.values_are_keys, self.shares_cache = bool(values_are_keys), bool(shares_cache)
        # norms and a rotation together, or what only the one launch of both knows
        self.one_prepare = (self.unit_qk or self.values_are_keys or self.shares_cache or
                            (self.qk_norm_names is not None and (qk_norm_scope == "head" or self.rotary is not None)))
        if self.one_prepare and (isinstance(qkv, str) or bias or self.value_norm or self.q_temp is not None or self.gate_name is not None
                                 or self.conv is not None):
            raise ValueError(f"attention {prefix!r}: norms a head, norms with a rotation, values that are keys and another entry's "
                             "cache come with q, k and v stored apart, without value norms, temperatures, gates or convolutions")
        if self.values_are_keys and value_dim is not None and int(value_dim) != int(head_dim):
            raise ValueError(f"attention {prefix!r}: values that are the keys have the keys' size, not {value_dim}")
        if value_mix is not None and (self.shares_cache or self.values_are_keys or not (self.one_prepare or conv is not None)):
            raise ValueError(f"attention {prefix!r}: values that are kept or blended come with values of the layer's own, after norms "
                             "a head or convolutions")
        if conv is not None and (qk_norm is not None or value_norm or q_temp is not None):
            raise ValueError(f"attention {prefix!r}: convolutions come without norms and temperatures")
        self.biased = (self.slope_base is not None or self.sink_name is not None or self.fixed_sink is not None
                       or self.chunk > 0 or self.head_scale_name is not None or distance_bias is not None)
        if (self.prepared or self.one_prepare or slope_base_or_sink(distance_slope_base, sink)) and bias:
            raise ValueError(f"attention {prefix!r}: norms, gates, slopes and sinks come without biases")
        self.extended = int(keep_first) > 0 or value_dim is not None or self.prepared or self.biased or self.one_prepare
        self.value_dim = self.head_dim if value_dim is None else int(value_dim)
        if not 1 <= self.value_dim <= 256:
            raise ValueError(f"attention {prefix!r}: value size {self.value_dim} is not in [1, 256]")
        if self.keep_first < 0 or self.window < 0:
            raise ValueError(f"attention {prefix!r}: window {self.window}, keep_first {self.keep_first}")
        self.split = not isinstance(qkv, str)      # q, k and v stored as three matrices
        if self.split and (len(qkv) != 3 or bias):
            raise ValueError(f"attention {prefix!r}: three names for q, k and v, and no biases with them")
        self.qkv_name = tuple(prefix + n for n in qkv) if self.split else prefix + qkv
        self.out_name, self.stored, self.bias, self.suffix = prefix + out, stored, bias, suffix
        self.init_std, self.out_init_std, self.bias_init_std = init_std, out_init_std, bias_init_std
        self.q_width = self.n_heads * self.head_dim
        self.o_width = self.n_heads * self.value_dim
        self.widths = (self.q_width, self.kv_heads * self.head_dim, self.kv_heads * self.value_dim)
        self.qkv_width = sum(self.widths)
        self.w_qkv = self.b_qkv = self.w_out = self.b_out = None
        self.q_gain = self.k_gain = self.sinks = self.slopes = self.dist_bias = None

    def _shape(self, n_in, n_out):
        return (n_in, n_out) if self.stored == "in_out" else (n_out, n_in)

    def _projections(self):
        """(name, output width) of the matrices that the layer has of q, k and v stored apart."""
        return list(zip(self.qkv_name, self.widths))[:1 if self.shares_cache else (2 if self.values_are_keys else 3)]

    def weight_specs(self):
        if self.split:
            specs = [WeightSpec(n + self.suffix, self._shape(self.width, w), std=self.init_std)
                     for n, w in self._projections()]
        else:
            specs = [WeightSpec(self.qkv_name + self.suffix, self._shape(self.width, self.qkv_width), std=self.init_std)]
        specs.append(WeightSpec(self.out_name + self.suffix, self._shape(self.o_width, self.width), std=self.out_init_std))
        if self.bias:
            specs += [WeightSpec(self.qkv_name + ".bias", (self.qkv_width,), std=self.bias_init_std),
                      WeightSpec(self.out_name + ".bias", (self.width,), std=self.bias_init_std)]
        if self.qk_norm_names is not None:
            per_head = self.qk_norm_scope == "head"
            specs += [WeightSpec(n, (self.head_dim if per_head else w,), mean=1.0, std=0.1)
                      for n, w in list(zip(self.qk_norm_names, self.widths))[:1 if self.shares_cache else 2]]
        if self.sink_name is not None:
            specs.append(WeightSpec(self.sink_name, (self.n_heads,), std=1.0))
        if self.gate_name is not None:
            n = self.n_heads if self.gate_scope == "head" else self.o_width
            specs.append(WeightSpec(self.gate_name + self.suffix, self._shape(self.width, n), std=self.init_std))
        if self.out_bias_name is not None:
            specs.append(WeightSpec(self.out_bias_name, (self.width,), std=self.bias_init_std))
        if self.distance_bias is not None:
            specs.append(WeightSpec(self.distance_bias[0], (self.distance_bias[2], self.n_heads), std=1.0, free=(0,)))
        if self.value_lambda_name is not None:
            specs.append(WeightSpec(self.value_lambda_name, (), mean=0.5, std=0.1))
        if self.qkv_bias_suffix is not None:
            specs += [WeightSpec(n + self.qkv_bias_suffix, (w,), std=self.bias_init_std * 10) for n, w in self._projections()]
        if self.conv is not None:
            specs += [WeightSpec(n + self.conv[1], (w, self.conv[0]), std=0.5) for n, w in zip(self.qkv_name, self.widths)]
        if self.head_scale_name is not None:
            specs.append(WeightSpec(self.head_scale_name, (self.n_heads,), mean=1.0, std=0.2))
        return specs

    def load(self, get, runtime):
        import torch
        if runtime.dtype == torch.bfloat16 and not self.extended and (self.head_dim % 16 or self.width % 8):
            # (the true 32-bit path takes every head size up to 256 and every width)
            raise ValueError(f"attention {self.prefix!r}: the bfloat16 kernels take head sizes that are multiples of 16 "
                             f"and widths that are multiples of 8 (here {self.head_dim} and {self.width}); "
                             "the float32 path takes this model")
        t = self.stored == "in_out"
        if self.split:
            self.w_qkv = torch.cat([runtime.matrix(get(n + self.suffix), transpose=t) for n, _ in self._projections()]).contiguous()
        else:
            self.w_qkv = runtime.matrix(get(self.qkv_name + self.suffix), transpose=t)
        self.w_out = runtime.matrix(get(self.out_name + self.suffix), transpose=t)
        if self.gate_name is not None:      # the gate's rows under q | k | v, each part from a multiple of 8 columns on
            self.gate_col = -(-self.qkv_width // 8) * 8
            pad = torch.zeros((self.gate_col - self.qkv_width, self.width), dtype=self.w_qkv.dtype, device=self.w_qkv.device)
            self.w_qkv = torch.cat([self.w_qkv, pad, runtime.matrix(get(self.gate_name + self.suffix), transpose=t)]).contiguous()
        if self.qk_norm_names is not None:
            self.q_gain = runtime.vector(get(self.qk_norm_names[0]))
            self.k_gain = None if self.shares_cache else runtime.vector(get(self.qk_norm_names[1]))
        if self.sink_name is not None:
            self.sinks = runtime.vector(get(self.sink_name))
        if self.slope_base is not None:
            self.slopes = torch.tensor([2.0 ** (-self.slope_base * (h + 1) / self.n_heads) for h in range(self.n_heads)],
                                       dtype=torch.float32, device=self.w_qkv.device)
        if self.bias:
            self.b_qkv = runtime.vector(get(self.qkv_name + ".bias"))
            self.b_out = runtime.vector(get(self.out_name + ".bias"))
        if self.out_bias_name is not None:
            self.b_out = runtime.vector(get(self.out_bias_name))
        if self.distance_bias is not None:      # spread over the distances: [heads, distances], the last column for all beyond
            from .position import distance_buckets
            table = runtime.vector(get(self.distance_bias[0]))
            of = distance_buckets(table.shape[0], self.distance_bias[1])
            of = of[:max(1, min(len(of), self.chunk or self.window or len(of)))]
            self.dist_bias = table[torch.tensor(of, device=table.device)].t().contiguous()
        if self.value_lambda_name is not None:
            self.value_lambda = float(get(self.value_lambda_name))
        if self.qkv_bias_suffix is not None:
            self.b_qkv = torch.cat([runtime.vector(get(n + self.qkv_bias_suffix)) for n, _ in self._projections()]).contiguous()
        if self.conv is not None:
            self.conv_w = torch.cat([runtime.vector(get(n + self.conv[1])) for n in self.qkv_name]).contiguous()
            self.conv_b = torch.zeros(self.qkv_width, dtype=torch.float32, device=self.conv_w.device)
        if self.rotary is not None:
            self.rotary.load(get, runtime)
        if self.fixed_sink is not None:
            self.sinks = torch.full((self.n_heads,), self.fixed_sink, dtype=torch.float32, device=self.w_qkv.device)
        self.head_scales = None
        if self.head_scale_name is not None:
            self.head_scales = runtime.vector(get(self.head_scale_name))
            # (the tensor-core kernels take their exponents against a running maximum of the raw products, which
            # needs factors above zero; any other head takes the plain kernel)
            self.head_scales_positive = bool((self.head_scales > 0).all())

    def stream_weights(self):
        return [self.w_qkv, self.w_out]

    def state_need(self):
        if self.conv is None or self.conv[0] <= 1:
            return None
        return {"conv": StateNeed((self.conv[0] - 1, self.qkv_width))}     # the projected rows before the step's first, oldest first

    def cache_need(self):
        if self.chunk > 0:
            return CacheNeed("chunk", self.kv_heads, self.head_dim, self.chunk, 0,
                             0 if self.value_dim == self.head_dim else self.value_dim)
        windowed = self.window > 0
        return CacheNeed("window" if windowed else "full", self.kv_heads, self.head_dim, self.window,
                         self.keep_first if windowed else 0, 0 if self.value_dim == self.head_dim else self.value_dim)

    def _attend_prepared(self, ctx, h, app):
        import torch
        ops = ctx.ops
        if app.writes_cache == self.shares_cache:
            raise ValueError(f"attention {self.prefix!r}: a layer with keys and values of its own writes the cache, a layer "
                             "without them reads another entry's")
        proj = ops.linear(h, self.w_qkv, self.b_qkv, out_dtype=torch.float32)            # float32 [T, q (| k (| v))]
        norm = None if self.qk_norm_names is None else self.qk_norm_scope
        qkv = ops.qkv_prepare(proj, ctx.plan, app.cache, self.n_heads, self.kv_heads, self.head_dim, self.value_dim, ctx.dtype,
                              store=not self.shares_cache, v_col=self.q_width if self.values_are_keys else None, norm=norm,
                              q_gain=self.q_gain, k_gain=self.k_gain, eps=self.norm_eps, rotary=self.rotary, unit_after=self.unit_qk,
                              **self._value_mix(ctx, proj))
        more = self._sight()
        if self._plain_sight():
            return ops.attention(qkv, app.cache, ctx.plan, self.n_heads, self.kv_heads, self.head_dim, self.scale, self.window,
                                 out_dtype=ctx.dtype, store=False)
        return ops.attention(qkv, app.cache, ctx.plan, self.n_heads, self.kv_heads, self.head_dim, self.scale, self.window,
                             out_dtype=ctx.dtype, store=False, keep_first=self.keep_first if self.window > 0 else 0,
                             value_dim=self.value_dim, **more)

    def _sight(self) -> dict:
        """What the attention's kernels take beside heads, scale and window."""
        more = dict(slopes=self.slopes, sinks=self.sinks, chunk=self.chunk, head_scales=self.head_scales,
                    head_scales_positive=self.head_scales is None or self.head_scales_positive)
        if self.dist_bias is not None:
            more["dist_bias"] = self.dist_bias
        return more

    def _value_mix(self, ctx, rows) -> dict:
        """`rows` [T, q | k | v ...]: keeps the columns of the values for later layers of the step, or names those kept and
        their weight in the blend."""
        if self.value_mix is None:
            return {}
        if self.value_mix == "keep":
            ctx.kept["values"] = rows[:, sum(self.widths[:2]):self.qkv_width]
            return {}
        return {"mix": (ctx.kept["values"], self.value_lambda)}

    def _plain_sight(self) -> bool:
        """Nothing but a window on the scores, and the head size at which the kernels for such heads are the faster ones (one
        token each of 8 sequences at 2,048 positions, 16 heads over 4: 8.9 against 14.9 microseconds at 64, 25 against 19 at 128)."""
        return (not self.biased and self.keep_first == 0 and self.value_dim == self.head_dim == 64
                and self.n_heads // self.kv_heads <= 8 and self.scale > 0)

    def _attend(self, ctx, h, app):
        ops = ctx.ops
        if self.one_prepare:
            return self._attend_prepared(ctx, h, app)
        if self.prepared:
            import torch
            proj = ops.linear(h, self.w_qkv, None, out_dtype=torch.float32)          # float32 [T, q | k | v (| 0 | g)]
            coef, every = self.q_temp or (0.0, 1)
            qkv = ops.qkv_norm(proj, ctx.plan.positions, self.n_heads, self.kv_heads, self.head_dim, self.value_dim, ctx.dtype,
                               q_gain=self.q_gain, k_gain=self.k_gain, unit_values=self.value_norm, eps=self.norm_eps,
                               temp_coef=coef, temp_every=every)
            ctx.position.apply_qk(ctx, qkv, self.n_heads, self.kv_heads, self.head_dim)
            o = ops.attention(qkv, app.cache, ctx.plan, self.n_heads, self.kv_heads, self.head_dim, self.scale, self.window,
                              out_dtype=ctx.dtype, store=app.writes_cache, keep_first=self.keep_first if self.window > 0 else 0,
                              value_dim=self.value_dim, slopes=self.slopes, sinks=self.sinks)
            return o if self.gate_name is None else self._gated(ctx, o, proj)
        qkv = proj = ops.linear(h, self.w_qkv, self.b_qkv, out_dtype=ctx.dtype)
        store = app.writes_cache
        if self.conv is not None:
            state = app.state.get("conv") if isinstance(app.state, dict) else None
            qkv = ops.conv_silu(qkv, 0, self.qkv_width, self.conv_w, self.conv_b, state, ctx.plan, act="none")
        ctx.position.apply_qk(ctx, qkv, self.n_heads, self.kv_heads, self.head_dim)
        if self.rotary is not None:
            self.rotary.apply_qk(ctx, qkv, self.n_heads, self.kv_heads, self.head_dim)
        if self.value_mix is not None:      # the keys and the blended values go into the cache by a launch of their own
            ops.qkv_prepare(qkv, ctx.plan, app.cache, self.n_heads, self.kv_heads, self.head_dim, self.value_dim, ctx.dtype,
                            store=True, queries=False, **self._value_mix(ctx, qkv))
            store = False
        if not self.extended:
            o = ops.attention(qkv, app.cache, ctx.plan, self.n_heads, self.kv_heads, self.head_dim, self.scale,
                              self.window, out_dtype=ctx.dtype, store=store)
        else:
            o = ops.attention(qkv, app.cache, ctx.plan, self.n_heads, self.kv_heads, self.head_dim, self.scale, self.window,
                              out_dtype=ctx.dtype, store=store, keep_first=self.keep_first if self.window > 0 else 0,
                              value_dim=self.value_dim, **self._sight())
        return o if self.gate_name is None else self._gated(ctx, o, proj)

    def _gated(self, ctx, o, proj):
        return ctx.ops.gate_mul(o, proj, self.gate_col, "sigmoid", **({"span": self.value_dim} if self.gate_scope == "head" else {}))

    def forward(self, ctx, h, residual, app):
        return ctx.ops.linear(self._attend(ctx, h, app), self.w_out, self.b_out, residual=residual)

    def branches(self, ctx, h, app):
        import torch
        return [(ctx.ops.linear(self._attend(ctx, h, app), self.w_out, self.b_out, out_dtype=torch.float32), 1.0)]


register_part("mixer", "causal_attention", CausalAttention)
