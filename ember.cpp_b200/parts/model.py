"""A decoder built from a ModelSpec: token table, position encoding, the layers in their run
order, final norm, head.

The order is ember.cpp's for every decoder it runs: embed nodes, the block nodes once per
layer, then the head nodes on the wanted rows only (graph_ir.cpp:3010-3066; rows trimmed before
the head :3049-3061): `h = norm(x_rows)`, `logits = h Whead^T` without bias, Whead being the
token table when the head is tied (graph_ir.cpp:624-628, 757-762).  What other decoders put
around that order is data of the spec, not code of a model: a factor on the embedded rows, a bias
on the logits, a cap on them (cap * tanh(logits / cap)); GPT-2 uses none of the three.
"""
from __future__ import annotations

import torch

from .base import WeightSpec, build_block, build_part
from .spec import ModelSpec


class DecoderModel:
    def __init__(self, spec: ModelSpec):
        spec.check()
        self.spec = spec
        self.position = build_part("position", spec.position)
        self.blocks = []
        for layer in spec.layers:
            norm = lambda part: None if part is None else build_part("norm", part)  # noqa: E731
            self.blocks.append(build_block(layer.block, norm(layer.norm1), build_part("mixer", layer.mixer), norm(layer.norm2),
                                           None if layer.ffn is None else build_part("ffn", layer.ffn), {name: norm(part) for name, part in layer.more_norms},
                                           layer.block_params))
            self.blocks[-1].addons = [build_part("addon", part) for part in layer.addons]
        self.final_norm = build_part("norm", spec.final_norm)
        self.embed_parts = [build_part("embed", part) for part in spec.embed_parts]
        self.embed_norm = None if spec.embed_norm is None else build_part("norm", spec.embed_norm)
        self.table = None
        self.head = None
        self.head_bias = None
        self.keeps_history = any(getattr(p, "reads_history", False) for b in self.blocks for p in b.addons)
        self.reads_tokens = any(getattr(p, "needs_tokens", False) for p in self.all_parts())

    # ------------------------------------------------------------------ tensors
    def all_parts(self):
        parts = [self.position] + self.embed_parts + ([] if self.embed_norm is None else [self.embed_norm])
        for b in self.blocks:
            parts += b.parts()
        return parts + [self.final_norm]

    def weight_specs(self) -> list[WeightSpec]:
        s = self.spec
        specs = [WeightSpec(s.token_table, (s.vocab_size, s.width), std=s.table_init_std)]
        if s.head is not None:
            specs.append(WeightSpec(s.head, (s.vocab_size, s.width), std=s.table_init_std))
        if s.head_bias is not None:
            specs.append(WeightSpec(s.head_bias, (s.vocab_size,), std=s.table_init_std))
        for p in self.all_parts():
            specs += p.weight_specs()
        seen: dict[str, WeightSpec] = {}
        for w in specs:
            if w.name in seen and seen[w.name].shape != w.shape:
                raise ValueError(f"tensor {w.name!r} is wanted with shapes {seen[w.name].shape} and {w.shape}")
            seen.setdefault(w.name, w)
        return list(seen.values())

    def load(self, tensors: dict, runtime) -> None:
        """`tensors`: name -> tensor as stored (checked by the loader against weight_specs())."""
        get = tensors.__getitem__
        self.table = runtime.table(get(self.spec.token_table))
        self.head = self.table if self.spec.head is None else runtime.table(get(self.spec.head))
        self.head_bias = None if self.spec.head_bias is None else runtime.vector(get(self.spec.head_bias))
        for p in self.all_parts():
            p.load(get, runtime)

    # ------------------------------------------------------------------ what the cache must hold
    def max_positions(self) -> int | None:
        return self.position.max_positions()

    def application_needs(self):
        """(cache need, state need) of each entry of the schedule; an entry that reads another's
        cache has no cache need of its own, but that cache must hold what it reads as well."""
        mixers = [self.blocks[app.layer].mixer for app in self.spec.schedule]
        needs = [None if app.cache_of is not None else m.cache_need() for app, m in zip(self.spec.schedule, mixers)]
        for app, m in zip(self.spec.schedule, mixers):
            read = None if app.cache_of is None else m.cache_need()
            if read is not None and needs[app.cache_of] is not None:
                needs[app.cache_of] = needs[app.cache_of].joined(read)
        return [(need, m.state_need()) for need, m in zip(needs, mixers)]

    def model_state_needs(self) -> dict:
        """Per-sequence state that belongs to no layer: what the parts in front of the first layer carry,
        by the part's place among them (and the state's name where a part keeps several)."""
        need = {}
        for i, part in enumerate(self.embed_parts):
            s = part.state_need()
            if s is None:
                continue
            for key, one in (s.items() if isinstance(s, dict) else [("", s)]):
                need[f"embed{i}.{key}"] = one
        return need

    def _embed_state(self, ctx, i, part):
        s = part.state_need()
        if s is None:
            return None
        states = ctx.model_state
        return {key: states[f"embed{i}.{key}"] for key in s} if isinstance(s, dict) else states[f"embed{i}."]

    # ------------------------------------------------------------------ one step
    def forward(self, ctx):
        """Runs the tokens of `ctx.plan` through every entry of the schedule and returns float32
        logits [wanted rows, vocab] (None if no row is wanted)."""
        plan, ops = ctx.plan, ctx.ops
        ids = getattr(plan, "device_ids", None)   # sampled ids on the device that this step's tokens are taken from
        if ids is not None and self.reads_tokens:
            # a part looks its tokens up in a table of its own: the ids are put into the description first
            ops.take_tokens(plan.tokens, plan.token_src, ids, self.spec.vocab_size)
            ids = None
        scale = self.spec.embedding_scale
        in_kernel = scale != 1.0 and not self.spec.scale_positions    # the factor on the token's row alone: the embedding's own
        more = {"token_scale": scale} if in_kernel else {}
        if ids is not None:
            x = ops.embed(plan.tokens, plan.positions, self.table, self.position.embedding_table(),
                          token_src=plan.token_src, ids=ids, **more)
        else:
            x = ops.embed(plan.tokens, plan.positions, self.table, self.position.embedding_table(), **more)
        if scale != 1.0 and not in_kernel:
            x = ops.scale_cap(x, scale=scale)
        for i, part in enumerate(self.embed_parts):
            x = part.forward(ctx, x, self._embed_state(ctx, i, part))
        if self.embed_norm is not None:
            x = self.embed_norm.forward(ctx, x, torch.float32)
        if self.keeps_history:      # (a copy where the first layer would add into it)
            ctx.history = [x.clone() if ctx.apps and self.blocks[ctx.apps[0].layer].in_place else x]
        for i, app in enumerate(ctx.apps):
            # (a hint for the kernels: the first matrix that the block after this one streams)
            following = ctx.apps[i + 1].layer if i + 1 < len(ctx.apps) else None
            ctx.next_weights = self.blocks[following].mixer.stream_weights()[:1] if following is not None else ()
            x = self.blocks[app.layer].forward(ctx, x, app)
        if plan.n_want == 0:
            return None
        rows = x if plan.wants_every_row else ops.gather_rows(x, plan.want_rows, plan.n_want)
        h = self.final_norm.forward(ctx, rows, ctx.dtype)
        logits = ops.linear(h, self.head, self.head_bias, out_dtype=torch.float32)
        if self.spec.logit_cap is not None or self.spec.logit_scale != 1.0:
            logits = ops.scale_cap(logits, scale=self.spec.logit_scale, cap=self.spec.logit_cap)
        return logits
