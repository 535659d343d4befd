"""Griffin's recurrent block as a mixer with per-sequence state and no cache (De et al., "Griffin: Mixing Gated
Linear Recurrences with Local Attention for Efficient Language Models"): two branches, of which one passes a short
causal convolution and a real-gated linear recurrence and the other gates the result.

    y_t = gelu_tanh(W_y h_t + b_y)          u_t = conv(W_x h_t + b_x)
    r_t = sigmoid(R u_t + b_r)              i_t = sigmoid(I u_t + b_i)       (R, I: a square matrix for each of `blocks` parts)
    log a_t = -factor * r_t * softplus(lam)
    S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t      (element by element, S starts at zero)      out_t = W_o (S_t * y_t)

The convolution is causal, a filter and a bias a channel, the last tap on the current token, zeros before the sequence's
start, no activation.  One stacked projection makes y | x in the compute type, as does the convolution; the gates'
products keep their float32 sums, and gates, decays, the recurrence and its state are float32 in every mode.

What a sequence carries from step to step: S (`StateNeed` "S", `inner` values) and the last `conv` - 1 rows that entered
the convolution ("conv").
"""
from __future__ import annotations

from .base import Mixer, StateNeed, WeightSpec, register_part


class RealGatedLRU(Mixer):

    def __init__(self, prefix: str, width: int, inner: int, blocks: int, conv: int, factor: float, out_branch: str = "y",
                 in_branch: str = "x", conv_name: str = "conv", gate_r: str = "ra", gate_i: str = "ri", lam: str = "lam",
                 bias_suffix: str = ".b", out: str = "o", init_std: float = 0.02, out_init_std: float = 0.02):
        super().__init__(prefix)
        self.width, self.inner, self.blocks, self.taps, self.factor = int(width), int(inner), int(blocks), int(conv), float(factor)
        if self.inner <= 0 or self.blocks <= 0 or self.inner % self.blocks:
            raise ValueError(f"rglru {prefix!r}: {self.inner} channels do not split into {self.blocks} equal parts")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"rglru {prefix!r}: a convolution of {self.taps} taps is not in [1, 16]")
        if self.factor < 0:
            raise ValueError(f"rglru {prefix!r}: factor {self.factor} must not be negative")
        self.part = self.inner // self.blocks
        self.names = {k: prefix + v for k, v in dict(y=out_branch, x=in_branch, conv=conv_name, r=gate_r, i=gate_i, lam=lam,
                                                     out=out).items()}
        self.bias_suffix = bias_suffix
        self.init_std, self.out_init_std = init_std, out_init_std
        self.w_in = self.w_out = None

    def weight_specs(self):
        n, b, m = self.names, self.bias_suffix, self.inner
        gates = (self.blocks, self.part, self.part)
        return [WeightSpec(n["y"], (m, self.width), std=self.init_std), WeightSpec(n["y"] + b, (m,), std=0.1),
                WeightSpec(n["x"], (m, self.width), std=self.init_std), WeightSpec(n["x"] + b, (m,), std=0.1),
                WeightSpec(n["conv"], (m, self.taps), std=0.5), WeightSpec(n["conv"] + b, (m,), std=0.1),
                WeightSpec(n["r"], gates, std=0.1), WeightSpec(n["r"] + b, gates[:2], std=0.5),
                WeightSpec(n["i"], gates, std=0.1), WeightSpec(n["i"] + b, gates[:2], std=0.5),
                WeightSpec(n["lam"], (m,), mean=-4.0, std=1.0),
                WeightSpec(n["out"], (self.width, m), std=self.out_init_std)]

    def load(self, get, runtime):
        import torch
        n, b = self.names, self.bias_suffix
        # both branches start on a multiple of 8 columns (rows of zeros behind the first where its size is none)
        self.x_col = -(-self.inner // 8) * 8
        rows, biases = [], []
        for k in ("y", "x"):
            w, bias = runtime.matrix(get(n[k])), runtime.vector(get(n[k] + b))
            pad = self.x_col - self.inner
            if pad:
                w = torch.cat([w, torch.zeros((pad, self.width), dtype=w.dtype, device=w.device)])
                bias = torch.cat([bias, torch.zeros(pad, dtype=bias.dtype, device=bias.device)])
            rows.append(w)
            biases.append(bias)
        self.w_in, self.b_in = torch.cat(rows).contiguous(), torch.cat(biases).contiguous()
        self.conv_w, self.conv_b = runtime.vector(get(n["conv"])), runtime.vector(get(n["conv"] + b))
        # a part's two matrices under one another: the gates' products read u once
        self.w_gates = torch.cat([runtime.matrix(get(n["r"])), runtime.matrix(get(n["i"]))], dim=1).contiguous()
        self.b_r, self.b_i = (runtime.vector(get(n[k] + b)).reshape(-1).contiguous() for k in ("r", "i"))
        lam = runtime.vector(get(n["lam"])).double()
        self.rate = (self.factor * torch.logaddexp(lam, torch.zeros_like(lam))).float().contiguous()     # factor * softplus(lam)
        self.w_out = runtime.matrix(get(n["out"]))

    def stream_weights(self):
        return [self.w_in, self.w_out]

    def state_need(self):
        need = {"S": StateNeed((self.inner,))}
        if self.taps > 1:
            need["conv"] = StateNeed((self.taps - 1, self.inner))      # the rows before the step's first, oldest first
        return need

    def _mix(self, ctx, h, app):
        ops = ctx.ops
        proj = ops.linear(h, self.w_in, self.b_in, out_dtype=ctx.dtype)                   # [T, y (| 0) | x (| 0)]
        u = ops.conv_silu(proj, self.x_col, self.inner, self.conv_w, self.conv_b, app.state.get("conv"), ctx.plan, act="none")
        return ops.rglru(u, proj, 0, self.w_gates, self.b_r, self.b_i, self.rate, app.state["S"], ctx.plan)

    def forward(self, ctx, h, residual, app):
        return ctx.ops.linear(self._mix(ctx, h, app), self.w_out, None, residual=residual)

    def branches(self, ctx, h, app):
        import torch
        return [(ctx.ops.linear(self._mix(ctx, h, app), self.w_out, None, out_dtype=torch.float32), 1.0)]


register_part("mixer", "rglru", RealGatedLRU)
