"""Mamba-2: a mixer whose heads keep a matrix state that decays by one input-dependent number a
token.

    [z | x | b | c | dt] = W_in h                         x, z [H P], b, c [G N], dt [H]
    x, b, c   = silu(conv([x | b | c]) + bias)            causal over time, per channel, `taps` wide
    dt        = softplus(dt + dt_bias);  a = -exp(A_log) dt
    S         <- exp(a) S + dt b x^T;  y = S^T c + D x     per head, S [N, P]; head h reads group
                                                          h // (H / G) of b and c
    out       = W_o [ parts of (y silu(z)) over their root mean squares * norm ]

The slot of a request keeps S of every head and the convolution's last ``taps`` - 1 inputs, float32.
The state, the step sizes, decays and read-outs are float32 in both dtypes.

A step of single tokens: the input product, one kernel from the projection to the read-outs, the
gate with its norm, the output product.  Portions: convolution and rates of all tokens first, then
short portions token by token and longer ones in chunks of tokens (``csrc/ssm.cu``).
"""

from __future__ import annotations

import numpy as np

from ..kernels import ssm
from .base import StateSpec, compute_matrix, register_mixer
from .context import StepPrep
from .recurrent import ProjectedMixer, stack_segments, vector32


class Mamba2(ProjectedMixer):
    kind = "mamba2"

    def __init__(self, width: int, heads: int, groups: int, state_dim: int, value_dim: int,
                 taps: int, norm_groups: int, eps: float, dtype, device) -> None:
        super().__init__(dtype, device)
        if min(heads, groups, state_dim, value_dim, taps, norm_groups) <= 0 or heads % groups:
            raise ValueError(f"mamba2: sizes must be positive and heads ({heads}) a multiple of "
                             f"groups ({groups})")
        if state_dim > ssm.MAX_STATE:
            raise ValueError(f"mamba2: a state of {state_dim} rows is beyond {ssm.MAX_STATE}")
        self.width, self.norm_groups, self.eps = width, norm_groups, float(eps)
        self.sizes = ssm.Sizes(heads, groups, state_dim, value_dim, taps)
        if self.sizes.inner % norm_groups:
            raise ValueError(f"mamba2: norm_groups ({norm_groups}) must divide heads * value_dim "
                             f"({self.sizes.inner})")

    def tensors(self):
        d, s = self.width, self.sizes
        return {"in": ((s.inner + s.channels + s.heads, d), "matrix"),
                "conv": ((s.channels, s.taps), "matrix"), "conv.b": ((s.channels,), "bias"),
                "dt_bias": ((s.heads,), "bias"), "A_log": ((s.heads,), "bias"),
                "D": ((s.heads,), "vector"), "norm": ((s.inner,), "vector"),
                "o": ((d, s.inner), "matrix")}

    def load(self, tensors):
        s = self.sizes
        z, xbc, dt = tensors["in"].split([s.inner, s.channels, s.heads], dim=0)
        self._host_in, offsets = stack_segments([z, xbc, dt])
        _, self.xbc_col, self.dt_col = offsets
        self.w_o = compute_matrix(tensors["o"], self.dtype, self.device)
        dev = self.device
        self.weights = ssm.Weights(vector32(tensors["conv"].t(), dev),
                                   vector32(tensors["conv.b"], dev),
                                   vector32(tensors["dt_bias"], dev),
                                   vector32(tensors["A_log"], dev), vector32(tensors["D"], dev))
        self.norm = vector32(tensors["norm"], dev)
        self.w_in = None

    def input_matrix(self):
        return self._host_in

    def kernel_modules(self):
        return ("ssm",)

    def cache_spec(self):
        return StateSpec((self.sizes.slot_size,))

    # the step's longer portions cut into chunks; the same for layers of all sizes
    prepare_key = "mamba2"

    def prepare(self, prep: StepPrep) -> None:
        if prep.has("mamba2/items"):
            return
        qlen, qstart = prep.host.seq_qlen, prep.host.seq_qstart
        items, portions = [], []
        for s in np.nonzero(qlen > ssm.SHORT_PORTION)[0]:
            first = np.arange(0, qlen[s], ssm.CHUNK, dtype=np.int32)
            part = np.zeros((len(first), 4), dtype=np.int32)
            part[:, 0], part[:, 1] = s, qstart[s] + first
            part[:, 2] = np.minimum(ssm.CHUNK, qlen[s] - first)
            portions.append((s, sum(len(p) for p in items), len(first), 0))
            items.append(part)
        prep.add("mamba2/items", np.concatenate(items) if items else np.zeros((0, 4)))
        prep.add("mamba2/portions", np.array(portions) if portions else np.zeros((0, 4)))
        # 0: single tokens only; else whether some portions are short
        prep.notes["mamba2"] = 0 if int(qlen.max()) == 1 else (
            2 if int(qlen.min()) <= ssm.SHORT_PORTION else 1)

    def run(self, proj, ctx, cache, ahead=None, out_dtype=None):
        if cache is None or cache.kind != "state" or not cache.writes:
            raise ValueError("mamba2 needs a state slot of its own: it advances it")
        n, s, state, f32 = proj.shape[0], self.sizes, cache.state, self.norm.dtype
        z = proj[:, : s.inner]
        xbc = proj[:, self.xbc_col: self.xbc_col + s.channels]
        dt = proj[:, self.dt_col: self.dt_col + s.heads]
        y = ctx.buffer("mamba2.y", (n, s.inner), f32)
        if ctx.notes["mamba2"] == 0:
            ssm.step(s, self.weights, xbc, dt, state, y, ctx)
        else:
            ready = ctx.buffer("mamba2.ready", (n, s.channels), f32)
            rates = ctx.buffer("mamba2.rates", (n, 2 * s.heads), f32)
            ssm.prep(s, self.weights, xbc, dt, state, ready, rates, ctx)
            items = ctx.arrays["mamba2/items"]
            if items.shape[0]:
                states = ctx.buffer("mamba2.states", (items.shape[0], s.state_size), f32)
                decays = ctx.buffer("mamba2.decays", (items.shape[0], s.heads), f32)
                products = ctx.buffer("mamba2.products", (items.shape[0], s.groups, ssm.CHUNK,
                                                          ssm.CHUNK), f32)
                ssm.chunk_state(s, ready, rates, items, states, decays, products)
                ssm.chunk_pass(s, states, decays, ctx.arrays["mamba2/portions"], state, ctx)
                ssm.chunk_out(s, self.weights, ready, rates, items, states, products, y)
            if ctx.notes["mamba2"] == 2:
                ssm.walk(s, self.weights, ready, rates, state, y, ctx)
        gated = ctx.buffer("mamba2.gated", (n, s.inner))
        ssm.gated_group_norm(y, z, self.norm, self.norm_groups, self.eps, gated, ctx,
                             keep=(s, xbc, state) if s.taps > 1 else None)
        return self.project_out(gated, "mamba2.out", ctx, ahead, out_dtype=out_dtype)


register_mixer("mamba2", Mamba2)
