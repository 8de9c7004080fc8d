"""A gated linear recurrence (a real-gated linear recurrent unit in a block of two branches): a
mixer that keeps one number per channel.

    y         = gelu_tanh(W_y h + b_y)                 [inner]
    u         = conv(W_x h + b_x) + bias               causal over time, per channel, `taps` wide
    r, i      = sigmoid(M u_b + bias)                  per equal part u_b of u, square matrices
    log a     = -8 r softplus(lam)
    S         <- a S + sqrt(1 - a^2) i u
    out       = W_o (S y)

The slot of a request keeps S and the convolution's last inputs, float32.  The convolution's sums,
the gates, decays and the state are float32 in both dtypes; the gates' products take u with 16 bits
of mantissa on the tensor cores and in plain float32 elsewhere.

A step of single tokens is one kernel between the input product and the output product; with
portions of prompts the recurrence goes in chunks of consecutive tokens (``csrc/lru.cu``).
"""

from __future__ import annotations

import torch

from ..kernels import lru
from .base import StateSpec, compute_matrix, register_mixer
from .context import StepPrep
from .recurrent import ProjectedMixer, stack_segments, vector32


class GatedRecurrence(ProjectedMixer):
    kind = "gated_recurrence"

    def __init__(self, width: int, inner: int, blocks: int, taps: int, dtype, device,
                 rate: float = 8.0) -> None:
        super().__init__(dtype, device)
        if min(inner, blocks, taps) <= 0 or inner % blocks:
            raise ValueError(f"gated_recurrence: sizes must be positive and blocks ({blocks}) "
                             f"divide inner ({inner})")
        if taps > lru.MAX_TAPS:
            raise ValueError(f"gated_recurrence: {taps} taps are beyond {lru.MAX_TAPS}")
        self.width, self.rate = width, float(rate)
        self.sizes = lru.Sizes(inner, blocks, taps)

    def tensors(self):
        d, s = self.width, self.sizes
        W, n, b = s.width, s.part, s.blocks
        return {"y": ((W, d), "matrix"), "y.b": ((W,), "bias"), "x": ((W, d), "matrix"),
                "x.b": ((W,), "bias"), "conv": ((W, s.taps), "matrix"), "conv.b": ((W,), "bias"),
                "ra": ((b, n, n), "matrix"), "ra.b": ((b, n), "bias"),
                "ri": ((b, n, n), "matrix"), "ri.b": ((b, n), "bias"), "lam": ((W,), "bias"),
                "o": ((d, W), "matrix")}

    def load(self, tensors):
        s, dev = self.sizes, self.device
        self._host_in, offsets = stack_segments([tensors["x"], tensors["y"]])
        self.y_col = offsets[1]
        self.w_o = compute_matrix(tensors["o"], self.dtype, dev)
        self.w_in = None

        def gate(name):
            return compute_matrix(tensors[name].reshape(s.width, s.part), self.dtype, dev)

        rate = self.rate * torch.nn.functional.softplus(tensors["lam"].to(torch.float64))
        self.weights = lru.Weights(
            x_bias=vector32(tensors["x.b"], dev), y_bias=vector32(tensors["y.b"], dev),
            taps=vector32(tensors["conv"].t(), dev), bias=vector32(tensors["conv.b"], dev),
            r=gate("ra"), i=gate("ri"), r_bias=vector32(tensors["ra.b"].reshape(-1), dev),
            i_bias=vector32(tensors["ri.b"].reshape(-1), dev), rate=vector32(rate, dev))

    def input_matrix(self):
        return self._host_in

    def kernel_modules(self):
        return ("lru",)

    def cache_spec(self):
        return StateSpec((self.sizes.slot_size,))

    # whether the step brings single tokens only; the same for layers of all sizes
    prepare_key = "gated_recurrence"

    def prepare(self, prep: StepPrep) -> None:
        prep.notes["gated_recurrence"] = int(prep.host.seq_qlen.max()) == 1

    def output_rows(self) -> int:
        return self.sizes.width

    def run(self, proj, ctx, cache, ahead=None, out_dtype=None):
        rows = ctx.buffer("gated_recurrence.rows", (proj.shape[0], self.sizes.width))
        self.run_into(proj, ctx, cache, rows)
        return self.project_out(rows, "gated_recurrence.out", ctx, ahead, out_dtype=out_dtype)

    def run_into(self, proj, ctx, cache, out, out_scale: float = 1.0) -> None:
        if cache is None or cache.kind != "state" or not cache.writes:
            raise ValueError("gated_recurrence needs a state slot of its own: it advances it")
        s, n = self.sizes, proj.shape[0]
        W = s.width
        common = (s, self.weights, proj[:, :W], proj[:, self.y_col: self.y_col + W], cache.state, out)
        if ctx.notes["gated_recurrence"]:
            lru.step(*common, ctx, scale=out_scale)
            return
        f32 = torch.float32
        prod = ctx.buffer("gated_recurrence.prod", (n, W), f32)
        local = ctx.buffer("gated_recurrence.local", (n, W), f32)
        terms = None
        if self.dtype == torch.bfloat16:
            terms = ctx.buffer("gated_recurrence.terms", (2, n, W))
        lru.gates(*common, prod, local, ctx, terms)
        carry = None
        if n > lru.CHUNK:
            carry = ctx.buffer("gated_recurrence.carry", (-(-n // lru.CHUNK), W), f32)
            lru.carry_on(*common, prod, local, carry, ctx)
        lru.finish(*common, prod, local, carry, ctx, scale=out_scale)


register_mixer("gated_recurrence", GatedRecurrence)
