"""The kernels of the gated linear recurrence (``csrc/lru.cu``) as functions of torch tensors.
Like ``ops``: every function launches on the current stream and checks what it passes on."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from . import library
from .ops import _check, _need, _ptr, _stream, _tag

CHUNK = 64               # tokens of a chunk
MAX_TAPS = 16
STATE_ALIGN = 4          # the kept rows begin at a multiple of this


@dataclass(frozen=True)
class Sizes:
    """``width`` channels in ``blocks`` equal parts; the convolution has ``taps`` taps."""
    width: int
    blocks: int
    taps: int

    @property
    def part(self) -> int:
        return self.width // self.blocks

    @property
    def kept_offset(self) -> int:
        """Where the convolution's kept inputs (a ring of ``taps`` rows) begin in a slot's row."""
        return (self.width + STATE_ALIGN - 1) // STATE_ALIGN * STATE_ALIGN

    @property
    def slot_size(self) -> int:
        kept = self.taps * self.width if self.taps > 1 else 0
        return (self.kept_offset + kept + STATE_ALIGN - 1) // STATE_ALIGN * STATE_ALIGN


@dataclass
class Weights:
    """On the device.  float32: the branches' biases ``x_bias`` and ``y_bias`` [W], ``taps`` [K, W]
    (the last row is the token's own), ``bias`` [W] of the convolution, the gates' ``r_bias`` and
    ``i_bias`` [W], ``rate`` [W].  Compute dtype: the gates' ``r`` and ``i`` [W, part], row b part + o
    being output o of part b."""
    x_bias: torch.Tensor
    y_bias: torch.Tensor
    taps: torch.Tensor
    bias: torch.Tensor
    r: torch.Tensor
    i: torch.Tensor
    r_bias: torch.Tensor
    i_bias: torch.Tensor
    rate: torch.Tensor


def _launch(stage: int, sz: Sizes, w: Weights, x: torch.Tensor, y: torch.Tensor,
            state: torch.Tensor, out: torch.Tensor, scale: float, ctx, prod=None, local=None,
            carry=None, terms=None) -> None:
    n, W = x.shape[0], sz.width
    for t, shape, name in ((w.x_bias, (W,), "x_bias"), (w.y_bias, (W,), "y_bias"),
                           (w.taps, (sz.taps, W), "taps"), (w.bias, (W,), "bias"),
                           (w.r_bias, (W,), "r_bias"), (w.i_bias, (W,), "i_bias"),
                           (w.rate, (W,), "rate")):
        _need(t.dtype == torch.float32 and t.is_contiguous() and tuple(t.shape) == shape,
              f"lru: {name} must be contiguous float32 {list(shape)}")
    for t, name in ((w.r, "r"), (w.i, "i")):
        _need(t.dtype == x.dtype and t.is_contiguous() and tuple(t.shape) == (W, sz.part),
              f"lru: {name} must be contiguous [W, part] of the activation dtype")
    _need(x.stride(1) == 1 and y.stride(1) == 1 and out.stride(1) == 1 and x.shape == (n, W)
          and y.shape == (n, W) and out.shape == (n, W) and x.dtype == y.dtype == out.dtype,
          "lru: x, y and out [N, W] of one dtype")
    _need(state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1
          and state.shape[1] >= sz.slot_size, "lru: state float32 [slots, slot_size]")
    for t, rows, name in ((prod, n, "prod"), (local, n, "local"), (carry, -(-n // CHUNK), "carry")):
        _need(t is None or (t.dtype == torch.float32 and t.is_contiguous()
                            and tuple(t.shape) == (rows, W)), f"lru: {name} float32 [{rows}, W]")
    _need(terms is None or (terms.dtype == x.dtype and terms.is_contiguous()
                            and tuple(terms.shape) == (2, n, W)),
          "lru: terms [2, N, W] of the activation dtype")
    lib = library.load("lru")
    _check(lib.de_lru(stage, _tag(x.dtype), x.data_ptr(), x.stride(0), y.data_ptr(), y.stride(0),
                      w.x_bias.data_ptr(), w.y_bias.data_ptr(), w.taps.data_ptr(),
                      w.bias.data_ptr(), w.r.data_ptr(), w.i.data_ptr(), w.r_bias.data_ptr(),
                      w.i_bias.data_ptr(), w.rate.data_ptr(), state.data_ptr(), state.stride(0),
                      sz.kept_offset, sz.taps, W, sz.part, n, ctx.token_seq.data_ptr(),
                      ctx.token_slot.data_ptr(), ctx.positions.data_ptr(),
                      ctx.seq_pos0.data_ptr(), ctx.seq_qlen.data_ptr(), out.data_ptr(),
                      out.stride(0), float(scale), _ptr(terms), _ptr(prod), _ptr(local),
                      _ptr(carry), _stream()), "lru")


def step(sz: Sizes, w: Weights, x: torch.Tensor, y: torch.Tensor, state: torch.Tensor,
         out: torch.Tensor, ctx, scale: float = 1.0) -> None:
    """A step in which every sequence brings one token: convolution, gates, state and out = S *
    gelu(y + y_bias) * scale in one kernel.  x, y, out: [N, W], row stride free."""
    _need(x.shape[0] == ctx.n_seqs, "lru step: one token a sequence")
    _launch(3, sz, w, x, y, state, out, scale, ctx)


def gates(sz, w, x, y, state, out, prod, local, ctx, terms=None) -> None:
    """``terms``: room for u's two bfloat16 terms [2, N, W], with which the gates' products go to
    the tensor cores where the sizes allow it.  prod and local [N, W]: S_t = prod S_start + local over the token's chunk of ``CHUNK``
    consecutive tokens of the step; a sequence's first token has prod 0 and its slot's S inside."""
    _launch(0, sz, w, x, y, state, out, 1.0, ctx, prod, local, terms=terms)


def carry_on(sz, w, x, y, state, out, prod, local, carry, ctx) -> None:
    """carry [chunks, W]: S at every chunk's start."""
    _launch(1, sz, w, x, y, state, out, 1.0, ctx, prod, local, carry)


def finish(sz, w, x, y, state, out, prod, local, carry, ctx, scale: float = 1.0) -> None:
    """out = S * gelu(y + y_bias) * scale; the slots' S and kept rows.  ``carry`` None: one chunk."""
    _launch(2, sz, w, x, y, state, out, scale, ctx, prod, local, carry)
