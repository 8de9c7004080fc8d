"""The kernels of the state-space mixer (``csrc/ssm.cu``) as functions of torch tensors.  Like
``ops``: every function launches on the current stream and checks what it passes on."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from . import library
from .ops import _check, _i32, _need, _ptr, _stream, _tag

MAX_STATE = 256          # rows of a head's state
CHUNK = 64               # tokens of a chunk of a longer portion
SHORT_PORTION = 16       # portions of up to this many tokens are walked token by token


@dataclass(frozen=True)
class Sizes:
    """``heads`` of ``value_dim`` values each on states of ``state_dim`` rows; ``groups`` of heads
    share b and c; the convolution has ``taps`` taps."""
    heads: int
    groups: int
    state_dim: int
    value_dim: int
    taps: int

    @property
    def inner(self) -> int:
        return self.heads * self.value_dim

    @property
    def channels(self) -> int:               # [x | b | c], what passes the convolution
        return self.inner + 2 * self.groups * self.state_dim

    @property
    def state_size(self) -> int:
        return self.heads * self.state_dim * self.value_dim

    @property
    def kept_offset(self) -> int:
        """Where the convolution's kept inputs begin in a slot's row (a multiple of 4)."""
        return (self.state_size + 3) // 4 * 4

    @property
    def slot_size(self) -> int:
        return (self.kept_offset + (self.taps - 1) * self.channels + 3) // 4 * 4

    def tuple(self) -> tuple:
        return self.heads, self.groups, self.state_dim, self.value_dim, self.taps


@dataclass
class Weights:
    """float32 on the device: ``taps`` [K, C] (the last row is the token's own), ``bias`` [C],
    ``dt_bias``, ``a_log`` and ``skip`` [H]."""
    taps: torch.Tensor
    bias: torch.Tensor
    dt_bias: torch.Tensor
    a_log: torch.Tensor
    skip: torch.Tensor


def _checked(sz: Sizes, w: Weights, xbc: torch.Tensor, dt: torch.Tensor,
             state: torch.Tensor) -> None:
    n = xbc.shape[0]
    for t, shape, name in ((w.taps, (sz.taps, sz.channels), "taps"), (w.bias, (sz.channels,), "bias"),
                           (w.dt_bias, (sz.heads,), "dt_bias"), (w.a_log, (sz.heads,), "a_log"),
                           (w.skip, (sz.heads,), "skip")):
        _need(t.dtype == torch.float32 and t.is_contiguous() and tuple(t.shape) == shape,
              f"ssm: {name} must be contiguous float32 {list(shape)}")
    _need(xbc.stride(1) == 1 and dt.stride(1) == 1 and xbc.shape == (n, sz.channels)
          and dt.shape == (n, sz.heads) and xbc.dtype == dt.dtype, "ssm: xbc [N, C], dt [N, H]")
    _state(sz, state)


def _state(sz: Sizes, state: torch.Tensor) -> None:
    _need(state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1
          and state.shape[1] >= sz.slot_size, "ssm: state float32 [slots, slot_size]")


def _rows(sz: Sizes, ready: torch.Tensor, rates: torch.Tensor) -> None:
    n = ready.shape[0]
    for t, shape in ((ready, (n, sz.channels)), (rates, (n, 2 * sz.heads))):
        _need(t.dtype == torch.float32 and t.is_contiguous() and tuple(t.shape) == shape,
              "ssm: prepared rows float32 [N, C] and rates [N, 2 H]")


def _results(sz: Sizes, y: torch.Tensor, n: int) -> None:
    _need(y.dtype == torch.float32 and y.is_contiguous() and tuple(y.shape) == (n, sz.inner),
          "ssm: y float32 [N, H P]")


def prep(sz: Sizes, w: Weights, xbc: torch.Tensor, dt: torch.Tensor, state: torch.Tensor,
         ready: torch.Tensor, rates: torch.Tensor, ctx) -> None:
    """ready [N, C] = silu(convolution(xbc) + bias), earlier inputs from the slots; rates [N, 2 H]
    = softplus(dt + dt_bias), then -exp(a_log) times that.  xbc and dt: columns of the projection
    (row stride free)."""
    _checked(sz, w, xbc, dt, state), _rows(sz, ready, rates)
    lib = library.load("ssm")
    _check(lib.de_ssm_prep(_tag(xbc.dtype), xbc.data_ptr(), xbc.stride(0), dt.data_ptr(),
                           dt.stride(0), w.taps.data_ptr(), w.bias.data_ptr(),
                           w.dt_bias.data_ptr(), w.a_log.data_ptr(), state.data_ptr(),
                           state.stride(0), sz.kept_offset, ctx.token_seq.data_ptr(),
                           ctx.token_slot.data_ptr(), ctx.positions.data_ptr(),
                           ctx.seq_pos0.data_ptr(), ready.data_ptr(), rates.data_ptr(),
                           xbc.shape[0], *sz.tuple(), _stream()), "ssm_prep")


def step(sz: Sizes, w: Weights, xbc: torch.Tensor, dt: torch.Tensor, state: torch.Tensor,
         y: torch.Tensor, ctx) -> None:
    """A step in which every sequence brings one token: convolution, rates, state and read-out
    y [N, H P] in one kernel (the kept inputs stay: ``gated_group_norm`` moves them on)."""
    _checked(sz, w, xbc, dt, state), _results(sz, y, xbc.shape[0])
    _need(xbc.shape[0] == ctx.n_seqs, "ssm step: one token a sequence")
    lib = library.load("ssm")
    _check(lib.de_ssm_walk(_tag(xbc.dtype), 1, xbc.data_ptr(), xbc.stride(0), dt.data_ptr(),
                           dt.stride(0), w.taps.data_ptr(), w.bias.data_ptr(),
                           w.dt_bias.data_ptr(), w.a_log.data_ptr(), None, None,
                           w.skip.data_ptr(), state.data_ptr(), state.stride(0), sz.kept_offset,
                           ctx.seq_slot.data_ptr(), ctx.seq_qstart.data_ptr(),
                           ctx.seq_qlen.data_ptr(), ctx.n_seqs, 1, y.data_ptr(), *sz.tuple(),
                           _stream()), "ssm_step")


def walk(sz: Sizes, w: Weights, ready: torch.Tensor, rates: torch.Tensor, state: torch.Tensor,
         y: torch.Tensor, ctx) -> None:
    """The sequences of at most ``SHORT_PORTION`` tokens, token by token."""
    _rows(sz, ready, rates), _results(sz, y, ready.shape[0]), _state(sz, state)
    lib = library.load("ssm")
    _check(lib.de_ssm_walk(_tag(torch.float32), 0, None, 0, None, 0, None, None, None,
                           w.a_log.data_ptr(), ready.data_ptr(), rates.data_ptr(),
                           w.skip.data_ptr(), state.data_ptr(), state.stride(0), sz.kept_offset,
                           ctx.seq_slot.data_ptr(), ctx.seq_qstart.data_ptr(),
                           ctx.seq_qlen.data_ptr(), ctx.n_seqs, SHORT_PORTION, y.data_ptr(),
                           *sz.tuple(), _stream()), "ssm_walk")


def _products(sz: Sizes, products: torch.Tensor, items: int) -> None:
    _need(products.dtype == torch.float32 and products.is_contiguous()
          and products.shape == (items, sz.groups, CHUNK, CHUNK),
          "ssm chunks: products float32 [items, G, CHUNK, CHUNK]")


def chunk_state(sz: Sizes, ready: torch.Tensor, rates: torch.Tensor, items: torch.Tensor,
                states: torch.Tensor, decays: torch.Tensor, products: torch.Tensor) -> None:
    """What every chunk adds to the state by itself: states [items, state_size] and how much of
    the state before it is left at its end, decays [items, H]; and its tokens' c . b, products
    [items, G, CHUNK, CHUNK].  items int32 [items, 4]: (sequence, first token, tokens, 0)."""
    _rows(sz, ready, rates), _i32(items, "items")
    m = items.shape[0]
    _need(items.shape == (m, 4) and states.dtype == decays.dtype == torch.float32
          and states.is_contiguous() and decays.is_contiguous()
          and states.shape == (m, sz.state_size) and decays.shape == (m, sz.heads),
          "ssm chunks: items [m, 4], states [m, H N P], decays [m, H]")
    _products(sz, products, m)
    lib = library.load("ssm")
    _check(lib.de_ssm_chunk_state(ready.data_ptr(), rates.data_ptr(), items.data_ptr(), m,
                                  states.data_ptr(), decays.data_ptr(), products.data_ptr(),
                                  *sz.tuple(), _stream()), "ssm_chunk_state")


def chunk_pass(sz: Sizes, states: torch.Tensor, decays: torch.Tensor, portions: torch.Tensor,
               state: torch.Tensor, ctx) -> None:
    """states become the states at the chunks' starts, the slots keep the last ones.  portions
    int32 [.., 4]: (sequence, its first chunk, chunks, 0)."""
    _state(sz, state), _i32(portions, "portions")
    lib = library.load("ssm")
    _check(lib.de_ssm_chunk_pass(states.data_ptr(), decays.data_ptr(), portions.data_ptr(),
                                 portions.shape[0], ctx.seq_slot.data_ptr(), state.data_ptr(),
                                 state.stride(0), sz.heads, sz.state_dim, sz.value_dim, _stream()),
           "ssm_chunk_pass")


def chunk_out(sz: Sizes, w: Weights, ready: torch.Tensor, rates: torch.Tensor,
              items: torch.Tensor, states: torch.Tensor, products: torch.Tensor,
              y: torch.Tensor) -> None:
    """The read-outs of the chunks' tokens from the states at the chunks' starts and the tokens'
    c . b."""
    _products(sz, products, items.shape[0])
    _rows(sz, ready, rates), _results(sz, y, ready.shape[0]), _i32(items, "items")
    lib = library.load("ssm")
    _check(lib.de_ssm_chunk_out(ready.data_ptr(), rates.data_ptr(), items.data_ptr(),
                                items.shape[0], states.data_ptr(), products.data_ptr(), w.skip.data_ptr(), y.data_ptr(),
                                *sz.tuple(), _stream()), "ssm_chunk_out")


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, parts: int,
                     eps: float, out: torch.Tensor, ctx,
                     keep: "tuple[Sizes, torch.Tensor, torch.Tensor] | None" = None) -> None:
    """out = y silu(z), every one of ``parts`` equal pieces of a row over its own root mean square
    (eps inside the root), times weight.  y float32 [N, cols], z and out [N, cols] of one dtype.
    ``keep`` = (sizes, xbc, state): the slots' kept convolution inputs also move on; the kernels
    that read the old ones have been launched before."""
    n, cols = y.shape
    _need(y.dtype == weight.dtype == torch.float32 and y.is_contiguous() and weight.is_contiguous()
          and weight.shape == (cols,) and z.shape == out.shape == (n, cols) and z.stride(1) == 1
          and out.is_contiguous() and z.dtype == out.dtype and cols % parts == 0,
          "gated_group_norm: y float32, z and out [N, cols], weight [cols], parts divide cols")
    extra = (None, 0, 0, 0, 0, None, 0)
    if keep is not None:
        sz, xbc, state = keep
        _state(sz, state)
        _need(xbc.stride(1) == 1 and xbc.shape == (n, sz.channels) and xbc.dtype == z.dtype,
              "gated_group_norm: xbc [N, C] of z's dtype")
        extra = (xbc.data_ptr(), xbc.stride(0), sz.channels, sz.taps, sz.kept_offset,
                 state.data_ptr(), state.stride(0))
    lib = library.load("ssm")
    _check(lib.de_gated_group_norm(_tag(z.dtype), y.data_ptr(), z.data_ptr(), z.stride(0),
                                   weight.data_ptr(), out.data_ptr(), n, cols, parts, float(eps),
                                   *extra, ctx.token_seq.data_ptr(), ctx.positions.data_ptr(),
                                   ctx.seq_pos0.data_ptr(), ctx.seq_qlen.data_ptr(),
                                   ctx.seq_slot.data_ptr(), _stream()), "gated_group_norm")
