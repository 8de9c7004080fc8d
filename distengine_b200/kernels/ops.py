"""The kernels as functions of torch tensors.  Every function launches on the current CUDA stream
and checks shapes, dtypes and strides before it passes pointers on; a size that a kernel does not
take is refused with an error that names it.  Nothing here falls back to the CPU or to library
model code.
"""

from __future__ import annotations

import os

import torch

from . import library
from .library import KernelsUnavailable

F32, BF16 = 0, 1

# how many kernels of this package were launched (bench.py reports it)
launch_count = 0


def _tag(dtype: torch.dtype) -> int:
    if dtype == torch.float32:
        return F32
    if dtype == torch.bfloat16:
        return BF16
    raise TypeError(f"kernels take float32 or bfloat16 tensors, got {dtype}")


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


def _stream() -> int:
    """The current CUDA stream's handle.  Every launch asks for it, so it takes the short way
    (a step of a few hundred launches spent more time in ``torch.cuda.current_stream()`` than in
    anything else on the host); it follows stream switches such as a graph capture."""
    if _raw_stream is not None:
        return _raw_stream(torch.cuda.current_device())
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: "torch.Tensor | None") -> int | None:
    return None if t is None else t.data_ptr()


def _check(code: int, what: str) -> None:
    global launch_count
    launch_count += 1
    if code == 0:
        return
    if code < 0:
        raise ValueError(f"{what}: the kernel refuses these sizes (code {code})")
    raise RuntimeError(f"{what}: CUDA error {code} at launch")


def _need(cond: bool, message: str) -> None:
    if not cond:
        raise ValueError(message)


def require_device(device: "torch.device | str") -> torch.device:
    """The CUDA device to run on; raises if there is none."""
    device = torch.device(device)
    if device.type != "cuda":
        raise KernelsUnavailable(f"distengine_b200 runs on a CUDA device only, got '{device}'")
    if not torch.cuda.is_available():
        raise KernelsUnavailable("distengine_b200 needs a CUDA device (sm_100a) and none is "
                                 "visible; there is no CPU path")
    return device


def _i32(t: torch.Tensor, name: str) -> None:
    _need(t.dtype == torch.int32 and t.is_contiguous() and t.is_cuda,
          f"{name} must be a contiguous int32 CUDA tensor")


# ------------------------------------------------------------------------------- embedding
def embed_rows(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor,
               scale: float = 1.0) -> None:
    """out[n] = float32(table[ids[n]]) * scale; ids int32 [N], table [V, H], out float32 [N, H]."""
    _i32(ids, "ids")
    n, (vocab, width) = ids.shape[0], table.shape
    _need(table.is_contiguous() and out.is_contiguous() and out.dtype == torch.float32
          and tuple(out.shape) == (n, width), "embed_rows: out must be float32 [N, H]")
    lib = library.load("core")
    _check(lib.de_embed_rows(_tag(table.dtype), ids.data_ptr(), table.data_ptr(), out.data_ptr(),
                             n, width, vocab, float(scale), _stream()), "embed_rows")


# ------------------------------------------------------------------------------- norm
def add_rmsnorm(resid: torch.Tensor, delta: "torch.Tensor | None", weight: torch.Tensor,
                eps: float, out: torch.Tensor, rows: "torch.Tensor | None" = None,
                groups: int = 1) -> None:
    """out = rmsnorm(resid + delta) * weight; resid (float32) takes the sum unless ``rows`` picks
    the rows to normalise (then out[i] comes from row rows[i] and resid is not written).
    ``groups`` > 1: every one of that many equal parts of a row has its own root mean square."""
    width = resid.shape[1]
    n_out = resid.shape[0] if rows is None else rows.shape[0]
    _need(resid.dtype == torch.float32 and resid.is_contiguous(), "resid must be float32")
    _need(out.is_contiguous() and tuple(out.shape) == (n_out, width), "add_rmsnorm: out shape")
    _need(weight.is_contiguous() and weight.shape == (width,), "add_rmsnorm: weight shape")
    if delta is not None:
        _need(delta.dtype == out.dtype and delta.is_contiguous()
              and delta.shape == resid.shape, "add_rmsnorm: delta must match resid's shape and "
              "the output's dtype")
    if rows is not None:
        _i32(rows, "rows")
    lib = library.load("core")
    if groups != 1:
        _need(groups > 0 and width % groups == 0, "add_rmsnorm: groups must divide the width")
        _check(lib.de_add_rmsnorm_grouped(_tag(out.dtype), _tag(weight.dtype), resid.data_ptr(),
                                          _ptr(delta), weight.data_ptr(), out.data_ptr(),
                                          _ptr(rows), n_out, width, groups, float(eps),
                                          _stream()), "add_rmsnorm (grouped)")
        return
    _check(lib.de_add_rmsnorm(_tag(out.dtype), _tag(weight.dtype), resid.data_ptr(), _ptr(delta),
                              weight.data_ptr(), out.data_ptr(), _ptr(rows), n_out, width,
                              float(eps), _stream()), "add_rmsnorm")


def add_layernorm(resid: torch.Tensor, delta: "torch.Tensor | None", weight: torch.Tensor,
                  bias: torch.Tensor, eps: float, out: torch.Tensor,
                  rows: "torch.Tensor | None" = None) -> None:
    """out = (x - mean(x)) / sqrt(var(x) + eps) * weight + bias with x = resid + delta; resid
    (float32) takes the sum unless ``rows`` picks the rows to normalise, as in ``add_rmsnorm``."""
    width = resid.shape[1]
    n_out = resid.shape[0] if rows is None else rows.shape[0]
    _need(resid.dtype == torch.float32 and resid.is_contiguous(), "resid must be float32")
    _need(out.is_contiguous() and tuple(out.shape) == (n_out, width), "add_layernorm: out shape")
    _need(weight.is_contiguous() and weight.shape == (width,) and bias.is_contiguous()
          and bias.shape == (width,) and bias.dtype == weight.dtype,
          "add_layernorm: weight and bias must be [width] of one dtype")
    if delta is not None:
        _need(delta.dtype == out.dtype and delta.is_contiguous()
              and delta.shape == resid.shape, "add_layernorm: delta must match resid's shape and "
              "the output's dtype")
    if rows is not None:
        _i32(rows, "rows")
    lib = library.load("core")
    _check(lib.de_add_layernorm(_tag(out.dtype), _tag(weight.dtype), resid.data_ptr(),
                                _ptr(delta), weight.data_ptr(), bias.data_ptr(), out.data_ptr(),
                                _ptr(rows), n_out, width, float(eps), _stream()), "add_layernorm")


# ------------------------------------------------------------------------------- element-wise
ACTIVATIONS = {"relu2": 0, "tanh": 1, "silu": 2, "gelu_tanh": 3, "gelu_erf": 4}


def activation(x: torch.Tensor, out: torch.Tensor, kind: str) -> None:
    """out = act(x) element by element (float32 arithmetic): ``relu2`` the square of relu,
    ``tanh``, ``silu``, ``gelu_tanh``, ``gelu_erf`` (the exact form).  x and out [N, cols] with free row strides; out may be x."""
    _need(kind in ACTIVATIONS, f"activation: unknown kind '{kind}'; known: {sorted(ACTIVATIONS)}")
    _need(x.dim() == 2 and x.shape == out.shape and x.dtype == out.dtype and x.stride(1) == 1
          and out.stride(1) == 1, "activation: x and out [N, cols] of one dtype")
    lib = library.load("core")
    _check(lib.de_activation(_tag(x.dtype), x.data_ptr(), x.stride(0), out.data_ptr(),
                             out.stride(0), x.shape[0], x.shape[1], ACTIVATIONS[kind], _stream()),
           "activation")


def softcap_(x: torch.Tensor, cap: float) -> None:
    """x <- cap * tanh(x / cap) in place; x float32, contiguous."""
    _need(x.dtype == torch.float32 and x.is_contiguous() and cap > 0, "softcap_: float32, cap > 0")
    lib = library.load("core")
    _check(lib.de_softcap(x.data_ptr(), x.numel(), float(cap), _stream()), "softcap")


def scaled_sum(a: torch.Tensor, b: torch.Tensor, sa: float, sb: float, out: torch.Tensor) -> None:
    """out = sa * a + sb * b; a, b float32, out of any kernel dtype, all contiguous of one shape."""
    _need(a.dtype == b.dtype == torch.float32 and a.shape == b.shape == out.shape
          and a.is_contiguous() and b.is_contiguous() and out.is_contiguous(),
          "scaled_sum: a, b float32 and out, contiguous and of one shape")
    lib = library.load("core")
    _check(lib.de_scaled_sum(_tag(out.dtype), a.data_ptr(), b.data_ptr(), float(sa), float(sb),
                             out.data_ptr(), out.numel(), _stream()), "scaled_sum")


def residual_add(resid: torch.Tensor, a: "torch.Tensor | None", b: "torch.Tensor | None" = None,
                 extra: "torch.Tensor | None" = None,
                 rows: "torch.Tensor | None" = None) -> None:
    """resid += (a + b) + extra in float32: ``a`` and ``b`` are branch outputs (bfloat16 or
    float32, either may be None), ``extra`` is float32; ``rows`` receives the new residual in its
    own dtype.  All contiguous and of resid's shape."""
    _need(resid.dtype == torch.float32 and resid.is_contiguous(), "residual_add: resid float32")
    for t in (a, b, extra, rows):
        _need(t is None or (t.is_contiguous() and t.shape == resid.shape),
              "residual_add: operands are contiguous and of resid's shape")
    _need(extra is None or extra.dtype == torch.float32, "residual_add: extra is float32")
    if a is None and b is None and extra is None and rows is None:
        return
    lib = library.load("core")
    _check(lib.de_residual_add(resid.data_ptr(), 0 if a is None else _tag(a.dtype), _ptr(a),
                               0 if b is None else _tag(b.dtype), _ptr(b), _ptr(extra),
                               0 if rows is None else _tag(rows.dtype), _ptr(rows),
                               resid.numel(), _stream()), "residual_add")


def act_mul(x: torch.Tensor, out: torch.Tensor, kind: str) -> None:
    """out[n, i] = act(x[n, i]) * x[n, inner + i]; x [N, 2 inner], out [N, inner]."""
    n, inner = out.shape
    _need(kind in ACTIVATIONS, f"act_mul: unknown kind '{kind}'")
    _need(x.stride(1) == 1 and out.stride(1) == 1 and x.shape == (n, 2 * inner)
          and x.dtype == out.dtype, "act_mul: x must be [N, 2 inner] and out [N, inner]")
    lib = library.load("core")
    _check(lib.de_act_mul(_tag(x.dtype), x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0),
                          n, inner, ACTIVATIONS[kind], _stream()), "act_mul")


def act_mul_row(z: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor,
                kind: str) -> None:
    """out[n, i] = act(z[n, i]) * table[ids[n], i]; z, out [N, dim], table [V, dim]."""
    n, dim = out.shape
    _i32(ids, "ids")
    _need(kind in ACTIVATIONS, f"act_mul_row: unknown kind '{kind}'")
    _need(z.shape == out.shape and z.stride(1) == 1 and out.stride(1) == 1
          and table.is_contiguous() and table.dim() == 2 and table.shape[1] == dim
          and z.dtype == out.dtype == table.dtype and ids.shape == (n,),
          "act_mul_row: z, out [N, dim] and table [V, dim] of one dtype")
    lib = library.load("core")
    _check(lib.de_act_mul_row(_tag(z.dtype), z.data_ptr(), z.stride(0), ids.data_ptr(),
                              table.data_ptr(), table.shape[0], out.data_ptr(), out.stride(0), n,
                              dim, ACTIVATIONS[kind], _stream()), "act_mul_row")


def add_normed(resid: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float) -> None:
    """resid += y / sqrt(mean(y^2) + eps) * weight row by row, in float32."""
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and y.is_contiguous()
          and y.shape == resid.shape and weight.is_contiguous()
          and weight.shape == (resid.shape[1],), "add_normed: resid float32, y and weight")
    lib = library.load("core")
    _check(lib.de_add_normed(_tag(y.dtype), _tag(weight.dtype), resid.data_ptr(), y.data_ptr(),
                             weight.data_ptr(), resid.shape[0], resid.shape[1], float(eps),
                             _stream()), "add_normed")


def rmsnorm_cols(x: torch.Tensor, weight: torch.Tensor, eps: float, out: torch.Tensor) -> None:
    """out = x / sqrt(mean(x^2) + eps) * weight over the columns of x [N, cols] (row strides
    free: x may be a block of columns of a product's output)."""
    _need(x.dim() == 2 and x.shape == out.shape and x.stride(1) == 1 and out.stride(1) == 1
          and x.dtype == out.dtype and weight.is_contiguous() and weight.shape == (x.shape[1],),
          "rmsnorm_cols: x, out [N, cols] of one dtype and weight [cols]")
    lib = library.load("core")
    _check(lib.de_rmsnorm_cols(_tag(x.dtype), _tag(weight.dtype), x.data_ptr(), x.stride(0),
                               weight.data_ptr(), out.data_ptr(), out.stride(0), x.shape[0],
                               x.shape[1], float(eps), _stream()), "rmsnorm_cols")


# ------------------------------------------------------------------------------- rotation + cache write
def _wtag(weight: torch.Tensor) -> int:
    _need(weight.dtype in (torch.float32, torch.bfloat16) and weight.is_contiguous(),
          "a norm's weight is contiguous float32 or bfloat16")
    return _tag(weight.dtype)


def norm_stream(resid: torch.Tensor, weight: torch.Tensor, eps: float,
                rows: "torch.Tensor | None" = None) -> None:
    """resid <- resid / sqrt(mean(resid^2) + eps) * weight row by row, in place on the float32
    stream; ``rows`` [N, width] (bfloat16 or float32) also receives the result, rounded."""
    n, width = resid.shape
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and weight.shape == (width,),
          "norm_stream: resid float32 [N, width], weight [width]")
    _need(rows is None or (rows.is_contiguous() and rows.shape == resid.shape),
          "norm_stream: rows [N, width]")
    lib = library.load("sublayer")
    _check(lib.de_norm_stream(_tag(rows.dtype) if rows is not None else 0, _wtag(weight),
                              resid.data_ptr(), weight.data_ptr(), _ptr(rows), n, width,
                              float(eps), _stream()), "norm_stream")


def gated_normed_add(y: torch.Tensor, gate: torch.Tensor, bias: torch.Tensor, weight: torch.Tensor,
                     eps: float, resid: torch.Tensor, out: torch.Tensor,
                     rows: "torch.Tensor | None" = None) -> None:
    """out = resid + g / sqrt(mean(g^2) + eps) * weight with g = y * sigmoid(gate + bias), row by
    row in float32.  y [N, width] (the gate's dtype or float32), gate [N, width] (row stride
    free), bias float32 [width]; resid and out float32 [N, width] (the same tensor or two);
    ``rows`` of gate's dtype also receives out, rounded."""
    n, width = out.shape
    _need(resid.dtype == out.dtype == bias.dtype == torch.float32 and resid.is_contiguous()
          and out.is_contiguous() and resid.shape == out.shape and bias.shape == (width,)
          and bias.is_contiguous() and weight.shape == (width,),
          "gated_normed_add: resid, out float32 [N, width], bias and weight [width]")
    _need(y.is_contiguous() and y.shape == out.shape and gate.shape == out.shape
          and gate.stride(1) == 1 and y.dtype in (gate.dtype, torch.float32),
          "gated_normed_add: y and gate [N, width]")
    _need(rows is None or (rows.is_contiguous() and rows.shape == out.shape
                           and rows.dtype == gate.dtype), "gated_normed_add: rows [N, width]")
    lib = library.load("sublayer")
    _check(lib.de_gated_normed_add(_tag(gate.dtype), _tag(y.dtype), _wtag(weight), y.data_ptr(),
                                   gate.data_ptr(), gate.stride(0), bias.data_ptr(),
                                   weight.data_ptr(), resid.data_ptr(), out.data_ptr(), _ptr(rows),
                                   n, width, float(eps), _stream()), "gated_normed_add")


def join_rmsnorm(resid: torch.Tensor, y: "torch.Tensor | None", branch_norm=None,
                 vector: "torch.Tensor | None" = None, norm=None,
                 out: "torch.Tensor | None" = None, rows: "torch.Tensor | None" = None) -> None:
    """resid += y / sqrt(mean(y^2) + eps) * weight + vector row by row in float32, with weight and
    eps of ``branch_norm`` (None: y as it is), y [N, width] (None: no branch) and vector float32
    [width] (None: none); y may also be the terms of a weighted sum (``parts.context.MixedRows``:
    ``rows`` [N top, width], ``weight`` [N, top], ``shared``, ``side``).  Then, with ``out``, out =
    the RMS norm ``norm`` of the new rows, or the new rows themselves (rounded) without ``norm``.
    ``rows`` (int32): out[i] is the norm of row rows[i], and resid stays as it is."""
    n, width = resid.shape
    mix = (None, 0, None, None)
    if y is not None and not isinstance(y, torch.Tensor):
        weight, shared, side, y = y.weight, y.shared, y.side, y.rows
        top = weight.shape[1]
        _need(weight.dtype == torch.float32 and weight.is_contiguous()
              and weight.shape == (n, top) and y.shape == (n * top, width) and y.is_contiguous()
              and (shared is None or (
                  shared.dtype == y.dtype and shared.is_contiguous()
                  and shared.shape == resid.shape and side.dtype == torch.float32
                  and side.shape == (n,) and side.is_contiguous())),
              "join_rmsnorm: rows [N top, width], weight [N, top], shared [N, width], side [N]")
        mix = (weight.data_ptr(), top, _ptr(shared), _ptr(side) if shared is not None else None)
    elif y is not None:
        _need(y.is_contiguous() and y.shape == resid.shape, "join_rmsnorm: y [N, width]")
    _need(resid.dtype == torch.float32 and resid.is_contiguous(), "join_rmsnorm: resid float32")
    _need(vector is None or (vector.dtype == torch.float32 and vector.is_contiguous()
                             and vector.shape == (width,)), "join_rmsnorm: vector float32 [width]")
    _need((norm is None or out is not None) and (rows is None or norm is not None),
          "join_rmsnorm: a norm has an output, and picked rows a norm")
    if y is None:
        branch_norm = None
    n_out = n
    if out is not None:
        n_out = out.shape[0]
        _need(out.is_contiguous() and out.shape[1] == width
              and n_out == (n if rows is None else rows.shape[0]), "join_rmsnorm: out [.., width]")
    if rows is not None:
        _i32(rows, "rows")
    weights = [w.weight for w in (branch_norm, norm) if w is not None]
    for w in weights:
        _need(w.shape == (width,) and _wtag(w) == _wtag(weights[0]),
              "join_rmsnorm: both weights [width] of one dtype")
    y_dtype = torch.float32 if y is None else y.dtype
    dtype = out.dtype if out is not None else torch.bfloat16
    lib = library.load("sublayer")
    _check(lib.de_join_rmsnorm(
        _tag(dtype), _tag(y_dtype), _wtag(weights[0]) if weights else 0, resid.data_ptr(), _ptr(y),
        *mix, None if branch_norm is None else branch_norm.weight.data_ptr(),
        0.0 if branch_norm is None else float(branch_norm.eps), _ptr(vector),
        None if norm is None else norm.weight.data_ptr(), 0.0 if norm is None else float(norm.eps),
        _ptr(out), _ptr(rows), n_out, width, _stream()), "join_rmsnorm")


def depth_mix(history: torch.Tensor, coef: torch.Tensor, out: torch.Tensor,
              rows: "torch.Tensor | None" = None) -> None:
    """out = sum_j coef[j] * history[j]; history float32 [count, N, width] (contiguous), coef
    float32 [count], out float32 [N, width]; ``rows`` also receives out, rounded."""
    count = history.shape[0]
    _need(history.dtype == out.dtype == coef.dtype == torch.float32 and history.is_contiguous()
          and out.is_contiguous() and tuple(history.shape[1:]) == tuple(out.shape)
          and coef.shape == (count,) and coef.is_contiguous(),
          "depth_mix: history float32 [count, N, width], coef [count], out [N, width]")
    _need(rows is None or (rows.is_contiguous() and rows.shape == out.shape),
          "depth_mix: rows [N, width]")
    lib = library.load("sublayer")
    _check(lib.de_depth_mix(_tag(rows.dtype) if rows is not None else 0, history.data_ptr(),
                            out.numel(), coef.data_ptr(), count, out.numel(), out.data_ptr(),
                            _ptr(rows), _stream()), "depth_mix")


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float, out: torch.Tensor) -> None:
    """out = a N(z) + b N(z^2) + c N(z^3) + e with coef = (a, b, c, e) float32 on the device and N
    dividing a row by its root mean square (eps inside the root); float32 arithmetic."""
    _need(z.dim() == 2 and z.stride(1) == 1 and out.stride(1) == 1 and out.shape == z.shape
          and out.dtype == z.dtype and coef.dtype == torch.float32 and coef.shape == (4,),
          "poly_norm: z and out [N, cols] of one dtype, coef float32 [4]")
    lib = library.load("sublayer")
    _check(lib.de_poly_norm(_tag(z.dtype), z.data_ptr(), z.stride(0), coef.data_ptr(),
                            out.data_ptr(), out.stride(0), z.shape[0], z.shape[1], float(eps),
                            _stream()), "poly_norm")


def rope_kv_write(qkv: torch.Tensor, positions: torch.Tensor, token_slot: torch.Tensor,
                  inv_freq: "torch.Tensor | None", rotary_dim: int, heads: int, kv_heads: int,
                  head_dim: int, k_pages: torch.Tensor, v_pages: torch.Tensor,
                  block_table: torch.Tensor, write_kv: bool, status: torch.Tensor) -> None:
    """Rotate q and k of qkv [N, (heads + 2 kv_heads) * d] in place by position and store k, v in
    the pages [pages, kv_heads, page, d] through block_table [slots, max_pages]."""
    n = qkv.shape[0]
    _need(qkv.stride(1) == 1 and qkv.shape[1] == (heads + 2 * kv_heads) * head_dim,
          "rope_kv_write: qkv must be [N, (heads + 2 kv_heads) * head_dim]")
    _i32(positions, "positions"), _i32(token_slot, "token_slot"), _i32(block_table, "block_table")
    _i32(status, "status")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.shape == v_pages.shape
          and k_pages.dtype == qkv.dtype == v_pages.dtype and k_pages.dim() == 4
          and k_pages.shape[1] == kv_heads and k_pages.shape[3] == head_dim,
          "rope_kv_write: pages must be [pages, kv_heads, page, head_dim] of qkv's dtype")
    _need(rotary_dim % 2 == 0 and 0 <= rotary_dim <= head_dim,
          f"rope_kv_write: rotary_dim {rotary_dim} must be even and at most head_dim {head_dim}")
    if inv_freq is not None:
        _need(inv_freq.dtype == torch.float32 and inv_freq.is_contiguous()
              and inv_freq.shape == (rotary_dim // 2,), "rope_kv_write: inv_freq shape")
    lib = library.load("core")
    _check(lib.de_rope_kv_write(_tag(qkv.dtype), qkv.data_ptr(), qkv.stride(0),
                                positions.data_ptr(), token_slot.data_ptr(), _ptr(inv_freq),
                                rotary_dim, heads, kv_heads, head_dim, k_pages.data_ptr(),
                                v_pages.data_ptr(), block_table.data_ptr(), block_table.stride(0),
                                k_pages.shape[2], int(write_kv), k_pages.shape[0], n,
                                status.data_ptr(), _stream()), "rope_kv_write")


# ------------------------------------------------------------------------------- feed-forward
def silu_mul(x: torch.Tensor, out: torch.Tensor) -> None:
    """out[n, i] = silu(x[n, i]) * x[n, inner + i]; x [N, 2 inner], out [N, inner]."""
    n, inner = out.shape
    _need(x.is_contiguous() and out.is_contiguous() and x.shape == (n, 2 * inner)
          and x.dtype == out.dtype, "silu_mul: x must be [N, 2 inner] and out [N, inner]")
    lib = library.load("core")
    _check(lib.de_silu_mul(_tag(x.dtype), x.data_ptr(), out.data_ptr(), n, inner, _stream()),
           "silu_mul")


# ------------------------------------------------------------------------------- matrix products
def gemm_f32(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """out[n, m] = sum_k x[n, k] w[m, k] in IEEE float32 on the CUDA cores."""
    _need(x.dtype == w.dtype == out.dtype == torch.float32, "gemm_f32 takes float32 tensors")
    _need(x.dim() == 2 and w.dim() == 2 and x.shape[1] == w.shape[1]
          and tuple(out.shape) == (x.shape[0], w.shape[0]), "gemm_f32: shapes do not agree")
    _need(x.stride(1) == 1 and w.stride(1) == 1 and out.stride(1) == 1,
          "gemm_f32: rows must be contiguous")
    lib = library.load("gemm_f32")
    _check(lib.de_gemm_f32(x.data_ptr(), w.data_ptr(), out.data_ptr(), x.shape[0], w.shape[0],
                           x.shape[1], x.stride(0), w.stride(0), out.stride(0), _stream()),
           "gemm_f32")


# Up to this many tokens a product streams the weights through linear_small (the kernel takes up
# to 32; measured on B200 in decode steps, the library product is faster from 17 rows on: batch
# 24: 1.17 against 1.42 ms a step, batch 32: 1.21 against 1.56; at 12 rows linear_small wins).
SMALL_ROWS = int(os.environ.get("DISTENGINE_B200_SMALL_ROWS", "16"))


def _small_ok(x: torch.Tensor, w: torch.Tensor) -> bool:
    return (0 < x.shape[0] <= SMALL_ROWS and x.shape[1] % 8 == 0 and x.stride(1) == 1
            and w.is_contiguous() and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0
            and w.data_ptr() % 16 == 0)


# The RMS norm between two weight-streaming products can ride on them (``csrc/linear_small.cu``):
# the product before it adds to the residual and leaves residual * norm weight plus shares of the
# rows' sums of squares, the product after it applies the rows' factors to its sums.
# DISTENGINE_B200_NORM_RIDE=0 keeps the norm a kernel of its own (for measurements).
NORM_RIDE = os.environ.get("DISTENGINE_B200_NORM_RIDE", "1") != "0"
NORM_RIDE_ROWS = 16


# From SMALL_ROWS + 1 to this many tokens a product goes to the swapped-operand tcgen05 kernel
# (``csrc/linear_mid.cu``, which takes up to 128); DISTENGINE_B200_MID_ROWS=0 gives those to the
# library product.  Measured on B200 in decode steps (TinyLlama shape, a step in ms, this kernel
# against the library product with separate norm and activation kernels): batch 20 1.12 / 1.16,
# batch 32 1.18 / 1.20, batch 48 1.36 / 1.28, batch 64 1.42 / 1.33.
MID_ROWS = int(os.environ.get("DISTENGINE_B200_MID_ROWS", "32"))


def _mid_ok(x: torch.Tensor, w: torch.Tensor) -> bool:
    return (SMALL_ROWS < x.shape[0] <= MID_ROWS and x.shape[1] % 8 == 0 and x.stride(1) == 1
            and w.is_contiguous() and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0
            and w.data_ptr() % 16 == 0)


def _linear_mid(x, w, out, gated, before, after, status) -> None:
    global _tcgen05_status
    n_out = w.shape[0] // 2 if gated else w.shape[0]
    _need(out.dtype in (torch.bfloat16, torch.float32) and out.stride(1) == 1
          and tuple(out.shape) == (x.shape[0], n_out), "linear_mid: out [tokens, n]")
    if status is None:
        if _tcgen05_status is None or _tcgen05_status.device != x.device:
            _tcgen05_status = torch.zeros(1, dtype=torch.int32, device=x.device)
        status = _tcgen05_status
    in_parts = in_count = width = 0
    eps = 0.0
    if before is not None:
        parts = before.parts
        _need(parts.dtype == torch.float32 and parts.is_contiguous()
              and parts.shape[0] == x.shape[0], "linear: before.parts must be float32 [rows, count]")
        in_parts, in_count, width, eps = parts.data_ptr(), parts.shape[1], before.width, before.eps
    resid = ld_resid = weight = out_parts = 0
    lib = library.load("linear_mid")
    if after is not None:
        _need(after.resid.dtype == torch.float32 and after.resid.stride(1) == 1
              and tuple(after.resid.shape) == tuple(out.shape) and out.dtype == torch.bfloat16
              and after.weight.dtype == torch.bfloat16 and after.weight.is_contiguous()
              and after.weight.shape == (n_out,) and after.parts.dtype == torch.float32
              and after.parts.is_contiguous()
              and tuple(after.parts.shape) == (x.shape[0], lib.de_linear_mid_parts(n_out)),
              "linear: after needs resid float32 [rows, n], weight bfloat16 [n] and parts "
              "float32 [rows, norm_ride_parts(...)]")
        resid, ld_resid = after.resid.data_ptr(), after.resid.stride(0)
        weight, out_parts = after.weight.data_ptr(), after.parts.data_ptr()
    _check(lib.de_linear_mid(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(),
                             out.stride(0), x.shape[0], n_out, x.shape[1],
                             int(out.dtype == torch.float32), int(gated), in_parts, in_count,
                             int(width), float(eps), resid, ld_resid, weight, out_parts, 0,
                             status.data_ptr(), _stream()), "linear_mid")


def norm_ride_parts(rows: int, w: torch.Tensor, dtype: torch.dtype) -> int:
    """How many shares of every row's sum of squares a product of ``rows`` rows against ``w``
    leaves when it does the following norm's work (``linear(..., after=)``), or 0 if such a
    product does not go to the weight-streaming kernel.  The same condition says whether a product
    against ``w`` can apply a preceding norm's row factors (``linear(..., before=)``)."""
    if not (NORM_RIDE and dtype == torch.bfloat16 and w.dtype == torch.bfloat16
            and w.shape[1] % 8 == 0 and w.is_contiguous() and w.data_ptr() % 16 == 0):
        return 0
    if 0 < rows <= min(SMALL_ROWS, NORM_RIDE_ROWS):
        return int(library.load("linear_small").de_linear_small_parts(w.shape[0]))
    if SMALL_ROWS < rows <= MID_ROWS:
        return int(library.load("linear_mid").de_linear_mid_parts(w.shape[0]))
    return 0


def _linear_small_norm(x, w, out, gated, before, after, status=None) -> None:
    if _mid_ok(x, w):
        _linear_mid(x, w, out, gated, before, after, status)
        return
    n_out = w.shape[0] // 2 if gated else w.shape[0]
    _need(_small_ok(x, w) and x.shape[0] <= NORM_RIDE_ROWS and out.dtype == torch.bfloat16
          and out.stride(1) == 1, "linear: a product that carries a norm must be one the "
          "weight-streaming kernel takes (see norm_ride_parts)")
    in_parts = in_count = width = 0
    eps = 0.0
    if before is not None:
        parts = before.parts
        _need(parts.dtype == torch.float32 and parts.is_contiguous()
              and parts.shape[0] == x.shape[0], "linear: before.parts must be float32 [rows, count]")
        in_parts, in_count, width, eps = parts.data_ptr(), parts.shape[1], before.width, before.eps
    resid = ld_resid = weight = out_parts = 0
    if after is not None:
        lib_parts = norm_ride_parts(x.shape[0], w, x.dtype)
        _need(after.resid.dtype == torch.float32 and after.resid.stride(1) == 1
              and tuple(after.resid.shape) == tuple(out.shape)
              and after.weight.dtype == torch.bfloat16 and after.weight.is_contiguous()
              and after.weight.shape == (n_out,) and after.parts.dtype == torch.float32
              and after.parts.is_contiguous()
              and tuple(after.parts.shape) == (x.shape[0], lib_parts),
              "linear: after needs resid float32 [rows, n], weight bfloat16 [n] and parts "
              "float32 [rows, norm_ride_parts(...)]")
        resid, ld_resid = after.resid.data_ptr(), after.resid.stride(0)
        weight, out_parts = after.weight.data_ptr(), after.parts.data_ptr()
    lib = library.load("linear_small")
    _check(lib.de_linear_small_norm(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0),
                                    out.data_ptr(), out.stride(0), x.shape[0], n_out, x.shape[1],
                                    int(gated), in_parts, in_count, int(width), float(eps), resid,
                                    ld_resid, weight, out_parts, _stream()),
           "linear_small (with norm)")


TCGEN05_ROWS = 1024     # from this many rows on, products go to this package's tcgen05 kernel
_tile_fits: dict[tuple[int, int], bool] = {}


def _tcgen05_fits(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> bool:
    """Whether a plain product of this shape goes to this package's tcgen05 kernel: many rows, and
    a shape whose tiles fill the SMs in whole rounds with wide tiles.  (Measured on B200 against
    cuBLAS at 2,048 rows: equal or within 4% where this holds, up to a third slower where the
    tiles have to be narrow or the last round is nearly empty; with few rows cuBLAS splits k,
    which this kernel does not.)"""
    m, n = x.shape[0], w.shape[0]
    if (m < TCGEN05_ROWS or x.shape[1] % 8 or x.stride(0) % 8 or w.stride(0) % 8 or x.stride(1) != 1
            or w.stride(1) != 1 or x.data_ptr() % 16 or w.data_ptr() % 16):
        return False
    key = (m, n)
    fits = _tile_fits.get(key)
    if fits is None:
        lib = library.load("gemm_tcgen05")
        bn, sms = lib.de_gemm_tcgen05_tile(m, n, 0), lib.de_gemm_tcgen05_sms()
        tiles = -(-m // 128) * -(-n // bn)
        rounds = -(-tiles // sms)
        fits = _tile_fits[key] = bn >= 192 and m * n >= 0.75 * rounds * sms * 128 * bn
    return fits


def linear(x: torch.Tensor, w: torch.Tensor, out: "torch.Tensor | None" = None,
           out_dtype: "torch.dtype | None" = None,
           status: "torch.Tensor | None" = None, before=None, after=None,
           act: "str | None" = None) -> torch.Tensor:
    """x @ w^T, float32 accumulation.  ``act`` (a key of ``ACTIVATIONS``): the activation that the
    outputs pass, in the weight-streaming kernel's epilogue for steps of up to 16 tokens, as a
    kernel of its own otherwise.

    ``before`` (``.parts`` float32 [rows, count], ``.width``, ``.eps``): x is the output of an RMS
    norm but for the rows' factors rsqrt(sum of the row's parts / width + eps), which the product
    applies to its sums.  ``after`` (``.resid`` float32 [rows, n], ``.weight`` bfloat16 [n],
    ``.parts`` float32 [rows, norm_ride_parts(...)]): the result is added to ``resid`` and ``out``
    becomes resid * weight, ``parts`` the shares of the rows' sums of squares - what ``before``
    of the next product needs.  Both only where ``norm_ride_parts`` is not 0.

    float32: this package's own CUDA-core kernel (true 32-bit).  bfloat16 with up to 16 rows
    (decode steps): this package's weight-streaming kernel (``csrc/linear_small.cu``).  bfloat16
    with a thousand rows or more in a shape that suits it: this package's tcgen05 kernel
    (``csrc/gemm_tcgen05.cu``).  Otherwise the library matrix product (cuBLAS through torch),
    where the reference calls a library too (src/layers/linear.py:19-20).  The output is bfloat16
    or float32.  ``status`` (int32 [1]): where the tcgen05 kernel records a wait that ran out."""
    out_dtype = out_dtype or (out.dtype if out is not None else x.dtype)
    if out is None:
        out = torch.empty((x.shape[0], w.shape[0]), dtype=out_dtype, device=x.device)
    if x.shape[0] == 0:
        return out
    _need(act is None or (act in ACTIVATIONS and before is None and after is None),
          f"linear: act is one of {sorted(ACTIVATIONS)} and goes with no norm")
    if x.dtype == torch.float32:
        _need(out.dtype == torch.float32, "linear: a float32 product has a float32 output")
        _need(before is None and after is None, "linear: float32 products carry no norm")
        gemm_f32(x, w, out)
        if act is not None:
            activation(out, out, act)
        return out
    _need(x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16,
          "linear: operands must both be bfloat16 or both float32")
    _need(x.shape[1] == w.shape[1] and tuple(out.shape) == (x.shape[0], w.shape[0])
          and out.stride(1) == 1, "linear: shapes do not agree")
    if before is not None or after is not None:
        _linear_small_norm(x, w, out, False, before, after, status)
    elif _mid_ok(x, w):
        _linear_mid(x, w, out, False, None, None, status)
    elif _small_ok(x, w):
        lib = library.load("linear_small")
        _check(lib.de_linear_small(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0),
                                   out.data_ptr(), out.stride(0), x.shape[0], w.shape[0],
                                   x.shape[1], int(out.dtype == torch.float32), 0,
                                   0 if act is None else ACTIVATIONS[act] + 1, _stream()),
               "linear_small")
        return out
    elif _tcgen05_fits(x, w, out):
        gemm_tcgen05(x, w, out, status=status)
    elif out.dtype == torch.bfloat16:
        torch.mm(x, w.t(), out=out)
    else:
        torch.mm(x, w.t(), out_dtype=torch.float32, out=out)
    if act is not None:
        activation(out, out, act)
    return out


def gated_needs_scratch(x: torch.Tensor, w_gate_up: torch.Tensor) -> bool:
    """Whether ``linear_gated`` forms the [gate | up] product in memory for these operands: not
    for bfloat16 with up to 16 rows (weight-streaming kernel) or with a thousand rows or more
    (tcgen05 kernel; with fewer rows its tiles leave most SMs idle and the library product plus
    the activation kernel is faster)."""
    if x.dtype != torch.bfloat16 or w_gate_up.dtype != torch.bfloat16:
        return True
    if _small_ok(x, w_gate_up) or _mid_ok(x, w_gate_up):
        return False
    return not (x.shape[0] >= TCGEN05_ROWS and x.shape[1] % 8 == 0 and x.stride(0) % 8 == 0
                and w_gate_up.stride(0) % 8 == 0 and x.stride(1) == 1
                and w_gate_up.stride(1) == 1 and x.data_ptr() % 16 == 0
                and w_gate_up.data_ptr() % 16 == 0)


def linear_gated(x: torch.Tensor, w_gate_up: torch.Tensor, out: torch.Tensor,
                 scratch: "torch.Tensor | None" = None,
                 status: "torch.Tensor | None" = None, before=None) -> torch.Tensor:
    """out[n, i] = silu(x . gate_i) * (x . up_i) for w_gate_up = [gate rows; up rows] of shape
    [2 inner, k].  bfloat16: one kernel whose epilogue applies the activation, the
    weight-streaming one up to 16 rows, the tcgen05 one from 1,024 rows.  float32 (or operands that are not
    16-byte aligned): the product into ``scratch`` [N, 2 inner], then ``silu_mul``."""
    inner = w_gate_up.shape[0] // 2
    _need(tuple(out.shape) == (x.shape[0], inner), "linear_gated: out must be [N, inner]")
    if x.shape[0] == 0:
        return out
    if before is not None:          # x lacks its norm's row factors (see ``linear``)
        _linear_small_norm(x, w_gate_up, out, True, before, None, status)
        return out
    if (x.dtype == torch.bfloat16 and _mid_ok(x, w_gate_up) and out.stride(1) == 1
            and out.dtype == torch.bfloat16):
        _linear_mid(x, w_gate_up, out, True, None, None, status)
        return out
    if x.dtype == torch.bfloat16 and _small_ok(x, w_gate_up) and out.stride(1) == 1:
        lib = library.load("linear_small")
        _check(lib.de_linear_small(x.data_ptr(), x.stride(0), w_gate_up.data_ptr(),
                                   w_gate_up.stride(0), out.data_ptr(), out.stride(0), x.shape[0],
                                   inner, x.shape[1], 0, 1, 0, _stream()), "linear_small (gated)")
        return out
    if not gated_needs_scratch(x, w_gate_up) and out.stride(1) == 1 and out.dtype == x.dtype:
        return gemm_tcgen05(x, w_gate_up, out, gated=True, status=status)
    if scratch is None:
        scratch = torch.empty((x.shape[0], 2 * inner), dtype=x.dtype, device=x.device)
    linear(x, w_gate_up, out=scratch)
    silu_mul(scratch, out)
    return out


_tcgen05_status: "torch.Tensor | None" = None


def gemm_tcgen05(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, gated: bool = False,
                 status: "torch.Tensor | None" = None) -> torch.Tensor:
    """out = x @ w^T on the 5th-generation tensor cores (``csrc/gemm_tcgen05.cu``: TMA loads,
    tcgen05.mma with the accumulator in tensor memory), bfloat16 operands, bfloat16 or float32
    output.  ``gated``: w = [gate rows; up rows] ([2 n, k]) and out [m, n] = silu(gate) * up.
    ``status`` (int32 [1]) receives 3 if a wait inside the kernel ran out."""
    global _tcgen05_status
    n = w.shape[0] // 2 if gated else w.shape[0]
    _need(x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and x.dim() == 2
          and w.dim() == 2 and x.shape[1] == w.shape[1] and tuple(out.shape) == (x.shape[0], n)
          and x.stride(1) == 1 and w.stride(1) == 1 and out.stride(1) == 1,
          "gemm_tcgen05: x [m, k] and w [n, k] bfloat16 with contiguous rows, out [m, n]")
    _need(out.dtype in (torch.bfloat16, torch.float32), "gemm_tcgen05: out bfloat16 or float32")
    if status is None:
        if _tcgen05_status is None or _tcgen05_status.device != x.device:
            _tcgen05_status = torch.zeros(1, dtype=torch.int32, device=x.device)
        status = _tcgen05_status
    lib = library.load("gemm_tcgen05")
    _check(lib.de_gemm_tcgen05(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0),
                               out.data_ptr(), out.stride(0), x.shape[0], n, x.shape[1],
                               int(out.dtype == torch.float32), int(gated), status.data_ptr(),
                               _stream()), "gemm_tcgen05")
    return out


# ------------------------------------------------------------------------------- sampling
def sample_rows(logits: torch.Tensor, out: torch.Tensor,
                temperature: "torch.Tensor | None" = None, seed: "torch.Tensor | None" = None,
                position: "torch.Tensor | None" = None) -> None:
    """out[r] = arg-max of row r (temperature null or 0) or a seeded draw from
    softmax(logits / temperature)."""
    rows, vocab = logits.shape
    _need(logits.dtype == torch.float32 and logits.is_contiguous(), "logits must be float32")
    _i32(out, "out")
    if temperature is not None:
        _need(temperature.dtype == torch.float32 and seed is not None and position is not None
              and seed.dtype == torch.int64 and position.dtype == torch.int32
              and temperature.shape[0] == seed.shape[0] == position.shape[0] == rows,
              "sample_rows: temperature float32, seed int64, position int32, one per row")
    lib = library.load("core")
    _check(lib.de_sample_rows(logits.data_ptr(), rows, vocab, _ptr(temperature), _ptr(seed),
                              _ptr(position), out.data_ptr(), _stream()), "sample_rows")
