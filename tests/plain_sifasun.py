"""A plain, slow implementation of the Sifasun decoder, one function per mechanism, whole sequences
only, in float64 (or float32) on the CPU.  It shares no code with the engine: the engine's parts
and kernels are compared with it.

``act`` (None or torch.bfloat16) models the engine's bfloat16 mode: the results of matrix products,
the rows that enter one, queries, cached keys and values are rounded to it (``rnd``); the residual
stream, norm statistics, angles, scores, softmax weights, the gated recurrence and its gates are
not.

Notation: T tokens, width D.  A weight matrix is stored [out, in]; ``lin`` applies it.  ``w`` maps
tensor names to tensors, ``config`` is the parsed config.json.
"""

from __future__ import annotations

import math

import torch


def rnd(x: torch.Tensor, act) -> torch.Tensor:
    return x if act is None else x.to(act).to(x.dtype)


def lin(x: torch.Tensor, weight: torch.Tensor, act=None) -> torch.Tensor:
    return rnd(rnd(x, act) @ weight.to(x.dtype).t(), act)


def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def plus_one_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """The model's norm: its weight is stored around zero."""
    return over_rms(x, eps) * (1.0 + weight.to(x.dtype))


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(z, torch.zeros_like(z))


# ----------------------------------------------------------------------------- attention
def frequencies(rot: dict) -> torch.Tensor:
    """f_i = base^(-2i / dims), all divided by the scaling's factor if there is one."""
    dims = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))
    if rot.get("scaling") is not None:
        f = f / float(rot["scaling"]["factor"])
    return f


def turn_halves(x: torch.Tensor, positions: torch.Tensor, rot: "dict | None") -> torch.Tensor:
    """x [T, heads, d]: feature i < dims / 2 of every head is turned together with feature
    i + dims / 2 by the angle position * f_i; features from dims on stay."""
    if rot is None or rot["dims"] == 0:
        return x
    dims, half = rot["dims"], rot["dims"] // 2
    angle = positions.to(torch.float64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat((u * c - v * s, v * c + u * s, x[..., dims:]), dim=-1)


def visible(positions: torch.Tensor, window: "int | None") -> torch.Tensor:
    """[T, T]: whether row i sees key j."""
    back = positions[:, None] - positions[None, :]
    seen = back >= 0
    return seen if window is None else seen & (back < window)


def soft_cap(s: torch.Tensor, cap: "float | None") -> torch.Tensor:
    return s if cap is None else cap * torch.tanh(s / cap)


def weights_plus_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum_j exp(s_j)) over the last axis (masked scores are -inf)."""
    top = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def attention(h, w, prefix, m, eps, form, positions=None, act=None):
    """Windowed grouped-query attention whose values are its keys' projections.  ``form`` "sink"
    (the stand-alone mixer): turn, then a root-mean-square norm per head without a weight, capped
    scores, the weights with one in the denominator; ``form`` "plain" (the left branch): a weighted
    norm over the whole projection, then the turn, an ordinary softmax.  Returns the heads' results
    [T, H vdim] before the output matrix."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    positions = torch.arange(T) if positions is None else positions
    q, k = lin(h, w[prefix + "q"], act), lin(h, w[prefix + "k"], act)
    v = k.reshape(T, G, d)
    if form == "plain":
        q = over_rms(q, eps) * w[prefix + "q.norm"].to(q.dtype)
        k = over_rms(k, eps) * w[prefix + "k.norm"].to(k.dtype)
    q = turn_halves(q.reshape(T, H, d), positions, m.get("rot"))
    k = turn_halves(k.reshape(T, G, d), positions, m.get("rot"))
    if form == "sink":
        q, k = over_rms(q, eps), over_rms(k, eps)
    q, k = rnd(q, act), rnd(k, act)
    serves = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, serves]) * m["scale"]
    window = None if m.get("mask") is None else m["mask"]["size"]
    if form == "sink":
        s = soft_cap(s, m.get("softcap"))
    s = s.masked_fill(~visible(positions, window)[None], float("-inf"))
    p = weights_plus_one(s) if form == "sink" else torch.softmax(s, dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v[:, serves]).reshape(T, H * d)


# ----------------------------------------------------------------------------- gated recurrence
def causal_convolution(x, taps, bias):
    """y_t = bias + sum_k taps[:, k] x_(t - K + 1 + k) per channel, zeros before the start."""
    K, T = taps.shape[1], x.shape[0]
    padded = torch.cat((x.new_zeros(K - 1, x.shape[1]), x))
    y = bias.to(x.dtype).expand(T, -1).clone()
    for k in range(K):
        y = y + padded[k: k + T] * taps[:, k].to(x.dtype)
    return y


def block_gate(u, weight, bias):
    """sigmoid(M_b u_b + bias_b) for every one of the equal parts u_b of u's rows; weight
    [blocks, n, n] as [out, in]."""
    blocks, n, _ = weight.shape
    parts = u.reshape(u.shape[0], blocks, n)
    z = torch.einsum("boi,tbi->tbo", weight.to(u.dtype), parts) + bias.to(u.dtype)
    return sigmoid(z).reshape(u.shape)


def decays(r, lam):
    """(a, what an input is multiplied by): log a = -8 r softplus(lam), and sqrt(1 - a^2)."""
    log_a = -8.0 * r * softplus(lam.to(r.dtype))
    return torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a))


def linear_recurrence(a, b, state=None):
    """Token by token: S <- a_t S + b_t per channel, from zero.  Returns (all S, the last)."""
    S = torch.zeros_like(a[0]) if state is None else state
    out = []
    for t in range(a.shape[0]):
        S = a[t] * S + b[t]
        out.append(S)
    return torch.stack(out), S


def gated_recurrence(h, w, prefix, m, act=None):
    """Two branches, y = gelu(W_y h + b_y) and u = convolution(W_x h + b_x); the recurrence on u
    with its gates; S * y, before the output matrix."""
    y = gelu_tanh(lin(h, w[prefix + "y"], act) + w[prefix + "y.b"].to(h.dtype))
    x = lin(h, w[prefix + "x"], act) + w[prefix + "x.b"].to(h.dtype)
    u = causal_convolution(x, w[prefix + "conv"], w[prefix + "conv.b"])
    r = block_gate(u, w[prefix + "ra"], w[prefix + "ra.b"])
    i = block_gate(u, w[prefix + "ri"], w[prefix + "ri.b"])
    a, keep = decays(r, w[prefix + "lam"])
    S, _ = linear_recurrence(a, keep * i * u)
    return S * y


# ----------------------------------------------------------------------------- layers, model
def mixer(kind, h, w, prefix, m, eps, act=None):
    if kind == "attention":
        return lin(attention(h, w, prefix, m, eps, "sink", act=act), w[prefix + "o"], act)
    left = attention(h, w, prefix + "left.", m["left"], eps, "plain", act=act)
    right = gated_recurrence(h, w, prefix + "right.", m["right"], act)
    # the engine forms the weighted sum of both branches as one product: it rounds scaled rows
    left = rnd(left * m["left_scale"], act) @ w[prefix + "left.o"].to(h.dtype).t()
    right = rnd(right * m["right_scale"], act) @ w[prefix + "right.o"].to(h.dtype).t()
    return rnd(left + right, act)


def feed_forward(h, w, prefix, act=None):
    g, u = lin(h, w[prefix + "gate"], act), lin(h, w[prefix + "up"], act)
    return lin(g * sigmoid(g) * u, w[prefix + "down"], act)


def source(config, i: int) -> int:
    """The layer whose tensors layer i uses."""
    j = config["layers"][i].get("weights_of")
    return i if j is None else source(config, j)


def layer(x, config, w, i, act=None):
    entry, base, eps = config["layers"][i], f"l{source(config, i)}.", config["norm"]["eps"]
    y = mixer(entry["type"], rnd(x, act), w, base + "mix.", entry["mixer"], eps, act)
    x = x + plus_one_norm(y, w[base + "norm1"], eps)
    if entry.get("mlp") is not None:
        y = feed_forward(rnd(x, act), w, base + "mlp.", act)
        x = x + plus_one_norm(y, w[base + "norm2"], eps)
    return x


def forward(config, w, tokens, dtype=torch.float64, act=None, layers=None):
    """Logits [T, vocab] of a whole sequence; ``layers``: a list that receives the stream after
    every layer."""
    x = w["embed"].to(dtype)[torch.as_tensor(tokens)]
    for i in range(len(config["layers"])):
        x = layer(x, config, w, i, act)
        if layers is not None:
            layers.append(x)
    last = rnd(plus_one_norm(x, w["final.norm"], config["norm"]["eps"]) * config["logit_scale"], act)
    return last @ w["embed"].to(dtype).t()


def greedy(config, w, prompt, count, dtype=torch.float64, act=None):
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(forward(config, w, tokens, dtype, act)[-1].argmax()))
    return tokens[len(prompt):]


# ----------------------------------------------------------------------------- weights
def tensor_shapes(config) -> "dict[str, tuple]":
    D, V = config["width"], config["vocab"]
    out = {"embed": (V, D), "final.norm": (D,)}
    for i, entry in enumerate(config["layers"]):
        if entry.get("weights_of") is not None:
            continue
        base, m = f"l{i}.", entry["mixer"]
        out[base + "norm1"] = (D,)

        def heads(prefix, a, normed):
            qn, kn = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            out[prefix + "q"], out[prefix + "k"] = (qn, D), (kn, D)
            out[prefix + "o"] = (D, a["heads"] * a["vdim"])
            if normed:
                out[prefix + "q.norm"], out[prefix + "k.norm"] = (qn,), (kn,)

        if entry["type"] == "attention":
            heads(base + "mix.", m, False)
        else:
            heads(base + "mix.left.", m["left"], True)
            r, p = m["right"], base + "mix.right."
            W, n = r["width"], r["width"] // r["blocks"]
            for s in "xy":
                out[p + s], out[p + s + ".b"] = (W, D), (W,)
            out[p + "conv"], out[p + "conv.b"] = (W, r["conv"]), (W,)
            for s in ("ra", "ri"):
                out[p + s], out[p + s + ".b"] = (r["blocks"], n, n), (r["blocks"], n)
            out[p + "lam"], out[p + "o"] = (W,), (D, W)
        if entry.get("mlp") is not None:
            ff = entry["mlp"]["ff"]
            out[base + "norm2"] = (D,)
            out[base + "mlp.gate"] = out[base + "mlp.up"] = (ff, D)
            out[base + "mlp.down"] = (D, ff)
    return out


def random_weights(config, seed: int) -> "dict[str, torch.Tensor]":
    """float32 values that bfloat16 holds exactly, sizes chosen so that every mechanism matters:
    decays between fast and slow, gates away from their middles, norm weights away from zero."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(config).items():
        z = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = z * 0.5
        elif last in ("norm1", "norm2") or name == "final.norm":
            t = 0.3 * z
        elif last == "norm":
            t = 1.0 + 0.3 * z
        elif last == "lam":
            t = -3.0 + 2.0 * z
        elif last in ("b", "conv"):
            t = 0.4 * z
        else:
            t = z / math.sqrt(shape[-1])
        w[name] = t.to(torch.bfloat16).float()
    return w
