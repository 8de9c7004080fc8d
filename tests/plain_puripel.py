"""A plain, slow implementation of the Puripel decoder, one function per mechanism, whole sequences
only, in float64 (or float32) on the CPU.  It shares no code with the engine: the engine's parts
and kernels are compared with it.

``act`` (None or torch.bfloat16) models the engine's bfloat16 mode: the results of matrix products
and the norms' outputs are rounded to it (``rnd``); the residual stream, scores, softmax weights,
angles, router scores, norm statistics, step sizes, decays and the state are not.

Notation: T tokens, width D.  A weight matrix is stored [out, in]; ``lin`` applies it.  ``w`` maps
tensor names to tensors, ``config`` is the parsed config.json.
"""

from __future__ import annotations

import math

import torch


def rnd(x: torch.Tensor, act) -> torch.Tensor:
    return x if act is None else x.to(act).to(x.dtype)


def lin(x: torch.Tensor, weight: torch.Tensor, act=None) -> torch.Tensor:
    return rnd(x @ weight.to(x.dtype).t(), act)


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float, act=None) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return rnd(x / rms(x, eps) * weight.to(x.dtype), act)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(x, torch.zeros_like(x))


# ----------------------------------------------------------------------------- rotation
def turn_adjacent(x: torch.Tensor, positions: torch.Tensor, base: float) -> torch.Tensor:
    """x [T, ..., d]: the pair (x_2i, x_2i+1) at position p turned by the angle p base^(-2i / d)."""
    d = x.shape[-1]
    f = float(base) ** (-2.0 * torch.arange(d // 2, dtype=torch.float64) / max(d, 1))
    angle = positions.to(torch.float64)[:, None] * f[None, :]
    angle = angle.reshape(x.shape[0], *([1] * (x.dim() - 2)), d // 2)
    c, s = torch.cos(angle).to(x.dtype), torch.sin(angle).to(x.dtype)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack((u * c - v * s, v * c + u * s), dim=-1).reshape(x.shape)


# ----------------------------------------------------------------------------- mixers
def latent_attention(h, w, prefix, m, eps, positions=None, act=None):
    """Windowed attention whose keys and values are read from a small latent per token.

        cq = rms_norm(W_dq h) ; q = W_uq cq, per head [dim plain | rot_dim turned]
        [c | kr] = W_dkv h ; c = rms_norm(c) (kv_rank) ; kr turned (rot_dim), one for all heads
        k_h = W_uk c (dim per head) ; v_h = W_uv c (vdim per head)
        score = (q_plain . k_h + q_turned . kr) * scale over the keys 0 <= i - j < window
        out = W_o (heads' softmax-weighted sums of v_h)
    """
    T = h.shape[0]
    H, dim, rot_dim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(T) if positions is None else positions
    cq = rms_norm(lin(h, w[prefix + "dq"], act), w[prefix + "dq.norm"], eps, act)
    q = lin(cq, w[prefix + "uq"], act).reshape(T, H, dim + rot_dim)
    kv = lin(h, w[prefix + "dkv"], act)
    c = rms_norm(kv[:, :rank], w[prefix + "dkv.norm"], eps, act)
    q_rot = turn_adjacent(q[..., dim:], positions, m["rot"]["base"])
    k_rot = turn_adjacent(kv[:, rank:], positions, m["rot"]["base"])
    k = lin(c, w[prefix + "uk"], act).reshape(T, H, dim)
    v = lin(c, w[prefix + "uv"], act).reshape(T, H, vdim)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :dim], k)
              + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    back = positions[:, None] - positions[None, :]
    seen = (back >= 0) & (back < m["mask"]["size"])
    p = torch.softmax(scores.masked_fill(~seen[None], float("-inf")), dim=-1)
    heads = torch.einsum("hij,jhd->ihd", p, v).reshape(T, H * vdim)
    return lin(rnd(heads, act), w[prefix + "o"], act)


def causal_convolution(x, taps, bias):
    """y_t = bias + sum_k taps[:, k] x_(t - K + 1 + k) per channel, zeros before the start."""
    K, T = taps.shape[1], x.shape[0]
    padded = torch.cat((x.new_zeros(K - 1, x.shape[1]), x))
    y = bias.to(x.dtype).expand(T, -1).clone()
    for k in range(K):
        y = y + padded[k: k + T] * taps[:, k].to(x.dtype)
    return y


def selective_scan(x, b, c, dt, a_log, d, state=None):
    """Token by token: x [T, H, P], b and c [T, H, N], dt [T, H].  Per head
    S <- exp(-exp(a_log) dt) S + dt b x^T ; y = S^T c + d x.  Returns (y, S)."""
    T, H, P = x.shape
    S = x.new_zeros(H, b.shape[2], P) if state is None else state.clone()
    out = []
    for t in range(T):
        decay = torch.exp(-torch.exp(a_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, c[t]) + d[:, None] * x[t])
    return torch.stack(out), S


def gated_group_norm(y, z, weight, parts, eps):
    """y silu(z), then every one of ``parts`` equal pieces of the row over its own root mean
    square, then the weight."""
    g = y * silu(z)
    T, n = g.shape
    pieces = g.reshape(T, parts, n // parts)
    return (pieces / rms(pieces, eps)).reshape(T, n) * weight.to(y.dtype)


def mamba2(h, w, prefix, m, eps, act=None):
    """W_in h = [z | x | B | C | dt]; x, B and C through the convolution and silu; the scan with
    head h reading group h // (heads / groups); the gate, the norm in parts, W_o."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = lin(h, w[prefix + "in"], act)
    z, xbc, dt = proj[:, :inner], proj[:, inner: 2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_convolution(xbc, w[prefix + "conv"], w[prefix + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    group = torch.arange(H) // (H // G)
    b = xbc[:, inner: inner + G * N].reshape(T, G, N)[:, group]
    c = xbc[:, inner + G * N:].reshape(T, G, N)[:, group]
    dt = softplus(dt + w[prefix + "dt_bias"].to(h.dtype))
    y, _ = selective_scan(x, b, c, dt, w[prefix + "A_log"].to(h.dtype), w[prefix + "D"].to(h.dtype))
    y = gated_group_norm(y.reshape(T, inner), z, w[prefix + "norm"], m["norm_groups"], eps)
    return lin(rnd(y, act), w[prefix + "o"], act)


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2}


# ----------------------------------------------------------------------------- feed-forward
def clipped_gate(gate, up, limit):
    """g sigmoid(1.702 g) (u + 1) with g = min(gate, limit) and u = up clamped to +- limit."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def expert(h, w, prefix, limit, act=None):
    inner = clipped_gate(lin(h, w[prefix + "gate"], act), lin(h, w[prefix + "up"], act), limit)
    return lin(rnd(inner, act), w[prefix + "down"], act)


def choose(scores, correction, top, groups, keep):
    """The ``top`` experts with the largest choice scores (score + correction) among the ``keep``
    groups whose two best choice scores have the largest sum."""
    choice = scores + correction
    T, E = choice.shape
    size = E // groups
    grouped = choice.reshape(T, groups, size)
    value = torch.topk(grouped, min(2, size), dim=-1).values.sum(dim=-1)
    kept = torch.topk(value, keep, dim=-1).indices
    open_ = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, kept, True)
    open_ = open_[:, :, None].expand(T, groups, size).reshape(T, E)
    return torch.topk(choice.masked_fill(~open_, float("-inf")), top, dim=-1).indices


def routed_feed_forward(h, w, prefix, mlp, act=None, chosen=None):
    """sum over the chosen experts of s_e / (sum of the chosen s + 1e-20) * scale * expert_e(h),
    s = sigmoid(W_router h), plus the shared expert times sigmoid(W_sg h).  ``chosen`` [T, top]
    takes the place of the router's choice (an implementation in bfloat16 sees slightly different
    scores, and where two are nearly tied it may pick the other)."""
    r, limit = mlp["router"], mlp["expert"]["limit"]
    s = torch.sigmoid(h @ w[prefix + "router"].to(h.dtype).t())
    if chosen is None:
        chosen = choose(s, w[prefix + "correction"].to(h.dtype), r["top"], r["groups"]["count"],
                        r["groups"]["keep"])
    mine = torch.gather(s, 1, chosen.long())
    weights = mine / (mine.sum(dim=-1, keepdim=True) + 1e-20) * r["scale"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(chosen[t].tolist(), weights[t]):
            out[t] += weight * expert(h[t: t + 1], w, f"{prefix}e{e}.", limit, act)[0]
    shared = expert(h, w, prefix + "shared.", mlp["shared"]["limit"], act)
    return out + shared * torch.sigmoid(lin(h, w[prefix + "shared.sg"]))


# ----------------------------------------------------------------------------- the model
def run_order(config) -> "list[tuple[int, int | None]]":
    """(layer, the number of the pass that starts with it or None) for every layer run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, None) for i in range(start)]
    for t in range(times):
        order += [(i, t if i == start else None) for i in range(start, stop)]
    return order + [(i, None) for i in range(stop, n)]


def layer(x, w, config, index, act=None, chosen=None):
    """x <- x + norm1b(mixer(norm1 x)); x <- x + norm2b(ff(norm2 x))."""
    entry, eps, prefix = config["layers"][index], config["norm"]["eps"], f"l{index}."
    h = rms_norm(x, w[prefix + "norm1"], eps, act)
    y = MIXERS[entry["type"]](h, w, prefix + "mix.", entry["mixer"], eps, act=act)
    x = x + rms_norm(y, w[prefix + "norm1b"], eps)
    if entry.get("mlp") is not None:
        h = rms_norm(x, w[prefix + "norm2"], eps, act)
        y = routed_feed_forward(h, w, prefix + "mlp.", entry["mlp"], act, chosen)
        x = x + rms_norm(y, w[prefix + "norm2b"], eps)
    return x


def forward(tokens, w, config, act=None, dtype=torch.float64, trace=None, routing=None):
    """Logits [T, vocab] of one whole sequence.  ``trace``: a list that receives the residual
    stream after every layer run.  ``routing``: layer run -> chosen experts [T, top], in place of
    the router's choice in that run."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    x = w["embed"][tokens].clone()
    for run, (index, turn) in enumerate(run_order(config)):
        if turn is not None:
            x = x + w["loop.step"][turn]
        x = layer(x, w, config, index, act, None if routing is None else routing.get(run))
        if trace is not None:
            trace.append(x.clone())
    last = rms_norm(x, w["final.norm"], config["norm"]["eps"], act)
    return last @ w["embed"].t()


# ----------------------------------------------------------------------------- weights
def mixer_shapes(kind, m, D) -> dict[str, tuple[int, ...]]:
    if kind == "latent_attention":
        H = m["heads"]
        return {"dq": (m["q_rank"], D), "dq.norm": (m["q_rank"],),
                "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                "dkv": (m["kv_rank"] + m["rot_dim"], D), "dkv.norm": (m["kv_rank"],),
                "uk": (H * m["dim"], m["kv_rank"]), "uv": (H * m["vdim"], m["kv_rank"]),
                "o": (D, H * m["vdim"])}
    H, inner = m["heads"], m["heads"] * m["vdim"]
    channels = inner + 2 * m["groups"] * m["state"]
    return {"in": (inner + channels + H, D), "conv": (channels, m["conv"]), "conv.b": (channels,),
            "dt_bias": (H,), "A_log": (H,), "D": (H,), "norm": (inner,), "o": (D, inner)}


def mlp_shapes(mlp, D) -> dict[str, tuple[int, ...]]:
    E, F, S = mlp["router"]["experts"], mlp["expert"]["ff"], mlp["shared"]["ff"]
    out = {"router": (E, D), "correction": (E,), "shared.gate": (S, D), "shared.up": (S, D),
           "shared.down": (D, S), "shared.sg": (1, D)}
    for e in range(E):
        out.update({f"e{e}.gate": (F, D), f"e{e}.up": (F, D), f"e{e}.down": (D, F)})
    return out


def tensor_shapes(config) -> dict[str, tuple[int, ...]]:
    D, V = config["width"], config["vocab"]
    shapes: dict[str, tuple[int, ...]] = {"embed": (V, D), "final.norm": (D,)}
    if config.get("loop"):
        shapes["loop.step"] = (config["loop"]["times"], D)
    for i, entry in enumerate(config["layers"]):
        p = f"l{i}."
        shapes.update({p + "norm1": (D,), p + "norm1b": (D,)})
        shapes.update({p + "mix." + k: v
                       for k, v in mixer_shapes(entry["type"], entry["mixer"], D).items()})
        if entry.get("mlp") is not None:
            shapes.update({p + "norm2": (D,), p + "norm2b": (D,)})
            shapes.update({p + "mlp." + k: v for k, v in mlp_shapes(entry["mlp"], D).items()})
    return shapes


def draw(shapes, generator, spread: float = 1.0) -> dict[str, torch.Tensor]:
    """bfloat16 tensors by name: matrices N(0, spread^2 / fan-in), norm weights near 1, decays and
    step sizes from fast to slow, corrections of both signs."""
    g, out = generator, {}
    for name, shape in shapes.items():
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last.startswith("norm"):
            t = 1.0 + 0.2 * r
        elif last == "A_log":
            t = -4.0 + 5.0 * torch.rand(shape, generator=g)
        elif last == "dt_bias":
            t = -3.0 + 1.5 * r
        elif last == "D":
            t = 1.0 + 0.5 * r
        elif name == "embed":
            t = r
        elif last in ("correction", "step", "b"):
            t = 0.3 * r
        elif last == "conv":
            t = 0.6 * r
        else:
            t = r * spread / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def random_weights(config, seed: int, spread: float = 1.0) -> dict[str, torch.Tensor]:
    return draw(tensor_shapes(config), torch.Generator().manual_seed(seed), spread)
