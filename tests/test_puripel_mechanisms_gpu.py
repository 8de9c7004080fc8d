"""Each mechanism of the Puripel parts alone, built through the registries and run through the
engine's step machinery, against the plain function in ``plain_puripel``: windowed latent attention
in portions and single tokens, with the keys at the window's edge made decisive; Mamba-2 in
portions of every kind, with long memory and with fast decay; the gate and the norm in parts; the
grouped router, the clipped experts and the shared one; the norms on both sides of a sublayer."""

import math

import pytest
import torch

import plain_puripel as pp
import puripel_configs as pc
from gpu_helpers import PagedFixture, PartHarness, assert_close, run_paged_attention

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def _spec():
    from distengine_b200.config.model import PartSpec
    return PartSpec


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _act(dtype):
    return None if dtype == torch.float32 else torch.bfloat16


def _double(w):
    return {k: v.double() for k, v in w.items()}


def _run_in_portions(mixer, h, xs, portions):
    """Feeds the requests' rows in the given portions ({request: count} per step); returns what
    the mixer gave for every request's rows in order."""
    fed = {rid: 0 for rid in xs}
    got = {rid: [] for rid in xs}
    for step in portions:
        entries = [(rid, n) for rid, n in step if n]
        x = torch.cat([xs[rid][fed[rid]: fed[rid] + n] for rid, n in entries]).to(DEV)
        out = h.run(entries, lambda ctx, b: mixer.forward(x, ctx, b[0]).clone()).float().cpu()
        at = 0
        for rid, n in entries:
            got[rid].append(out[at: at + n])
            at += n
            fed[rid] += n
    assert all(fed[rid] == xs[rid].shape[0] for rid in xs)
    return {rid: torch.cat(parts) for rid, parts in got.items()}


# ----------------------------------------------------------------------------- latent attention
def _latent(dtype, width, m, eps):
    from distengine_b200.parts import build_mixer
    return build_mixer(_spec().of(
        "latent_attention", width=width, heads=m["heads"], key_dim=m["dim"],
        rotary_dim=m["rot_dim"], value_dim=m["vdim"], q_rank=m["q_rank"], kv_rank=m["kv_rank"],
        scale=m["scale"], theta=m["rot"]["base"], eps=eps, window=m["mask"]["size"],
        adjacent=True, gated=False, exact_weights=True), dtype, torch.device(DEV))


def _latent_weights(m, width, seed, spread=1.5):
    return {k: v.float() for k, v in pp.draw(pp.mixer_shapes("latent_attention", m, width),
                                             _gen(seed), spread).items()}


LATENT = [
    # heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, base; page
    ((3, 6, 2, 5, 9, 7, 0.6, 5, 100.0), 16),          # rows of 9: no 16-byte piece
    ((8, 16, 8, 16, 24, 24, 0.4, 16, 50000.0), 8),    # the one-launch decode; whole pages
    ((12, 8, 16, 8, 16, 16, 0.3, 17, 10000.0), 4),    # more than 8 heads
    ((1, 32, 4, 1, 8, 60, 0.3, 1, 500.0), 8),         # one head, values of size 1, itself only
    ((5, 4, 32, 24, 40, 8, 0.5, 40, 20.0), 32),       # mostly turned
    ((6, 24, 16, 20, 32, 48, 0.3, 23, 10000.0), 16),  # cached rows of 64 and of 128 features
    ((4, 32, 32, 16, 24, 96, 0.2, 64, 1e6), 16),
    ((7, 12, 16, 20, 24, 80, 0.3, 2, 10000.0), 4),    # a window of two tokens
    ((4, 8, 8, 8, 8, 16, 0.3, 4096, 10000.0), 16),    # a window beyond everything
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes,page", LATENT)
def test_windowed_latent_attention_in_portions(dtype, sizes, page):
    """Two requests in unequal portions beside single tokens, then steps of single tokens only,
    against the plain function over each whole sequence; pages behind the window are given back
    and poisoned."""
    width, eps = 44, 1e-5
    m = pc.latent(*sizes)
    mixer = _latent(dtype, width, m, eps)
    w = _latent_weights(m, width, sizes[0] * 7 + sizes[5])
    assert {k: v[0] for k, v in mixer.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
    mixer.load(w)
    spec = mixer.cache_spec()
    assert (spec.head_dim, spec.v_dim, spec.window) == (m["kv_rank"] + m["rot_dim"], m["kv_rank"],
                                                        m["mask"]["size"])
    g = _gen(5)
    xs = {"a": torch.randn(142, width, generator=g).to(dtype),
          "b": torch.randn(46, width, generator=g).to(dtype)}
    want = {rid: pp.latent_attention(x.double(), _double(w), "", m, eps, act=_act(dtype))
            for rid, x in xs.items()}
    h = PartHarness([mixer], [spec], dtype, page_size=page, num_pages=4 + 224 // page)
    portions = [[("a", 90), ("b", 1)], [("a", 2), ("b", 1)], [("a", 1), ("b", 17)], [("a", 25)],
                [("a", 17), ("b", 21)]] + [[("a", 1), ("b", 1)]] * 6 + [[("a", 1)]]
    got = _run_in_portions(mixer, h, xs, portions)
    for rid in xs:
        assert_close(got[rid], want[rid], dtype, f"latent attention {rid}")


@pytest.mark.parametrize("decoded", [0, 70])
@pytest.mark.parametrize("window", [16, 33, 48])
@pytest.mark.parametrize("place", [0, 15, 16, 31, 32])
def test_the_windows_edge_decides(place, window, decoded):
    """One key's input row is made large (its turned part is not normed) and the scale sharp, so
    that the last token that sees it differs from what any window one shorter would give, and the
    next token from any window one longer: one token off shows."""
    width, eps, T = 40, 1e-6, 90
    m = pc.latent(4, 8, 8, 12, 16, 24, 1.5, window)
    mixer = _latent(torch.float32, width, m, eps)
    w = _latent_weights(m, width, 31, spread=2.0)
    mixer.load(w)
    inside, outside = place + window - 1, place + window
    plain = lambda x, size: pp.latent_attention(x.double(), _double(w), "",
                                                dict(m, mask={"size": size}), eps)
    for seed in range(200):
        x = torch.randn(T, width, generator=_gen(1000 * window + 10 * place + seed))
        x[place] *= 6.0
        want, shorter, longer = plain(x, window), plain(x, window - 1), plain(x, window + 1)
        big = 0.1 * want.abs().max()
        if ((want - shorter)[inside].abs().max() > big
                and (want - longer)[outside].abs().max() > big):
            break
    else:
        raise AssertionError("no input was found whose key decides at both edges")
    h = PartHarness([mixer], [mixer.cache_spec()], torch.float32, page_size=16, num_pages=12)
    head = T - decoded
    portions = [[("a", head - 7)], [("a", 7)]] + [[("a", 1)]] * decoded
    got = _run_in_portions(mixer, h, {"a": x}, portions)
    assert_close(got["a"], want, torch.float32, f"window {window} key {place}")


def test_pages_behind_the_window_are_used_again():
    """Many requests, one after the other and side by side, in a pool that holds the windows of
    two of them only (freed pages are poisoned)."""
    width, eps = 32, 1e-5
    m = pc.latent(3, 8, 4, 8, 12, 12, 0.4, 11)
    mixer = _latent(torch.float32, width, m, eps)
    w = _latent_weights(m, width, 9)
    mixer.load(w)
    h = PartHarness([mixer], [mixer.cache_spec()], torch.float32, page_size=4, num_pages=20,
                    max_seqs=3)
    g = _gen(2)
    for rnd in range(5):
        a, b = f"r{rnd}a", f"r{rnd}b"
        xs = {a: torch.randn(61 + rnd, width, generator=g), b: torch.randn(20, width, generator=g)}
        portions = [[(a, 30), (b, 9)], [(a, 21 + rnd), (b, 2)]] + [[(a, 1), (b, 1)]] * 9 + [[(a, 1)]]
        got = _run_in_portions(mixer, h, xs, portions)
        for rid, x in xs.items():
            assert_close(got[rid], pp.latent_attention(x.double(), _double(w), "", m, eps),
                         torch.float32, f"turn {rnd} {rid}")
            h.cache.release(rid)
        h.cache.check_invariants()


def test_two_layers_that_differ_in_their_window_only():
    """Their steps' work lists must not be shared: both run in one step."""
    width, eps = 32, 1e-5
    sizes = [pc.latent(6, 24, 16, 20, 32, 48, 0.3, window) for window in (7, 64)]
    for dtype in DTYPES:
        mixers = [_latent(dtype, width, m, eps) for m in sizes]
        ws = [_latent_weights(m, width, 3) for m in sizes]
        for mixer, w in zip(mixers, ws):
            mixer.load(w)
        h = PartHarness(mixers, [mixer.cache_spec() for mixer in mixers], dtype, num_pages=24)
        x = torch.randn(150, width, generator=_gen(8)).to(dtype)
        got = [[], []]
        at = 0
        for n in [100, 47, 1, 1, 1]:
            rows = x[at: at + n].to(DEV)
            outs = h.run([("a", n)], lambda ctx, b: [mixer.forward(rows, ctx, c).clone()
                                                     for mixer, c in zip(mixers, b)])
            for i, o in enumerate(outs):
                got[i].append(o.float().cpu())
            at += n
        for i, m in enumerate(sizes):
            want = pp.latent_attention(x.double(), _double(ws[i]), "", m, eps, act=_act(dtype))
            assert_close(torch.cat(got[i]), want, dtype, f"window {m['mask']['size']}")


@pytest.mark.parametrize("head_dim", [16, 64, 112, 256])
@pytest.mark.parametrize("window", [40, None])
@pytest.mark.parametrize("chunk", [0, 64])
def test_softmax_weights_are_not_rounded_to_sixteen_bits(head_dim, window, chunk):
    """On the tensor cores with ``exact_weights`` the result is the exact one rounded once, but for
    elements next to a tie; with weights of one bfloat16 term many more elements differ."""
    heads, lens, rows = 5, [150, 70], [130, 21]
    fx = PagedFixture(lens, 1, head_dim, 16, torch.bfloat16, DEV, seed=head_dim)
    g = _gen(head_dim + chunk)
    q = [torch.randn(n, heads, head_dim, generator=g).to(torch.bfloat16).float() for n in rows]
    scale, want = 0.7 / math.sqrt(head_dim), []
    for i, n in enumerate(rows):
        at, keys = torch.arange(lens[i] - n, lens[i])[:, None], torch.arange(lens[i])[None, :]
        seen = (keys <= at) & (at - keys < (window or 1 << 30))
        s = torch.einsum("ihd,jd->hij", q[i].double(), fx.k[i][:, 0].double()) * scale
        p = torch.softmax(s.masked_fill(~seen[None], float("-inf")), dim=-1)
        want.append(torch.einsum("hij,jd->ihd", p, fx.v[i][:, 0].double()).reshape(n, -1))
    want = torch.cat(want).to(torch.bfloat16).float()
    unequal = {}
    for exact in (True, False):
        got, _ = run_paged_attention(fx, q, heads, 1, head_dim, scale, window, chunk=chunk,
                                     exact_weights=exact)
        assert_close(got, want, torch.bfloat16, f"exact {exact}")
        unequal[exact] = (got != want).float().mean().item()
    assert unequal[True] < 0.01 < 0.05 < unequal[False], unequal


def test_neighbours_are_turned_as_complex_numbers():
    x = torch.randn(9, 3, 10, dtype=torch.float64, generator=_gen(1))
    positions = torch.tensor([0, 1, 2, 17, 300, 4095, 100000, 5, 6])
    z = torch.view_as_complex(x.reshape(9, 3, 5, 2).contiguous())
    f = 700.0 ** (-torch.arange(5, dtype=torch.float64) / 5)
    turned = torch.view_as_real(z * torch.exp(1j * positions[:, None, None] * f)).reshape(9, 3, 10)
    assert_close(pp.turn_adjacent(x, positions, 700.0), turned, torch.float32, "turned pairs")


# ----------------------------------------------------------------------------- Mamba-2
def _mamba(dtype, width, m, eps):
    from distengine_b200.parts import build_mixer
    return build_mixer(_spec().of("mamba2", width=width, heads=m["heads"], groups=m["groups"],
                                  state_dim=m["state"], value_dim=m["vdim"], taps=m["conv"],
                                  norm_groups=m["norm_groups"], eps=eps), dtype,
                       torch.device(DEV))


def _mamba_weights(m, width, seed, spread=1.5):
    return {k: v.float() for k, v in pp.draw(pp.mixer_shapes("mamba2", m, width), _gen(seed),
                                             spread).items()}


MAMBA = [
    # heads, groups, state, vdim, conv, norm_groups
    (6, 3, 5, 3, 4, 2),            # odd sizes
    (4, 1, 16, 8, 4, 1),           # one group for all heads
    (3, 3, 24, 20, 2, 3),          # a group a head
    (2, 2, 64, 64, 3, 4),          # parts of the norm that are halves of a head
    (2, 1, 128, 64, 4, 1),
    (1, 1, 7, 130, 5, 10),         # three tiles of columns, the last nearly empty
    (5, 5, 1, 1, 1, 1),            # a state of one number, no convolution state
    (2, 1, 200, 36, 6, 2),         # more rows than two tiles
    (4, 2, 96, 33, 4, 4),          # whole pieces along the state, none along the values
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", MAMBA)
def test_mamba2_in_portions(dtype, sizes):
    """Two requests in portions of one token up to many chunks, long and short ones in one step,
    then single tokens only."""
    width, eps = 40, 1e-5
    m = pc.mamba(*sizes)
    mixer = _mamba(dtype, width, m, eps)
    w = _mamba_weights(m, width, 11 * sizes[0] + sizes[2])
    assert {k: v[0] for k, v in mixer.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
    mixer.load(w)
    g = _gen(6)
    xs = {"a": torch.randn(441, width, generator=g).to(dtype),
          "b": torch.randn(106, width, generator=g).to(dtype)}
    want = {rid: pp.mamba2(x.double(), _double(w), "", m, eps, act=_act(dtype))
            for rid, x in xs.items()}
    h = PartHarness([mixer], [mixer.cache_spec()], dtype, max_seqs=3)
    portions = [[("a", 130), ("b", 1)], [("a", 2), ("b", 1)], [("a", 1), ("b", 17)], [("a", 64)],
                [("a", 16), ("b", 16)], [("a", 3), ("b", 65)], [("a", 200)], [("a", 17)],
                [("a", 2)]] + [[("a", 1), ("b", 1)]] * 6
    got = _run_in_portions(mixer, h, xs, portions)
    for rid in xs:
        assert_close(got[rid], want[rid], dtype, f"mamba2 {sizes} {rid}")


@pytest.mark.parametrize("sizes", [(4, 2, 16, 8, 4, 2), (2, 1, 128, 64, 4, 1), (3, 1, 9, 5, 3, 1)])
def test_mamba2_does_not_depend_on_the_cut(sizes):
    """One portion, token by token, pairs, and uneven portions give the same in 32-bit."""
    width, eps, T = 32, 1e-6, 150
    m = pc.mamba(*sizes)
    mixer = _mamba(torch.float32, width, m, eps)
    mixer.load(_mamba_weights(m, width, 2))
    x = {"a": torch.randn(T, width, generator=_gen(3))}
    results = []
    for cut in ([T], [1] * T, [2] * 75, [63, 1, 64, 22], [17, 16, 15, 102]):
        h = PartHarness([mixer], [mixer.cache_spec()], torch.float32, max_seqs=1)
        results.append(_run_in_portions(mixer, h, x, [[("a", n)] for n in cut])["a"])
    scale = max(1.0, results[0].abs().max().item())
    for other in results[1:]:
        assert (other - results[0]).abs().max().item() <= 5e-6 * scale


@pytest.mark.parametrize("kind", ["slow", "fast", "both", "jumps"])
def test_mamba2_memory(kind):
    """Decays near 1 (the first tokens still count hundreds of tokens later), decays near 0 with
    step sizes far on softplus's straight side, heads of both kinds in one layer, and step sizes
    that jump between next to nothing and hundreds from token to token: sums of large exponents
    whose small differences count."""
    width, eps, T = 24, 1e-6, 330
    m = pc.mamba(4, 2, 12, 8, 2, 2)
    w = _mamba_weights(m, width, 21)
    if kind == "slow":
        w["A_log"][:], w["dt_bias"][:] = -7.0, -1.0
    elif kind == "fast":
        w["A_log"][:], w["dt_bias"][:] = 2.0, 25.0
    elif kind == "both":
        w["A_log"][:], w["dt_bias"][:] = torch.tensor([-7.0, 3.0, -5.0, 1.0]), 0.0
    else:
        w["A_log"][:], w["dt_bias"][:] = torch.tensor([0.0, 1.0, -3.0, 0.5]), 0.0
        w["in"][-4:] *= 60.0
    mixer = _mamba(torch.float32, width, m, eps)
    mixer.load(w)
    x = torch.randn(T, width, generator=_gen(4))
    want = pp.mamba2(x.double(), _double(w), "", m, eps)
    if kind == "slow":
        later = x.clone()
        later[0] = 0.0
        gone = pp.mamba2(later.double(), _double(w), "", m, eps)
        assert (gone - want)[-1].abs().max() > 5e-4 * want.abs().max()     # far beyond rounding
    h = PartHarness([mixer], [mixer.cache_spec()], torch.float32)
    got = _run_in_portions(mixer, h, {"a": x}, [[("a", 200)], [("a", 9)], [("a", 90)]]
                           + [[("a", 1)]] * 31)
    assert_close(got["a"], want, torch.float32, f"memory {kind}")


def test_slots_start_from_zero_when_they_are_used_again():
    """A request that takes over a slot sees neither the state nor the convolution's kept inputs of
    the one before it, whatever the length of its first portion."""
    width, eps = 32, 1e-5
    m = pc.mamba(4, 2, 16, 8, 4, 2)
    mixer = _mamba(torch.float32, width, m, eps)
    w = _mamba_weights(m, width, 7)
    mixer.load(w)
    h = PartHarness([mixer], [mixer.cache_spec()], torch.float32, max_seqs=2)
    g = _gen(5)
    for rnd, first in enumerate((40, 1, 2, 70, 17)):
        a, b = f"r{rnd}a", f"r{rnd}b"
        xs = {a: torch.randn(first + 5, width, generator=g), b: torch.randn(6, width, generator=g)}
        got = _run_in_portions(mixer, h, xs, [[(a, first), (b, 1)]] + [[(a, 1), (b, 1)]] * 5)
        for rid, x in xs.items():
            assert_close(got[rid], pp.mamba2(x.double(), _double(w), "", m, eps), torch.float32,
                         f"turn {rnd} {rid}")
            h.cache.release(rid)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,cols,parts", [(5, 42, 3), (3, 64, 1), (7, 96, 8), (2, 4096, 4),
                                          (3, 2052, 1), (1, 15, 15)])
def test_the_gate_comes_before_the_norm_in_parts(dtype, n, cols, parts):
    """Rows of tiny numbers show eps inside the root; a part's root mean square is its own."""
    from distengine_b200.kernels import ssm
    eps, g = 1e-5, _gen(cols)
    y = torch.randn(n, cols, generator=g)
    y[0] *= 1e-3
    y[-1, : cols // parts] *= 50.0
    both = torch.randn(n, cols + 8, generator=g).to(dtype)
    z, weight = both[:, :cols], torch.rand(cols, generator=g) + 0.5
    out = torch.empty(n, cols, dtype=dtype, device=DEV)
    h = PartHarness([], [], dtype)
    h.run([("a", n)], lambda ctx, b: ssm.gated_group_norm(
        y.to(DEV), both.to(DEV)[:, :cols], weight.to(DEV), parts, eps, out, ctx))
    want = pp.gated_group_norm(y.double(), z.double(), weight.double(), parts, eps)
    assert_close(out, want, dtype, "gated group norm")
    after = pp.silu(z.double()) * (y.double() / pp.rms(y.double().reshape(n, parts, -1), eps)
                                   .expand(n, parts, cols // parts).reshape(n, cols)) * weight
    assert (after - want).abs().max() > 0.05          # the norm before the gate is something else


# ----------------------------------------------------------------------------- experts
def _route(x, router, correction, top, groups, keep, scale, side=False):
    from distengine_b200.kernels import latent as lk
    n = x.shape[0]
    chosen = torch.empty(n, top, dtype=torch.int32, device=DEV)
    weight = torch.empty(n, top, device=DEV)
    factor = torch.empty(n, device=DEV) if side else None
    lk.experts_route(x.to(DEV), router.to(DEV), correction.to(DEV), top, chosen, weight,
                     "grouped_sigmoid", groups, keep, scale, factor)
    return chosen.cpu().long(), weight.cpu(), None if factor is None else factor.cpu()


@pytest.mark.parametrize("experts,top,groups,keep", [
    (8, 3, 2, 1), (8, 3, 4, 2), (6, 2, 6, 3), (12, 4, 3, 3), (5, 5, 1, 1), (64, 8, 8, 4),
    (200, 6, 40, 7), (33, 2, 11, 1), (1, 1, 1, 1), (96, 32, 2, 1)])
def test_grouped_routing(experts, top, groups, keep):
    """Choice by corrected scores inside the best groups, weights from the scores alone; the
    corrections are so negative that every choice score is below zero."""
    width, n, scale = 48, 60, 1.9
    g = _gen(experts + top)
    x = torch.randn(n, width, generator=g)
    router = torch.randn(experts + 1, width, generator=g) * 1.5 / math.sqrt(width)
    correction = -2.0 + 0.5 * torch.randn(experts, generator=g)
    chosen, weight, side = _route(x, router, correction, top, groups, keep, scale, side=True)
    z = x.double() @ router.double().t()
    s = torch.sigmoid(z[:, :experts])
    want = pp.choose(s, correction.double(), top, groups, keep)
    assert torch.equal(chosen.sort(dim=1).values, want.sort(dim=1).values)
    mine = torch.gather(s, 1, chosen)
    assert_close(weight, mine / (mine.sum(dim=1, keepdim=True) + 1e-20) * scale, torch.float32,
                 "weights")
    assert_close(side, torch.sigmoid(z[:, experts]), torch.float32, "the shared expert's factor")
    if keep < groups < experts and top > 1:
        free = torch.topk(s + correction.double(), top, dim=1).indices
        assert not torch.equal(free.sort(dim=1).values, want.sort(dim=1).values)


def test_a_groups_value_is_that_of_its_two_best_and_ties_go_to_the_lower_group():
    """Router rows of zero: the choice scores are 1/2 + correction."""
    x, router = torch.randn(3, 16, generator=_gen(1)), torch.zeros(8, 16)
    # group 0 has the single best expert, group 1 the best pair
    correction = torch.tensor([0.9, -1.0, -1.0, -1.0, 0.4, 0.5, -1.0, -1.0])
    chosen, weight, _ = _route(x, router, correction, 2, 2, 1, 2.5)
    assert sorted(chosen[0].tolist()) == [4, 5]
    assert_close(weight, torch.full((3, 2), 1.25), torch.float32, "equal weights")
    chosen, _, _ = _route(x, router, torch.full((8,), -3.0), 3, 4, 2, 1.0)
    assert sorted(chosen[2].tolist()) == [0, 1, 2]
    # scores so small that their sum needs the guard: the weights stay finite
    router[:] = -40.0
    _, weight, _ = _route(torch.ones(3, 16), router, torch.zeros(8), 2, 2, 1, 1.0)
    assert torch.isfinite(weight).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,inner,limit,sharpness", [(7, 11, 0.8, 1.702), (5, 64, 1.5, 1.702),
                                                     (3, 20, 0.25, 0.9), (300, 512, 7.0, 1.702)])
def test_clipped_gate(dtype, n, inner, limit, sharpness):
    """The gate is cut above only, the other side on both; far beyond the limits too."""
    from distengine_b200.kernels import latent as lk
    x = (3.0 * torch.randn(n, 2 * inner, generator=_gen(inner))).to(dtype)
    x[0, 0], x[0, 1], x[1, inner], x[1, inner + 1] = 60.0, -60.0, 60.0, -60.0
    x[1, 0] = x[1, 1] = 0.5
    out = torch.empty(n, inner, dtype=dtype, device=DEV)
    lk.clipped_glu(x.to(DEV), out, limit, sharpness)
    gate, up = x.double().split(inner, dim=1)
    g, u = torch.clamp(gate, max=limit), torch.clamp(up, -limit, limit)
    assert_close(out, g * torch.sigmoid(sharpness * g) * (u + 1.0), dtype, "clipped gate")
    if sharpness == 1.702:
        assert_close(out, pp.clipped_gate(gate, up, limit), dtype, "clipped gate")


def _experts(dtype, width, mlp):
    from distengine_b200.parts import build_feed_forward
    r = mlp["router"]
    return build_feed_forward(_spec().of(
        "routed_experts", width=width, inner=mlp["expert"]["ff"], experts=r["experts"],
        top=r["top"], activation="clipped", gated=True, limit=mlp["expert"]["limit"],
        sharpness=1.702, scoring="grouped_sigmoid", bias_name="correction",
        groups=r["groups"]["count"], keep=r["groups"]["keep"], scale=r["scale"],
        shared_inner=mlp["shared"]["ff"], shared_limit=mlp["shared"]["limit"]), dtype,
        torch.device(DEV))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,n,mlp", [
    (42, 37, pc.moe(6, 2, 11, 3, 2, 1.7, 0.8, 13, 0.6)),          # odd sizes
    (64, 20, pc.moe(4, 4, 16, 2, 2, 0.5, 1.0, 8, 2.0)),           # every expert
    (40, 9, pc.moe(1, 1, 24, 1, 1, 1.0, 1.2, 16, 0.4)),           # one expert
    (72, 700, pc.moe(8, 3, 40, 4, 2, 2.5, 0.7, 56, 1.1)),         # many pairs
    (128, 400, pc.moe(32, 4, 96, 8, 2, 1.4, 1.0, 200, 1.5)),      # tiles that are mostly empty
    (256, 1100, pc.moe(4, 1, 136, 2, 1, 2.0, 0.9, 320, 0.8)),     # several tiles an expert
])
def test_routed_experts_beside_a_shared_one(dtype, width, n, mlp):
    """The whole feed-forward in both types (the plain function takes the engine's choice, which
    in 32-bit is its own), and in 32-bit cut into unequal steps."""
    ff = _experts(dtype, width, mlp)
    w = {k: v.float() for k, v in pp.draw(pp.mlp_shapes(mlp, width), _gen(n), 1.5).items()}
    assert {k: v[0] for k, v in ff.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
    ff.load(w)
    x = torch.randn(n, width, generator=_gen(6)).to(dtype)
    h = PartHarness([ff], [], dtype)
    caught = {}

    def fn(ctx, b):
        out = ff.forward(x.to(DEV), ctx).clone()
        caught["chosen"] = ctx.buffer("experts.chosen", (n, ff.top), torch.int32).clone().cpu()
        return out

    got = h.run([("a", n)], fn)
    assert got.dtype == torch.float32                       # joins the stream unrounded
    want = pp.routed_feed_forward(x.double(), _double(w), "", mlp, _act(dtype), caught["chosen"])
    assert_close(got, want, dtype, "routed experts")
    if dtype != torch.float32:
        return
    own = pp.routed_feed_forward(x.double(), _double(w), "", mlp)
    assert_close(own, want, dtype, "the engine's choice is the plain one's")
    for part in (slice(0, n // 3), slice(n // 3, n // 3 + 1), slice(n // 3 + 1, n)):
        xs = x[part].to(DEV)
        piece = h.run([("a", xs.shape[0])], lambda ctx, b: ff.forward(xs, ctx).clone())
        assert_close(piece, got[part], dtype, "a token's result depends on its step")


# ----------------------------------------------------------------------------- the block's norms
class _Norm:
    def __init__(self, weight, eps):
        self.weight, self.eps = weight.to(DEV), eps


@pytest.mark.parametrize("dtype,y_dtype", [(torch.float32, torch.float32),
                                           (torch.bfloat16, torch.bfloat16),
                                           (torch.bfloat16, torch.float32)])
@pytest.mark.parametrize("n,width", [(5, 42), (3, 64), (4, 700), (2, 2048), (3, 3000), (2, 8192),
                                     (2, 10000)])
def test_branch_norm_sum_vector_and_next_norm(dtype, y_dtype, n, width):
    """Every combination of branch norm, vector, picked rows and no output, with two different
    eps; a branch row of tiny numbers shows eps inside the root."""
    from distengine_b200.kernels import ops
    g = _gen(width)
    x, y = torch.randn(n, width, generator=g), torch.randn(n, width, generator=g).to(y_dtype)
    y[0] *= 1e-3
    vector = torch.randn(width, generator=g)
    wdt = torch.float32 if dtype == torch.float32 else torch.bfloat16
    after = _Norm((torch.rand(width, generator=g) + 0.5).to(wdt), 1e-5)
    before = _Norm((torch.rand(width, generator=g) + 0.5).to(wdt), 1e-3)
    rows = torch.tensor([n - 1, 0], dtype=torch.int32)

    def plain(with_y, with_norm, with_vector):
        new = x.double()
        if with_y:
            b = y.double()
            new = new + (pp.rms_norm(b, after.weight.cpu(), after.eps) if with_norm else b)
        if with_vector:
            new = new + vector.double()
        return new, pp.rms_norm(new, before.weight.cpu(), before.eps)

    for with_y, with_norm, with_vector in [(1, 1, 0), (1, 1, 1), (1, 0, 1), (0, 0, 1), (1, 0, 0)]:
        new, normed = plain(with_y, with_norm, with_vector)
        args = (y.to(DEV) if with_y else None, after if with_norm else None,
                vector.to(DEV) if with_vector else None)
        resid = x.to(DEV).clone()
        out = torch.empty(n, width, dtype=dtype, device=DEV)
        ops.join_rmsnorm(resid, *args, before, out)
        assert_close(resid, new, torch.float32, "the stream")
        assert_close(out, normed, dtype, "the next norm")
        resid = x.to(DEV).clone()
        picked = torch.empty(2, width, dtype=dtype, device=DEV)
        ops.join_rmsnorm(resid, *args, before, picked, rows.to(DEV))
        assert torch.equal(resid.cpu(), x)
        assert_close(picked, normed[rows.long()], dtype, "picked rows")
        ops.join_rmsnorm(resid, *args)
        assert_close(resid, new, torch.float32, "the sum alone")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,top", [(5, 42, 2), (3, 64, 1), (4, 1024, 5), (2, 9000, 3)])
def test_a_weighted_sum_is_formed_where_it_joins(dtype, n, width, top):
    """The experts' outputs and the shared expert's as the terms of a branch: weighted sum, branch
    norm, stream and next norm in one pass, with and without the shared rows."""
    from distengine_b200.kernels import ops
    from distengine_b200.parts.context import MixedRows
    g = _gen(width + top)
    x, rows = torch.randn(n, width, generator=g), torch.randn(n * top, width, generator=g).to(dtype)
    shared, side = torch.randn(n, width, generator=g).to(dtype), torch.rand(n, generator=g)
    weight = torch.rand(n, top, generator=g)
    after = _Norm((torch.rand(width, generator=g) + 0.5).to(dtype), 1e-5)
    before = _Norm((torch.rand(width, generator=g) + 0.5).to(dtype), 1e-6)
    total = (weight.double()[:, :, None] * rows.double().reshape(n, top, width)).sum(dim=1)
    for with_shared in (False, True):
        if with_shared:
            total = total + side.double()[:, None] * shared.double()
        extra = (shared.to(DEV), side.to(DEV)) if with_shared else ()
        resid, out = x.to(DEV).clone(), torch.empty(n, width, dtype=dtype, device=DEV)
        ops.join_rmsnorm(resid, MixedRows(rows.to(DEV), weight.to(DEV), *extra), after, None,
                         before, out)
        new = x.double() + pp.rms_norm(total, after.weight.cpu(), after.eps)
        assert_close(resid, new, torch.float32, "the stream")
        assert_close(out, pp.rms_norm(new, before.weight.cpu(), before.eps), dtype, "next norm")


@pytest.mark.parametrize("kind", ["rmsnorm", "grouped", "layernorm"])
def test_norms_fold_what_a_branch_norm_left_pending(kind):
    """A branch with its norm and a vector, read by norms that fold them themselves and by norms
    that have the stream settle first."""
    from distengine_b200.parts.base import build_norm
    from distengine_b200.parts.context import ResidualStream
    n, width, eps, g = 4, 48, 1e-5, _gen(3)
    x, y, v = (torch.randn(n, width, generator=g), torch.randn(n, width, generator=g),
               torch.randn(width, generator=g))
    wa, wb = torch.rand(width, generator=g) + 0.5, torch.rand(width, generator=g) + 0.5
    make = lambda name, **kw: build_norm(_spec().of(name, width=width, eps=eps, **kw),
                                         torch.float32, torch.device(DEV))
    after = make("branch_rmsnorm", tensor="w")
    after.load({"w": wa})
    with pytest.raises(RuntimeError):
        after.forward(None, None)
    new = x.double() + pp.rms_norm(y.double(), wa, eps) + v.double()
    if kind == "rmsnorm":
        norm, want = make("rmsnorm"), pp.rms_norm(new, wb, eps)
        norm.load({"weight": wb})
    elif kind == "grouped":
        norm = make("rmsnorm", groups=3)
        norm.load({"weight": wb})
        parts = new.reshape(n, 3, 16)
        want = (parts / pp.rms(parts, eps)).reshape(n, width) * wb.double()
    else:
        norm = make("layernorm")
        norm.load({"weight": wb, "bias": wa})
        c = new - new.mean(dim=1, keepdim=True)
        want = c / torch.sqrt((c * c).mean(dim=1, keepdim=True) + eps) * wb + wa

    def fn(ctx, b):
        stream = ResidualStream(x.to(DEV).clone())
        stream.pending, stream.pending_norm = y.to(DEV), after
        stream.add_vector(v.to(DEV))
        out = norm.forward(stream, ctx).clone()
        assert stream.pending is None and stream.pending_norm is None
        assert stream.pending_vector is None
        return out, stream.resid

    out, resid = PartHarness([], [], torch.float32).run([("a", n)], fn)
    assert_close(resid, new, torch.float32, "the stream")
    assert_close(out, want, torch.float32, kind)
