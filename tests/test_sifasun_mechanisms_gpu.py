"""Each mechanism of the Sifasun parts alone, built through the configuration and the registries and
run through the engine's step machinery, against the plain function in ``plain_sifasun``: both forms
of attention whose values are the projected keys, in portions and single tokens at sizes that are no
multiple of anything, with one key made decisive just inside and just outside the window (at page
borders, in prompts and in decoding), the term of one in the denominator, the cap, pages and slots
that are used again; the gated recurrence at odd and even sizes, in every cut, across the chunks'
borders, with long memory and fast decay; the joined product of two branches; the row kernel of the
block and the norm whose weight is stored around zero."""

import math

import pytest
import torch

import plain_sifasun as ps
import sifasun_configs as sc
from gpu_helpers import PartHarness, assert_close

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
WIDTH = 44


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _act(dtype):
    return None if dtype == torch.float32 else torch.bfloat16


def _build(mixer, dtype, width=WIDTH, seed=5, change=None, branch=None):
    """(the mixer, or one branch of it, as the model builds it; its weights' prefix; the weights in
    float64)."""
    from distengine_b200.config.sifasun import SifasunConfig
    from distengine_b200.parts import build_mixer
    config = sc.model(width, 16, [sc.layer(mixer, None)])
    spec, prefix = SifasunConfig.from_json(config).layer_specs()[0].mixer, "l0.mix."
    if branch is not None:
        name, spec = spec.params["branches"][branch]
        prefix += name + "."
    weights = ps.random_weights(config, seed)
    if change is not None:
        change(weights)
    part = build_mixer(spec, dtype, torch.device(DEV))
    part.load({local: weights[prefix + local] for local in part.tensors()})
    return part, prefix, {k: v.double() for k, v in weights.items()}


def _run_in_portions(mixer, h, xs, portions, release=()):
    fed = {rid: 0 for rid in xs}
    got = {rid: [] for rid in xs}
    for step in portions:
        entries = [(rid, n) for rid, n in step if n]
        x = torch.cat([xs[rid][fed[rid]: fed[rid] + n] for rid, n in entries]).to(DEV)
        out = h.run(entries, lambda ctx, b: mixer.forward(x, ctx, b[0]).float().clone()).cpu()
        at = 0
        for rid, n in entries:
            got[rid].append(out[at: at + n])
            at += n
            fed[rid] += n
    assert all(fed[rid] == xs[rid].shape[0] for rid in xs)
    return {rid: torch.cat(parts) for rid, parts in got.items()}


def _attention_out(x, wd, prefix, m, form, act=None):
    heads = ps.attention(x, wd, prefix, m, 1e-5, form, act=act)
    return ps.lin(heads, wd[prefix + "o"], act)


PORTIONS = [[("a", 30), ("b", 1)], [("a", 2), ("b", 1)], [("a", 1), ("b", 17)], [("a", 25)],
            [("a", 17), ("b", 21)]] + [[("a", 1), ("b", 1)]] * 6 + [[("a", 1)]]

ATTENTIONS = [
    # rows that are no 16-byte piece; an odd head size; a part of a head turned
    (sc.attention(6, 2, 5, 0.4, 7, (100.0, 2, 3.0), 2.0), 16),
    (sc.attention(6, 2, 10, 0.3, 16, (100.0, 6, 4.0), 1.5), 4),
    (sc.attention(3, 3, 6, 0.5, 17, (100.0, 6)), 16),              # half a part of odd size
    # whole pieces, up to 8 heads a kv head: single tokens take the one-block kernel
    (sc.attention(8, 1, 16, 0.25, 9, (30000.0, 16, 8.0), 4.0), 8),
    (sc.attention(8, 2, 32, 0.25, 8, (30000.0, 8), 50.0), 8),
    # more than 8 heads a kv head; everything seen; nothing turned
    (sc.attention(12, 1, 8, 0.3, None, (1000000.0, 4)), 16),
    (sc.attention(5, 5, 24, 0.3, 1), 8),
    (sc.attention(4, 4, 128, 0.1, 33, (500.0, 128, 2.0), 3.0), 32),
    (sc.attention(6, 3, 80, 0.12, 40, (500.0, 40)), 16),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", ["sink", "plain"])
@pytest.mark.parametrize("m,page", ATTENTIONS)
def test_attention_in_portions(dtype, form, m, page):
    """Two requests in unequal portions beside single tokens, then steps of single tokens only,
    against the plain function over each whole sequence; pages behind the window go back and are
    used again."""
    if form == "sink":
        mixer, prefix, wd = _build(m, dtype)
    else:
        m = {k: v for k, v in m.items() if k != "softcap"}
        mixer, prefix, wd = _build(sc.beside(m, 8, 2, 2, 1.0, 1.0), dtype, branch=0)
    g = _gen(5)
    xs = {"a": torch.randn(82, WIDTH, generator=g).to(dtype),
          "b": torch.randn(46, WIDTH, generator=g).to(dtype)}
    want = {rid: _attention_out(x.double(), wd, prefix, m, form, _act(dtype))
            for rid, x in xs.items()}
    h = PartHarness([mixer], [mixer.cache_spec()], dtype, page_size=page,
                    num_pages=4 + 160 // page)
    got = _run_in_portions(mixer, h, xs, PORTIONS)
    for rid in xs:
        assert_close(got[rid], want[rid], dtype, f"attention {form} {rid}")
    h.runner.cache.check_invariants()


def _far_setup(form, window, rot):
    """A mixer in which the last token's query is the far token's key: W_q reads the first half of
    the input as W_k reads the second."""
    dk, half = 32, WIDTH // 2
    m = sc.attention(4, 1, dk, 3.0 if form == "sink" else 1.5, window, rot)
    mixer = m if form == "sink" else sc.beside(m, 8, 2, 2, 1.0, 1.0)
    prefix = "l0.mix." if form == "sink" else "l0.mix.left."

    def change(w):
        w[prefix + "k"][:, :half] = 0
        wq = torch.zeros(dk, WIDTH)
        wq[:, :half] = w[prefix + "k"][:, half:]
        w[prefix + "q"] = wq.repeat(4, 1)
        if form == "plain":
            w[prefix + "q.norm"] = torch.ones(4 * dk)
            w[prefix + "k.norm"] = torch.ones(dk)

    return m, mixer, prefix, change, half


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", ["sink", "plain"])
@pytest.mark.parametrize("decoded", [0, 12])
@pytest.mark.parametrize("window,back", [(96, 95), (96, 96), (97, 96), (97, 97), (200, 199),
                                         (200, 200), (16, 15), (16, 16), (None, 300), (1, 1)])
def test_a_decisive_key_at_the_windows_edge(dtype, form, decoded, window, back):
    """One key among hundreds carries the last token's softmax if it is seen: just inside the
    window it must, just outside it must not, whatever page border it stands at; its value is its
    own key before the norm and the turn."""
    m, mixer_config, prefix, change, half = _far_setup(form, window, (1000000.0, 4))
    mixer, _, wd = _build(mixer_config, dtype, change=change,
                          branch=None if form == "sink" else 0)
    T = 330
    for seed, last in ((0, T - 1), (1, 320), (2, 319)):
        x = torch.randn(T, WIDTH, generator=_gen(40 * back + seed)).float()
        far = last - back
        x[last, :half] = 2.0 * x[far, half:]
        x = x[: last + 1].to(dtype)
        n = last + 1
        head = n - decoded
        portions = [[("a", head // 2)], [("a", head - head // 2)]] + [[("a", 1)]] * decoded
        h = PartHarness([mixer], [mixer.cache_spec()], dtype, page_size=16, num_pages=30)
        got = _run_in_portions(mixer, h, {"a": x}, portions)["a"]
        want = _attention_out(x.double(), wd, prefix, m, form, _act(dtype))
        assert_close(got, want, dtype, f"window {window} back {back}")
        # the key shows: a window one longer or one shorter gives something else
        if window is not None:
            other = dict(m, mask={"size": back if back < window else back + 1})
            differs = _attention_out(x.double(), wd, prefix, other, form, _act(dtype))[-1] - want[-1]
            assert differs.abs().max() > 0.15 * want.abs().max(), "the key decides nothing"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim", [(4, 2, 16), (3, 1, 10)])
def test_the_term_of_one_in_the_denominator(dtype, heads, kv_heads, dim):
    """Queries that oppose every key: all scores lie far below 0, the denominator is the added one
    and the results are nearly 0 (an ordinary softmax would average the values); and first tokens,
    which see themselves only."""
    m = sc.attention(heads, kv_heads, dim, 0.5, 40, None, 30.0)

    def change(w):
        w["l0.mix.q"] = -w["l0.mix.k"][:dim].repeat(heads, 1)
        w["l0.mix.k"] = w["l0.mix.k"][:dim].repeat(kv_heads, 1)

    mixer, prefix, wd = _build(m, dtype, change=change)
    base = torch.randn(1, WIDTH, generator=_gen(3))
    x = (base + 0.1 * torch.randn(50, WIDTH, generator=_gen(4))).to(dtype)
    want = _attention_out(x.double(), wd, prefix, m, "sink", _act(dtype))
    mean_value = ps.lin(ps.lin(x.double(), wd[prefix + "k"]).mean(0).reshape(kv_heads, dim)
                        .repeat_interleave(heads // kv_heads, 0).reshape(1, -1), wd[prefix + "o"])
    assert want.abs().max() < 0.5 * mean_value.abs().max()
    h = PartHarness([mixer], [mixer.cache_spec()], dtype, page_size=16, num_pages=8)
    got = _run_in_portions(mixer, h, {"a": x}, [[("a", 1)], [("a", 20)], [("a", 2)]]
                           + [[("a", 1)]] * 27)["a"]
    assert_close(got, want, dtype, "term of one")
    ordinary = ps.attention(x.double(), wd, prefix, m, 1e-5, "sink")
    s = ps.soft_cap(torch.tensor(-200.0, dtype=torch.float64), 30.0)
    assert -30.0 <= s < -29.9 and torch.isfinite(ordinary).all()


def test_the_cap_bends_the_scores():
    """Scores around a small cap: the capped softmax differs visibly from the plain one, and the
    engine follows the capped one in prompts and in decoding."""
    m = sc.attention(4, 2, 16, 1.0, 30, (100.0, 8), 1.5)
    mixer, prefix, wd = _build(m, torch.float32)
    x = torch.randn(60, WIDTH, generator=_gen(6))
    want = _attention_out(x.double(), wd, prefix, m, "sink")
    uncapped = _attention_out(x.double(), wd, prefix, dict(m, softcap=None), "sink")
    assert (want - uncapped).abs().max() > 0.1
    h = PartHarness([mixer], [mixer.cache_spec()], torch.float32, page_size=8, num_pages=12)
    got = _run_in_portions(mixer, h, {"a": x}, [[("a", 40)]] + [[("a", 1)]] * 20)["a"]
    assert_close(got, want, torch.float32, "cap")


def test_pages_and_slots_that_are_used_again():
    """Requests one after the other through one slot and a pool that holds one of them."""
    m = sc.beside(sc.attention(4, 2, 8, 0.4, 10, (100.0, 4)), 24, 2, 3, 0.6, 1.0)
    mixer, prefix, wd = _build(m, torch.float32)
    h = PartHarness([mixer], [mixer.cache_spec()], torch.float32, page_size=4, num_pages=6,
                    max_seqs=1, max_len=24)
    for i in range(4):
        x = torch.randn(19, WIDTH, generator=_gen(60 + i))
        got = _run_in_portions(mixer, h, {f"r{i}": x}, [[(f"r{i}", 11)], [(f"r{i}", 5)]]
                               + [[(f"r{i}", 1)]] * 3)[f"r{i}"]
        want = ps.mixer("parallel", x.double(), wd, "l0.mix.", m, 1e-5)
        assert_close(got, want, torch.float32, f"request {i}")
        h.runner.release(f"r{i}")
    h.runner.cache.check_invariants()


# ----------------------------------------------------------------------------- gated recurrence
RECURRENCES = [(15, 3, 4), (24, 1, 1), (40, 5, 2), (64, 2, 4), (96, 1, 3), (96, 3, 6), (160, 2, 4),
               (256, 2, 4), (48, 6, 5), (7, 7, 4), (272, 2, 2)]


def _recurrence(width, blocks, taps, dtype, change=None, seed=5):
    mixer = sc.beside(sc.attention(1, 1, 4, 1.0, 3), width, blocks, taps, 1.0, 1.0)
    part, prefix, wd = _build(mixer, dtype, branch=1, change=change, seed=seed)

    def plain(x, act=None):
        rows = ps.gated_recurrence(x, wd, prefix, mixer["right"], act)
        return ps.lin(rows, wd[prefix + "o"], act)

    return part, prefix, plain


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,blocks,taps", RECURRENCES)
def test_recurrence_in_portions(dtype, width, blocks, taps):
    """Portions of one to 150 tokens of three requests side by side, so that sequences begin and
    end inside the chunks of a step and on their borders, then single tokens only."""
    part, _, plain = _recurrence(width, blocks, taps, dtype)
    g = _gen(7)
    xs = {"a": torch.randn(240, WIDTH, generator=g).to(dtype),
          "b": torch.randn(96, WIDTH, generator=g).to(dtype),
          "c": torch.randn(75, WIDTH, generator=g).to(dtype)}
    h = PartHarness([part], [part.cache_spec()], dtype)
    portions = [[("a", 64), ("b", 1), ("c", 63)], [("a", 2), ("b", 62), ("c", 1)],
                [("b", 3), ("a", 150)], [("a", 3), ("c", 2), ("b", 1)], [("b", 19), ("a", 1)],
                [("a", 17), ("b", 2)]] + [[("a", 1), ("b", 1), ("c", 1)]] * 3 \
        + [[("b", 1), ("c", 1)]] * 5 + [[("c", 1)]]
    got = _run_in_portions(part, h, xs, portions)
    for rid, x in xs.items():
        assert_close(got[rid], plain(x.double(), _act(dtype)), dtype, f"recurrence {rid}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,blocks,taps", [(64, 2, 4), (15, 3, 4)])
def test_every_cut_of_a_sequence(dtype, width, blocks, taps):
    part, _, plain = _recurrence(width, blocks, taps, dtype)
    x = torch.randn(140, WIDTH, generator=_gen(8)).to(dtype)
    want = plain(x.double(), _act(dtype))
    for size in (1, 2, 3, 63, 64, 65, 128, 140):
        h = PartHarness([part], [part.cache_spec()], dtype)
        portions = [[("a", min(size, 140 - at))] for at in range(0, 140, size)]
        got = _run_in_portions(part, h, {"a": x}, portions)["a"]
        assert_close(got, want, dtype, f"portions of {size}")


@pytest.mark.parametrize("lam,bias", [(-12.0, 0.0), (-9.0, -4.0), (3.0, 2.0), (30.0, 3.0)])
@pytest.mark.parametrize("portion", [400, 70, 1])
def test_long_memory_and_fast_decay(lam, bias, portion):
    """Channels that keep nearly everything over hundreds of tokens (the first token, made large,
    still shows at the end) and channels that forget within a token (the products of decays run
    out of range)."""
    def change(w):
        p = "l0.mix.right."
        w[p + "lam"] = torch.full_like(w[p + "lam"], lam)
        w[p + "ra.b"] = torch.full_like(w[p + "ra.b"], bias)

    part, prefix, plain = _recurrence(32, 2, 3, torch.float32, change)
    T = 400 if portion > 1 else 90
    x = torch.randn(T, WIDTH, generator=_gen(9))
    x[0] *= 20.0
    want = plain(x.double())
    h = PartHarness([part], [part.cache_spec()], torch.float32)
    got = _run_in_portions(part, h, {"a": x},
                           [[("a", min(portion, T - at))] for at in range(0, T, portion)])["a"]
    assert torch.isfinite(got).all()
    assert_close(got, want, torch.float32, f"lam {lam}")
    if lam < -8:
        quiet = x.clone()
        quiet[0] = 0
        assert (plain(quiet.double())[-1] - want[-1]).abs().max() > 1e-2


def test_a_slot_starts_at_zero_again():
    part, _, plain = _recurrence(64, 2, 4, torch.float32)
    h = PartHarness([part], [part.cache_spec()], torch.float32, max_seqs=1)
    for i, head in enumerate((1, 2, 30, 66)):
        x = torch.randn(head + 3, WIDTH, generator=_gen(80 + i))
        got = _run_in_portions(part, h, {f"r{i}": x}, [[(f"r{i}", head)]] + [[(f"r{i}", 1)]] * 3)
        assert_close(got[f"r{i}"], plain(x.double()), torch.float32, f"request {i}")
        h.runner.release(f"r{i}")


@pytest.mark.parametrize("count", [1, 15, 16, 17, 40])
def test_many_single_tokens_in_a_step(count):
    """Steps of single tokens of more sequences than a block takes, each at another position."""
    part, _, plain = _recurrence(96, 3, 4, torch.bfloat16)
    xs = {f"r{i}": torch.randn(3 + i % 5, WIDTH, generator=_gen(200 + i)).to(torch.bfloat16)
          for i in range(count)}
    h = PartHarness([part], [part.cache_spec()], torch.bfloat16, max_seqs=count)
    longest = max(x.shape[0] for x in xs.values())
    portions = [[(r, 1) for r, x in xs.items() if x.shape[0] > at] for at in range(longest)]
    got = _run_in_portions(part, h, xs, portions)
    for rid, x in xs.items():
        assert_close(got[rid], plain(x.double(), torch.bfloat16), torch.bfloat16, rid)


# ----------------------------------------------------------------------------- both branches
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mixer", [
    sc.beside(sc.attention(3, 1, 7, 0.3, 21, (1000.0, 4)), 15, 3, 4, 0.7, 1.2),    # padded segments
    sc.beside(sc.attention(8, 2, 16, 0.3, 9, (5000.0, 8)), 48, 3, 2, -1.5, 0.4),
    sc.beside(sc.attention(4, 4, 8, 0.3, 70, (5000.0, 8)), 64, 2, 4, 0.0, 1.0),
    sc.beside(sc.attention(4, 4, 8, 0.3, 70, (5000.0, 8)), 64, 2, 4, 1.0, 0.0)])
def test_two_branches_in_one_product(dtype, mixer):
    part, _, wd = _build(mixer, dtype)
    g = _gen(11)
    xs = {"a": torch.randn(82, WIDTH, generator=g).to(dtype),
          "b": torch.randn(46, WIDTH, generator=g).to(dtype)}
    h = PartHarness([part], [part.cache_spec()], dtype, page_size=8, num_pages=30)
    got = _run_in_portions(part, h, xs, PORTIONS)
    for rid, x in xs.items():
        want = ps.mixer("parallel", x.double(), wd, "l0.mix.", mixer, 1e-5, _act(dtype))
        assert_close(got[rid], want, dtype, f"branches {rid}")


# ----------------------------------------------------------------------------- block
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [33, 44, 512, 1536, 4100, 9000])
def test_branch_norm_sum_and_rounding(dtype, width):
    """x + norm(y) with a weight stored around zero, in place, and its rounding for the products
    that read the stream itself."""
    from distengine_b200.kernels import ops
    from distengine_b200.parts import build_norm
    from distengine_b200.config.model import PartSpec
    g = _gen(width)
    x, y = torch.randn(5, width, generator=g), (3 * torch.randn(5, width, generator=g)).to(dtype)
    stored = (0.4 * torch.randn(width, generator=g)).to(torch.bfloat16)
    norm = build_norm(PartSpec.of("branch_rmsnorm", width=width, eps=1e-5, tensor="w", offset=1.0),
                      dtype, torch.device(DEV))
    norm.load({"w": stored})
    assert norm.weight.dtype == torch.float32
    want = x.double() + ps.plus_one_norm(y.double(), stored.double(), 1e-5)
    resid = x.to(DEV).contiguous()
    rows = torch.empty(5, width, dtype=dtype, device=DEV)
    ops.join_rmsnorm(resid, y.to(DEV), norm, out=rows)
    assert_close(resid, want, torch.float32, "stream")
    assert torch.equal(rows, resid.to(dtype))


def test_a_final_norm_with_a_gain():
    from distengine_b200.config.model import PartSpec
    from distengine_b200.parts import build_norm
    stored = (0.4 * torch.randn(40, generator=_gen(1))).to(torch.bfloat16)
    norm = build_norm(PartSpec.of("rmsnorm", width=40, eps=1e-5, tensor="w", offset=1.0, gain=1.7),
                      torch.bfloat16, torch.device(DEV))
    norm.load({"w": stored})
    assert_close(norm.weight, (1.0 + stored.double()) * 1.7, torch.float32, "weight")


def test_what_the_mixers_refuse():
    from distengine_b200.parts.gated_recurrence import GatedRecurrence
    from distengine_b200.parts.sink_attention import SinkAttention
    dev, f32 = torch.device("cpu"), torch.float32
    with pytest.raises(ValueError, match="blocks"):
        GatedRecurrence(8, 10, 3, 4, f32, dev)
    with pytest.raises(ValueError, match="taps"):
        GatedRecurrence(8, 10, 2, 17, f32, dev)
    with pytest.raises(ValueError, match="values that are keys"):
        SinkAttention(8, 2, 1, 4, 6, 1.0, 1e-5, f32, dev, values_from_keys=True)
    with pytest.raises(ValueError, match="window"):
        SinkAttention(8, 2, 1, 4, 4, 1.0, 1e-5, f32, dev, window=0)
    assert math.isclose(float(ps.softplus(torch.tensor(0.0))), math.log(2.0), rel_tol=1e-6)
