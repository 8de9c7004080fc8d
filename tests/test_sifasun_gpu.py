"""The Sifasun architecture through the engine against the plain implementation
(``plain_sifasun``): whole prompts, prefill against token-by-token decoding, portions down to two
tokens, mixed batches on pools so small that pages and slots are used again (freed pages
poisoned), the residual stream after every layer run, long decoding (also as CUDA graphs), a long
prompt at wide sizes, models of random sizes, and greedy generation through ``Engine`` and the
command line."""

import os
import tempfile

import numpy as np
import pytest
import torch

import plain_sifasun as ps
import sifasun_configs as sc
import trace_helpers as th
from gpu_helpers import assert_close

pytestmark = pytest.mark.gpu
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
LENGTHS = [70, 33, 100, 5, 64, 17, 90, 48, 1, 2]

_cache: dict = {}


def _plain(config, weights, ids, dtype_name):
    act = None if dtype_name == "float32" else torch.bfloat16
    return ps.forward(config, weights, ids, act=act).to(torch.float32).numpy()


def _model(name, model_root):
    if name not in _cache:
        folder, weights = sc.make_folder(name, model_root)
        requests = {f"r{i}": sc.tokens(name, n, i) for i, n in enumerate(LENGTHS)}
        reference = {dtype: {rid: _plain(sc.ALL[name], weights, t, dtype)
                             for rid, t in requests.items()} for dtype in DTYPES}
        _cache[name] = (folder, weights, requests, reference)
    return _cache[name]


def _replay(runner, steps, vocab):
    with tempfile.TemporaryDirectory() as out:
        th.replay_in_process(runner, steps, out)
        return th.collect(steps, out, vocab)


def _schedules(requests):
    return {
        "whole": (th.schedule_whole(requests), 128),
        "tail": (th.schedule_tail(requests, 32), 128),
        "portions": (th.schedule_portions(requests), 128),
        "pairs": (th.schedule_portions(requests, sizes=(2,)), 128),
        "mixed": (th.schedule_mixed(requests, 320, seed=3), 320),
        "mixed_tight": (th.schedule_mixed(requests, 192, seed=11, decode_tail=32), 192),
    }


# bfloat16 bounds of this file, as shares of a position's largest logit; the 32-bit runs are the
# sharp test (gpu_helpers.F32_REL).  A sublayer's result is divided by its own root mean square, so
# in these tiny models a small result, and its rounding, is normed up to full size.  One position in
# ten may lie over the bound, and the median is bounded too.
BF16_MAX, BF16_RMS, BF16_MEDIAN = 8e-2, 2e-2, 1.5e-2


def _compare(rows, reference, dtype, what):
    assert rows, "the replay wrote nothing"
    rms, over = [], []
    for (rid, position), got in rows.items():
        want = reference[rid][position]
        if dtype == torch.float32:
            assert_close(got, want, dtype, f"{what} {rid}@{position}")
            continue
        assert np.isfinite(got).all(), f"{what} {rid}@{position}: not finite"
        err, scale = np.abs(got - want), np.abs(want).max()
        rms.append(float(np.sqrt((err ** 2).mean()) / scale))
        if rms[-1] > BF16_RMS or err.max() > BF16_MAX * scale:
            over.append(f"{rid}@{position}: rms {rms[-1]:.3f}, max {err.max() / scale:.3f}")
    if rms:
        assert len(over) <= max(1, len(rms) // 10) and np.median(rms) <= BF16_MEDIAN, (
            f"{what}: {len(over)} of {len(rms)} positions over the bound, median rms "
            f"{np.median(rms):.3e} of the largest logit; " + "; ".join(over[:5]))


@pytest.mark.parametrize("name", ["sif_a", "sif_b", "sif_c"])
@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("schedule", ["whole", "tail", "portions", "pairs", "mixed", "mixed_tight"])
def test_replay_matches_plain(name, dtype_name, schedule, model_root):
    from distengine_b200.engine.replay import build_runner
    folder, _, requests, reference = _model(name, model_root)
    steps, max_tokens = _schedules(requests)[schedule]
    runner = build_runner(folder, dtype_name, max_tokens, page_size=sc.PAGES[name],
                          poison_freed_pages=True, live_requests=4)
    rows = _replay(runner, steps, sc.ALL[name]["vocab"])
    runner.cache.check_invariants()
    assert not runner.cache.live
    assert len(rows) == sum(len(e["want"]) for s in steps for e in s["entries"])
    _compare(rows, reference[dtype_name], DTYPES[dtype_name], f"{name} {schedule}")


@pytest.mark.parametrize("name", ["sif_a", "sif_b"])
def test_float32_cuts_agree_closely(name, model_root):
    """However a request is cut, its 32-bit logits agree far inside the tolerance."""
    from distengine_b200.engine.replay import build_runner
    folder, _, requests, _ = _model(name, model_root)
    got = {}
    for schedule in ("whole", "tail", "pairs", "mixed"):
        steps, max_tokens = _schedules(requests)[schedule]
        runner = build_runner(folder, "float32", max_tokens, page_size=sc.PAGES[name])
        got[schedule] = _replay(runner, steps, sc.ALL[name]["vocab"])
    for schedule in ("tail", "pairs", "mixed"):
        for key, row in got[schedule].items():
            scale = np.abs(got["whole"][key]).max()
            np.testing.assert_allclose(row, got["whole"][key], rtol=0, atol=2e-5 * max(scale, 1.0),
                                       err_msg=f"{schedule} {key}")


@pytest.mark.parametrize("name", ["sif_a", "sif_b", "sif_c"])
def test_the_stream_after_every_layer(name, model_root):
    """The residual stream behind every layer run, 32-bit: norms on the sublayers' results, layers
    that use another layer's weights."""
    from distengine_b200.engine.replay import build_runner
    from distengine_b200.engine.step import StepEntry
    from distengine_b200.parts import block as blocks
    folder, weights = sc.make_folder(name, model_root)
    ids = sc.tokens(name, 23, 9)
    want: list = []
    ps.forward(sc.ALL[name], weights, ids, layers=want)
    caught = []
    original = blocks.SublayerNormBlock.forward

    def forward(self, stream, ctx, cache, following=None):
        original(self, stream, ctx, cache, following)
        stream.settle()
        caught.append(stream.resid.clone())

    blocks.SublayerNormBlock.forward = forward
    try:
        runner = build_runner(folder, "float32", 64, page_size=8)
        runner.step([StepEntry("t", ids, [22])])
        runner.check_status()
    finally:
        blocks.SublayerNormBlock.forward = original
    assert len(caught) == len(want) == len(sc.ALL[name]["layers"])
    for index, (got, ref) in enumerate(zip(caught, want)):
        assert_close(got, ref, torch.float32, f"{name}: stream after run {index}")


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["sif_a", "sif_b"])
def test_long_decoding_with_graphs(name, dtype_name, model_root):
    """A short prompt, then 220 tokens one by one over many page borders and windows (pages
    behind the windows are given back, the convolution's kept rows go round at every token), also
    replayed as CUDA graphs."""
    from distengine_b200.engine.replay import build_runner
    folder, weights = sc.make_folder(name, model_root)
    ids = sc.tokens(name, 230, 77)
    steps = th.schedule_tail({"long": ids}, 220)
    want = {"long": _plain(sc.ALL[name], weights, ids, dtype_name)}
    runner = build_runner(folder, dtype_name, 256, page_size=16, poison_freed_pages=True)
    rows = _replay(runner, steps, sc.ALL[name]["vocab"])
    _compare(rows, want, DTYPES[dtype_name], "long decode")
    runner = build_runner(folder, dtype_name, 256, page_size=16, use_graphs=True,
                          poison_freed_pages=True)
    graphed = _replay(runner, steps, sc.ALL[name]["vocab"])
    assert runner.graph_replays > 100 and graphed.keys() == rows.keys()
    for key, row in rows.items():
        np.testing.assert_allclose(graphed[key], row, rtol=0, atol=1e-5 * np.abs(row).max(),
                                   err_msg=f"graphs {key}")


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_a_long_prompt_at_wide_sizes(dtype_name, model_root):
    """1,100 tokens in one step (products of a thousand rows and more, attention tiles of 64 rows,
    many chunks of the recurrence), then tokens one by one, then the same prompt in two uneven
    portions."""
    from distengine_b200.engine.replay import build_runner
    name = "sif_wide"
    folder, weights = sc.make_folder(name, model_root)
    ids = sc.tokens(name, 1112, 3)
    picked = [0, 1, 15, 16, 17, 63, 64, 65, 255, 256, 599, 999, 1000, 1001, 1099]
    head = {"step": 0, "end": [], "entries": [{"id": "w", "tokens": ids[:1100], "want": picked}]}
    tail = [{"step": 1 + i, "end": ["w"] if i == 11 else [],
             "entries": [{"id": "w", "tokens": [ids[1100 + i]], "want": [0]}]} for i in range(12)]
    cut = [{"step": 13, "end": [], "entries": [{"id": "c", "tokens": ids[:1027], "want": [1026]}]},
           {"step": 14, "end": ["c"], "entries": [{"id": "c", "tokens": ids[1027:],
                                                    "want": [0, 84]}]}]
    steps = [head] + tail + cut
    runner = build_runner(folder, dtype_name, 1152, page_size=16, poison_freed_pages=True)
    rows = _replay(runner, steps, sc.ALL[name]["vocab"])
    whole = _plain(sc.ALL[name], weights, ids, dtype_name)
    assert len(rows) == len(picked) + 12 + 3
    _compare(rows, {"w": whole, "c": whole}, DTYPES[dtype_name], f"wide {dtype_name}")


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_batch_of_unequal_requests_against_each_alone(dtype_name, model_root):
    """Four unequal requests in one step give what each gives alone."""
    from distengine_b200.engine.replay import build_runner
    from distengine_b200.engine.step import StepEntry
    name = "sif_b"
    folder, _, requests, reference = _model(name, model_root)
    picked = ["r0", "r3", "r8", "r5"]
    runner = build_runner(folder, dtype_name, 512, page_size=8)
    entries = [StepEntry(r, requests[r], list(range(len(requests[r])))) for r in picked]
    logits = runner.step(entries).cpu().numpy()
    runner.check_status()
    at, rows = 0, {}
    for r in picked:
        for i in range(len(requests[r])):
            rows[(r, i)] = logits[at + i]
        at += len(requests[r])
    _compare(rows, reference[dtype_name], DTYPES[dtype_name], "batched")


def _random_config(rng) -> dict:
    """A model of random sizes: both mixers in random order, layers that use another's weights,
    feed-forwards present or not."""
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]

    def heads(capped):
        kv = int(pick(1, 2, 3))
        dim = int(pick(3, 6, 8, 16, 20, 32))
        turned = int(pick(*[d for d in (0, 2, 4, 6, 8, 16) if d <= dim]))
        rot = (float(pick(20.0, 10000.0, 500000.0)), turned)
        if capped and rng.random() < 0.7:
            rot += (float(pick(0.5, 2.0, 8.0)),)
        return sc.attention(kv * int(pick(1, 2, 3, 9)), kv, dim, float(pick(0.1, 0.3, 1.0)),
                            pick(1, 2, 7, 16, 17, 30, 64, 500), rot if turned else None,
                            float(pick(1.0, 5.0, 50.0)) if capped else None)

    layers = []
    for i in range(int(pick(1, 2, 3, 4, 5))):
        own = [j for j in range(i) if "weights_of" not in layers[j]]
        if own and rng.random() < 0.4:
            j = int(pick(*own))
            layers.append(dict(layers[j], weights_of=j))
            continue
        if rng.random() < 0.5:
            mixer = heads(True)
        else:
            blocks = int(pick(1, 2, 3, 4))
            mixer = sc.beside(heads(False), blocks * int(pick(1, 5, 8, 16, 24, 32, 72)), blocks,
                              int(pick(1, 2, 3, 4, 6)), float(pick(0.5, 1.0, -0.7)),
                              float(pick(0.4, 1.0, 2.0)))
        layers.append(sc.layer(mixer, int(pick(4, 17, 32)) if rng.random() < 0.7 else None))
    return sc.model(int(pick(24, 40, 56, 72, 35)), int(pick(50, 111)), layers,
                    float(pick(1e-5, 1e-6)), float(pick(0.5, 1.0, 2.5)))


@pytest.mark.parametrize("seed", range(10))
def test_models_of_random_sizes_under_a_mixed_schedule(seed, model_root):
    from distengine_b200.engine.replay import build_runner
    rng = np.random.default_rng(4000 + seed)
    config = _random_config(rng)
    weights = ps.random_weights(config, 90 + seed)
    folder = sc.write_folder(config, os.path.join(model_root, f"sif_random_{seed}"), weights)
    requests = {f"q{i}": [int(t) for t in rng.integers(0, config["vocab"], size=n)]
                for i, n in enumerate((61, 9, 80, 2, 35, 50))}
    want = {rid: _plain(config, weights, t, "float32") for rid, t in requests.items()}
    steps = th.schedule_mixed(requests, 256, seed=seed, decode_tail=20)
    for graphs in (False, True):
        runner = build_runner(folder, "float32", 256, page_size=int(rng.choice([4, 8, 16])),
                              poison_freed_pages=True, use_graphs=graphs)
        rows = _replay(runner, steps, config["vocab"])
        runner.cache.check_invariants()
        _compare(rows, want, torch.float32, f"random model {seed} graphs={graphs}")
    runner = build_runner(folder, "bfloat16", 256, page_size=16, poison_freed_pages=True)
    want = {rid: _plain(config, weights, t, "bfloat16") for rid, t in requests.items()}
    _compare(_replay(runner, steps, config["vocab"]), want, torch.bfloat16,
             f"random model {seed} bfloat16")


def test_greedy_generation_through_the_engine(model_root):
    """``Engine.generate`` (scheduler, portions of prompts under a small token budget, sampling,
    step-ahead decoding with steps taken back) gives the plain implementation's greedy tokens in
    32-bit."""
    from distengine_b200 import Engine, EngineConfig
    name = "sif_a"
    folder, weights = sc.make_folder(name, model_root)
    prompts = [sc.tokens(name, n, 40 + i) for i, n in enumerate((3, 29, 50, 11, 1))]
    new = 12
    want = [ps.greedy(sc.ALL[name], weights, p, new) for p in prompts]
    engine = Engine(folder, EngineConfig(dtype="float32", block_size=16, num_blocks=24,
                                         decode_batch_size=3, max_batch_tokens=32,
                                         max_model_len=128))
    assert engine.generate(prompts, new) == want
    engine.cache.check_invariants()
    engine = Engine(folder, EngineConfig(dtype="bfloat16", block_size=16, num_blocks=24,
                                         decode_batch_size=3, max_batch_tokens=32,
                                         max_model_len=128))
    got = engine.generate(prompts, new)
    for prompt, tokens in zip(prompts, got):
        logits = ps.forward(sc.ALL[name], weights, prompt)[-1]
        gap = (logits.max() - logits[tokens[0]]).item()
        assert len(tokens) == new and gap <= 0.25 * logits.abs().max().item()


def test_preempted_requests_are_recomputed(model_root):
    """So few pages that running requests are preempted: they give back their pages and their
    slot, and cache and states are built again from their tokens; the greedy tokens stay the plain
    implementation's."""
    from distengine_b200 import Engine, EngineConfig
    name = "sif_c"
    folder, weights = sc.make_folder(name, model_root)
    prompts = [sc.tokens(name, n, 60 + i) for i, n in enumerate((30, 27, 33))]
    new = 24
    engine = Engine(folder, EngineConfig(dtype="float32", block_size=16, num_blocks=5,
                                         decode_batch_size=3, max_batch_tokens=48,
                                         max_model_len=64))
    assert engine.generate(prompts, new) == [ps.greedy(sc.ALL[name], weights, p, new)
                                             for p in prompts]
    assert engine.scheduler.num_preemptions > 0
    engine.cache.check_invariants()
    assert not engine.cache.live


def test_the_command_line_generates(model_root):
    import subprocess
    import sys
    folder, _ = sc.make_folder("sif_b", model_root)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    result = subprocess.run([sys.executable, "-m", "distengine_b200", "generate", "--model", folder,
                             "--prompt-ids", "5 17 3", "--max-new-tokens", "4", "--dtype",
                             "float32", "--num-blocks", "16", "--decode-batch-size", "2"],
                            cwd=root, capture_output=True, text=True, timeout=600)
    assert result.returncode == 0, result.stderr[-2000:]
    assert "Generated token IDs" in result.stdout
