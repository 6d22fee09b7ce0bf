"""The Radilix decoder on the GPU through the engine's own step function, cache manager and scheduler, against the plain
implementation in float64: every way of cutting (whole; most in one step and the last tokens one by one; portions of
changing size down to two tokens; mixed batches of unequal requests on a poisoned pool), tight pools whose pages and state
slots have several owners, long decoding, the first tokens, other page sizes, a request against itself in other company,
captured against eager steps, a marked token found again far away by each mixer, greedy generation through `LLMEngine`
with a preemption, a model of states alone, and the replay and command-line programs."""

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests.gpu_common import replay
from tests.helpers import mixed_trace, portions_trace, random_tokens, read_weights, tail_decode_trace, whole_trace
from tests.radilix_configs import ASKER, MARK, RADILIX, make_radilix_folder, planted_pair
from tests.plain import plain_radilix as pr

pytestmark = pytest.mark.gpu
LENGTHS = {"A": [5, 47, 1, 130, 2, 64, 33], "B": [5, 17, 150, 70, 1, 90, 2], "C": [40, 3, 25, 1, 18], "D": [30, 2, 300, 140],
           "E": [50, 3, 1, 90, 20]}
_cache = {}

# float32 kernels against float64: rounding alone stays far below this, a key wrongly seen or a lost state does not.
# bfloat16: three times what rounding alone causes in that request, measured with the plain implementation rounding its
# products' inputs and outputs (both sides see the weights rounded to bfloat16).  A router whose choice hangs on less
# than CLOSE_CALL of a score may choose otherwise once its input is rounded; from the first such token on a request is
# another one, and only its median is compared.
LIMIT_FLOAT32 = 3e-5
CLOSE_CALL = 1e-2


def distance(got, want, scale):
    """Per position: the root mean square over the vocabulary of the difference of the logits, each
    with its mean taken off, in units of the logits' own spread."""
    d = got.astype(np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / scale


class Wanted:
    """What a request's logits should be, and how far rounding may move them."""

    def __init__(self, raw, weights, tokens, dtype, scale=None):
        self.scale, self.sure, self.median = scale, np.ones(len(tokens), dtype=bool), np.inf
        if dtype == "float32":
            self.logits, self.limit = pr.forward(raw, weights, tokens).numpy(), LIMIT_FLOAT32
        else:
            weights = {k: (v.to(torch.bfloat16).float() if v.dim() >= 2 else v) for k, v in weights.items()}
            gaps = []
            self.logits = pr.forward(raw, weights, tokens, margins=gaps).numpy()
            rough = pr.forward(raw, weights, tokens, rounding=True).numpy()
        self.scale = scale or float(np.sqrt(np.var(self.logits, axis=-1).mean()))
        if dtype != "float32":
            err = distance(rough, self.logits, self.scale)
            if gaps:
                self.sure = np.cumsum(torch.stack(gaps).min(0).values.numpy() < CLOSE_CALL) == 0
            # (a request with a close call near its start has few sure positions to take the largest error from)
            typical = float(np.median(err))
            self.limit = max(2e-2, 3.0 * max(float(np.where(self.sure, err, 0.0).max()), 1.5 * typical))
            self.median = max(3e-2, 3.0 * typical)

    def check(self, got, what, rows=slice(None)):
        want, sure = self.logits[rows], self.sure[rows]
        assert got.shape == want.shape, f"{what}: shape {got.shape} vs {want.shape}"
        assert np.isfinite(got).all(), f"{what}: not finite"
        err = distance(got, want, self.scale)
        bad = np.nonzero(sure & (err > self.limit))[0]
        assert not len(bad), f"{what}: position {int(bad[0])} is off by {err[bad].max():.3e} (limit {self.limit:.1e})"
        if len(err) > 8:
            assert np.median(err) <= self.median, f"{what}: the median is off by {np.median(err):.3e}"


def reference(key, dtype, tmp_path_factory):
    """folder, requests, {id: Wanted}, scale"""
    if key not in _cache:
        folder = make_radilix_folder(tmp_path_factory.mktemp(f"radilix_{key}"), key)
        weights = read_weights(folder)
        requests = {f"r{i}": random_tokens(RADILIX[key]["vocab"], n, 300 + i) for i, n in enumerate(LENGTHS[key])}
        _cache[key] = (folder, weights, requests)
    folder, weights, requests = _cache[key]
    if (key, dtype) not in _cache:
        first = {i: Wanted(RADILIX[key], weights, tokens, "float32") for i, tokens in requests.items()}
        scale = float(np.sqrt(np.mean([np.var(w.logits, axis=-1).mean() for w in first.values()])))
        _cache[(key, dtype)] = ({i: Wanted(RADILIX[key], weights, tokens, dtype, scale) for i, tokens in requests.items()}, scale)
    want, scale = _cache[(key, dtype)]
    return folder, requests, want, scale


WAYS = {
    "whole": lambda reqs: whole_trace(reqs),
    "tail": lambda reqs: tail_decode_trace(reqs, 45),
    "portions": lambda reqs: portions_trace(reqs, [7, 2, 5, 3, 2, 15, 16, 17, 2, 31, 33]),
    "long_portions": lambda reqs: portions_trace(reqs, [64, 33, 2, 70, 1]),
    "mixed": lambda reqs: mixed_trace(reqs, seed=3),
    "mixed_other_order": lambda reqs: mixed_trace(dict(reversed(list(reqs.items()))), seed=11),
}


@pytest.mark.parametrize("way", list(WAYS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key,page", [("A", 16), ("B", 16), ("A", 8), ("B", 24), ("C", 4), ("C", 32), ("D", 16), ("D", 64), ("E", 16)])
def test_replay_matches_plain(tmp_path_factory, key, page, dtype, way):
    folder, requests, want, _ = reference(key, dtype, tmp_path_factory)
    steps = WAYS[way](requests)
    got, session = replay(folder, dtype, steps, poison=way.startswith("mixed"), page_size=page, max_live=4)
    assert session.runner.cache.whole(), "pages or slots were not given back"
    for ident in requests:
        want[ident].check(got[ident], f"{key} page {page} {dtype} {way} {ident}")


def pages_needed(steps, page):
    held, worst = {}, 0
    for record in steps:
        for entry in record["entries"]:
            held[entry["id"]] = held.get(entry["id"], 0) + len(entry["tokens"])
        worst = max(worst, sum(-(-n // page) for n in held.values()))
        for ident in record["end"]:
            held.pop(ident, None)
    return worst


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key,page", [("A", 8), ("B", 16), ("D", 16)])
def test_pages_and_slots_have_several_owners_on_a_tight_pool(tmp_path_factory, key, page, dtype):
    folder, requests, want, _ = reference(key, dtype, tmp_path_factory)
    steps = mixed_trace(requests, seed=5, max_live=3)
    num_pages = pages_needed(steps, page)
    assert num_pages < sum(-(-len(t) // page) for t in requests.values())
    got, session = replay(folder, dtype, steps, num_pages=num_pages, page_size=page, max_live=3, poison=True)
    shared = {pid: owners for pid, owners in session.page_owners.items() if len(owners) > 1}
    assert len({owner for owners in shared.values() for owner in owners}) >= 3
    assert session.runner.cache.whole()
    for ident in requests:
        want[ident].check(got[ident], f"reuse {key} {dtype} {ident}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "D"])
def test_long_decoding_token_by_token(tmp_path_factory, key, dtype):
    folder, _, _, scale = reference(key, dtype, tmp_path_factory)
    tokens = random_tokens(RADILIX[key]["vocab"], 300, 9)
    want = Wanted(RADILIX[key], read_weights(folder), tokens, dtype, scale)
    steps = [{"step": i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": ["x"] if i == 299 else []}
             for i, t in enumerate(tokens)]
    got, session = replay(folder, dtype, steps, page_size=16)
    want.check(got["x"], f"long decode {key} {dtype}")
    assert session.runner.cache.whole()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B", "C", "E"])
def test_first_tokens_of_a_sequence(tmp_path_factory, key, dtype):
    folder, _, _, scale = reference(key, dtype, tmp_path_factory)
    tokens = random_tokens(RADILIX[key]["vocab"], 4, 77)
    want = Wanted(RADILIX[key], read_weights(folder), tokens, dtype, scale)
    one_by_one = [{"step": i, "entries": [{"id": "f", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(tokens)]
    got, _ = replay(folder, dtype, one_by_one, max_tokens=64)
    want.check(got["f"], "first tokens one by one")
    two_two = [{"step": 0, "entries": [{"id": "f", "tokens": tokens[:2], "want": [0, 1]}], "end": []},
               {"step": 1, "entries": [{"id": "f", "tokens": tokens[2:], "want": [0, 1]}], "end": ["f"]}]
    got, _ = replay(folder, dtype, two_two, max_tokens=64)
    want.check(got["f"], "first tokens two and two")


@pytest.mark.parametrize("key", ["B", "D"])
def test_a_request_in_company_equals_itself_alone(tmp_path_factory, key):
    """float32: the logits of a position change by rounding at most with the cutting and the company."""
    folder, requests, want, scale = reference(key, "float32", tmp_path_factory)
    whole, _ = replay(folder, "float32", whole_trace(requests))
    mixed, _ = replay(folder, "float32", mixed_trace(requests, seed=3), poison=True)
    cut, _ = replay(folder, "float32", portions_trace(requests, [2, 9, 2, 33, 64]))
    for ident in requests:
        bound = np.maximum(1e-5, 3.0 * distance(whole[ident], want[ident].logits, scale))
        assert (distance(mixed[ident], whole[ident], scale) <= bound).all()
        assert (distance(cut[ident], whole[ident], scale) <= bound).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B"])
def test_captured_decode_steps_equal_eager_ones(tmp_path_factory, key, dtype):
    """Decode steps are replayed from CUDA graphs; the same trace with graphs off gives the same bits."""
    from shrike_b200.replay import TraceSession

    folder, requests, _, _ = reference(key, dtype, tmp_path_factory)
    steps = tail_decode_trace({k: v for k, v in list(requests.items())[:3]}, 20)
    results = []
    for graphs in (True, False):
        session = TraceSession(folder, dtype, 512, page_size=16, max_live=4)
        session.runner.use_graphs = graphs
        results.append([session.step(record).copy() for record in steps])
        if graphs:
            assert session.runner.capture_safe and session.runner._graphs, "no decode step was captured"
    for a, b in zip(*results):
        assert np.array_equal(a, b)


def follows(key, folder, dtype, prompts, outs, new, scale):
    """Every continuation is the plain implementation's, up to the first choice that hangs on less than the tolerance."""
    weights = read_weights(folder)
    if dtype == "bfloat16":
        weights = {k: (v.to(torch.bfloat16).float() if v.dim() >= 2 else v) for k, v in weights.items()}
    tie = 12 * scale * (LIMIT_FLOAT32 if dtype == "float32" else 6e-2)
    for prompt, out in zip(prompts, outs):
        want, margins = pr.greedy_continue(RADILIX[key], weights, prompt, new)
        for position, (a, b, margin) in enumerate(zip(out, want, margins)):
            if a != b:
                assert margin < tie, f"token {position}: engine {a}, plain {b}, gap {margin}"
                break   # after a tie went the other way the continuations differ


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key,lengths,new", [("A", (5, 17, 33), 8), ("D", (3, 40, 75), 8), ("E", (9, 30, 2), 8)])
def test_greedy_generation_through_the_engine(tmp_path_factory, key, lengths, new, dtype):
    from shrike_b200 import SamplingParams
    from shrike_b200.engine.llm_engine import LLMEngine

    folder, _, _, scale = reference(key, dtype, tmp_path_factory)
    engine = LLMEngine(str(folder), block_size=8, num_blocks=40, max_tokens_per_step=32, dtype=dtype)
    prompts = [random_tokens(RADILIX[key]["vocab"], n, 30 + n) for n in lengths]
    outs = engine.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))
    assert engine.block_manager.whole()
    follows(key, folder, dtype, prompts, outs, new, scale)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_generation_survives_preemption_with_states(tmp_path_factory, dtype):
    """A pool too small for three requests at once: one is preempted (pages and state slots returned) and
    computed again later from zero states; every continuation still equals the plain implementation's."""
    from shrike_b200 import SamplingParams
    from shrike_b200.engine.llm_engine import LLMEngine

    folder, _, _, scale = reference("B", dtype, tmp_path_factory)
    engine = LLMEngine(str(folder), block_size=8, num_blocks=15, max_tokens_per_step=32, dtype=dtype)
    prompts = [random_tokens(RADILIX["B"]["vocab"], n, 60 + n) for n in (30, 31, 29)]
    outs = engine.generate(prompts, SamplingParams(max_new_tokens=24, ignore_eos=True))
    assert engine.block_manager.whole() and engine.scheduler.num_preemptions >= 1
    follows("B", folder, dtype, prompts, outs, 24, scale)


def _one_layer(layer, width=64, vocab=61, **more):
    return dict({"architecture": "Radilix", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "residual_mult": 1.2, "layers": [layer]},
                **more)


def _pair(left_scale, right_scale):
    return {"type": "parallel", "mlp": None, "mixer": {
        "left": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "rot": {"dims": 8, "base": 20.0}, "scale": 0.4}, "left_scale": left_scale,
        "right": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 16, "conv": 4}, "right_scale": right_scale}}


MIXERS = {"gla": {"type": "gla", "mlp": None, "mixer": {"heads": 3, "dim": 32, "vdim": 16, "tau": 5.0}},
          "left": _pair(1.0, 0.1), "right": _pair(0.1, 1.0)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer,place", [("left", p) for p in (0, 1, 15, 16, 255, 256, 700)]
                         + [(m, p) for m in ("right", "gla") for p in (0, 1, 7, 8, 16, 400, 950)])
def test_a_far_token_is_found_again(tmp_path, dtype, mixer, place):
    """A thousand tokens on many pages: the last query finds the one marked token wherever it lies (the first tokens,
    either side of a page's or a block's border, far back), in prompts, portions and decoding; the states keep it in
    a row that barely decays beside one that forgets at once."""
    raw = _one_layer(MIXERS[mixer])
    seed = 9 if mixer == "right" else 5   # a draw in which no head's output nearly vanishes, which its norm would blow up
    folder = make_radilix_folder(tmp_path, mixer, raw=raw, seed=seed, change=planted_pair(raw, mixer))
    weights = read_weights(folder)
    tokens = [5 + t % 50 for t in random_tokens(1000, 1000, 8)]
    tokens[place], tokens[-1] = MARK, ASKER
    without = list(tokens)
    without[place] = 9
    want = Wanted(raw, weights, tokens, dtype)
    other = Wanted(raw, weights, without, dtype)
    assert distance(want.logits[-1:], other.logits[-1:], want.scale)[0] > 0.2
    for steps in (whole_trace({"a": tokens}), tail_decode_trace({"a": tokens}, 60), portions_trace({"a": tokens}, [2, 130, 1, 1, 65, 500])):
        got, _ = replay(folder, dtype, steps, page_size=16, max_live=1)
        want.check(got["a"], f"{mixer}: marked token at {place}")


def test_trace_run_program_serves_the_design(tmp_path):
    folder = make_radilix_folder(tmp_path, "B")
    vocab = RADILIX["B"]["vocab"]
    requests = {"a": random_tokens(vocab, 41, 1), "b": random_tokens(vocab, 9, 2)}
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": requests["a"][:30], "want": [0, 29]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": requests["a"][30:31], "want": []},
                                {"id": "b", "tokens": requests["b"], "want": [8]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": requests["a"][31:], "want": [9]}], "end": ["a"]},
    ]
    out = tmp_path / "out"
    program = Path(__file__).resolve().parents[1] / "bin" / "trace_run"
    for dtype in ("bfloat16", "float32"):
        done = subprocess.run(
            [sys.executable, str(program), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
            input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
        assert done.returncode == 0, done.stderr[-2000:]
        assert [line for line in done.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
        want = {i: Wanted(RADILIX["B"], read_weights(folder), tokens, dtype) for i, tokens in requests.items()}
        want["a"].check(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, vocab), "step 0", [0, 29])
        want["b"].check(np.fromfile(out / "1.f32", dtype="<f4").reshape(1, vocab), "step 1", [8])
        want["a"].check(np.fromfile(out / "2.f32", dtype="<f4").reshape(1, vocab), "step 2", [40])


def test_command_line_program_serves_the_design(tmp_path):
    """The one-prompt program on a folder: the model class comes from config.json."""
    import os

    bin_dir = Path(__file__).resolve().parents[1] / "bin"
    folder = make_radilix_folder(tmp_path, "A")
    prompt = [7, 200, 41, 41, 2]
    want, margins = pr.greedy_continue(RADILIX["A"], read_weights(folder), prompt, 6)
    assert min(margins) > 1e-4
    done = subprocess.run([sys.executable, str(bin_dir / "shrike_b200_complete"), " ".join(map(str, prompt)), "--model", str(folder),
                           "--max-tokens", "6", "--dtype", "float32", "--num-blocks", "8", "--block-size", "8"],
                          capture_output=True, text=True, timeout=900, env=dict(os.environ, PYTHONUNBUFFERED="1"))
    assert done.returncode == 0, done.stderr[-3000:]
    assert [int(t) for t in done.stdout.split()] == want
