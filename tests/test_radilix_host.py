"""Radilix on the CPU: the configuration reader, the tensor names (also where layers use another layer's tensors), ranks that
the tensors give, the run order, the caches (pages and two states a parallel layer, one state a linear one, each run its
own), and the whole model stepped through the engine's replay session with the stand-in kernels against the plain
implementation: whole, in portions down to two tokens, mixed on a tight pool; with weights planted so that a far key or a
lost state decides the logits."""

import copy

import numpy as np
import pytest
import torch

import shrike_b200.models  # noqa: F401
from shrike_b200.config import ConfigError, parse_config
from shrike_b200.config.model_config import GatedHeadAttentionSpec, GatedLinearAttentionSpec, HeadDeltaSpec, RoutedExpertsSpec
from shrike_b200.parts.base import PendingSum, RowScaled
from shrike_b200.parts.norm import RMSNorm
from shrike_b200.replay import TraceSession
from shrike_b200.weights.expected import expected_tensors
from shrike_b200.weights.loader import WeightError
from tests.emulated_ops import EmulatedOps
from tests.helpers import collect, mixed_trace, portions_trace, random_tokens, read_weights, tail_decode_trace, whole_trace
from tests.plain import plain_radilix as pr
from tests.radilix_configs import ASKER, MARK, RADILIX, RADILIX_A, RADILIX_B, RADILIX_C, RADILIX_D, make_radilix_folder, planted_pair


def test_config_gives_each_layer_its_parts_and_every_run_its_cache():
    config = parse_config(RADILIX_A)
    assert config.architecture == "Radilix" and config.num_layers == 3   # four runs, of which two share a layer
    assert [(run.layer, run.cache, run.writes_cache) for run in config.order] == [(0, 0, True), (1, 1, True), (0, 2, True), (2, 3, True)]
    gla, pair, other = (layer.mixer for layer in config.layers)
    assert isinstance(gla, GatedLinearAttentionSpec)
    assert (gla.num_heads, gla.head_dim, gla.value_dim, gla.tau, gla.eps) == (3, 24, 16, 8.0, 1e-5)
    (name, left, left_scale), (other_name, right, right_scale) = pair.branches
    assert (name, other_name, left_scale, right_scale) == ("left", "right", 0.8, 1.3)
    assert isinstance(left, GatedHeadAttentionSpec) and isinstance(right, HeadDeltaSpec)
    assert (left.num_heads, left.num_kv_heads, left.head_dim, left.value_dim, left.scale, left.rotary) == (6, 2, 24, 16, 0.21, (8, 10000.0))
    assert left.qkv_bias and not left.out_bias and left.element_gate and not left.head_gate and not left.qk_norm
    assert left.window is None and left.chunk is None
    assert (right.num_heads, right.num_kv_heads, right.head_dim, right.value_dim, right.conv, right.unit_eps) == (4, 2, 16, 24, 3, 1e-6)
    assert other.branches[0][2] == -0.6
    moe, none, last = (layer.feed_forward for layer in config.layers)
    assert isinstance(moe, RoutedExpertsSpec) and none is None
    assert (moe.experts, moe.top, moe.intermediate, moe.identity, moe.gated, moe.activation) == (6, 2, 24, 2, False, "gelu")
    assert (moe.scoring, moe.renormalise, moe.correction, moe.shared_intermediate, moe.groups) == ("softmax", False, True, None, None)
    assert (last.top, last.identity) == (3, 3)
    assert all(layer.block == "parallel" and layer.block_options == (("scale", 0.9),) for layer in config.layers)
    assert all(layer.feed_forward_norm is None and layer.mixer_norm.offset == 1.0 for layer in config.layers)
    assert config.final_norm.offset == 1.0 and not config.tie_word_embeddings
    # a layer that uses the tensors of one that uses a third's
    assert [run.layer for run in parse_config(RADILIX_D).order] == [0, 1, 1, 1, 2]
    assert parse_config(RADILIX_C).layers[1].feed_forward.identity == 0
    assert parse_config(RADILIX_B).layers[0].feed_forward.top == 5


def test_a_mixer_without_its_optional_sizes_takes_them_from_the_others():
    raw = copy.deepcopy(RADILIX_C)
    for part in (raw["layers"][1]["mixer"]["left"], raw["layers"][1]["mixer"]["right"], raw["layers"][0]["mixer"]):
        part.pop("kv_heads", None)
        part.pop("vdim")
    config = parse_config(raw)
    left, right = (branch for _, branch, _ in config.layers[1].mixer.branches)
    assert (left.num_kv_heads, left.value_dim, right.num_kv_heads, right.value_dim) == (3, 6, 3, 10)
    assert config.layers[0].mixer.value_dim == 10


def test_tensor_names_and_shapes():
    names = expected_tensors(parse_config(RADILIX_A))
    shapes = {"embed": (211, 96), "l0.norm1": (96,), "l0.mix.q": (72, 96), "l0.mix.k": (72, 96), "l0.mix.v": (48, 96), "l0.mix.g": (48, 96),
              "l0.mix.o": (96, 48), "l0.mix.norm": (16,), "l0.mix.a2.b": (72,), "l0.mlp.router": (8, 96), "l0.mlp.correction": (8,),
              "l0.mlp.e5.up": (24, 96), "l0.mlp.e0.down": (96, 24), "l1.mix.left.q": (144, 96), "l1.mix.left.q.b": (144,),
              "l1.mix.left.k": (48, 96), "l1.mix.left.k.b": (48,), "l1.mix.left.v": (32, 96), "l1.mix.left.v.b": (32,),
              "l1.mix.left.g": (96, 96), "l1.mix.left.o": (96, 96), "l1.mix.right.q": (32, 96), "l1.mix.right.q.conv": (32, 3),
              "l1.mix.right.v": (96, 96), "l1.mix.right.v.conv": (96, 3), "l1.mix.right.b": (4, 96), "l1.mix.right.a": (4, 96),
              "l1.mix.right.A_log": (4,), "l1.mix.right.dt_bias": (4,), "l1.mix.right.norm": (24,), "l1.mix.right.g": (96, 96),
              "l1.mix.right.o": (96, 96), "l3.mix.left.k": (40, 96), "l3.mlp.router": (8, 96), "final.norm": (96,), "head": (211, 96)}
    for name, shape in shapes.items():
        assert names[name].shape == shape, name
    assert names["l0.mix.a1"].free == (0,) and names["l0.mix.a2"].free == (1,)
    # a layer that uses another's tensors has none; identity experts have none; nor has a layer without a feed-forward
    assert not any(name.startswith("l2.") for name in names)
    for absent in ("l0.mlp.e6.up", "l1.mlp.router", "l0.norm2", "l0.mlp.e0.gate", "l1.mix.left.o.b"):
        assert absent not in names


def test_ranks_come_from_the_tensors_and_must_fit(tmp_path):
    def unequal(tensors):
        tensors["l0.mix.a1"] = torch.zeros(9, 96)

    with pytest.raises(ValueError, match="decay's low-rank product"):
        TraceSession(make_radilix_folder(tmp_path, "A", change=unequal), "float32", 64, device="cpu", ops=EmulatedOps())

    def extra(tensors):
        tensors["l2.norm1"] = torch.zeros(96)

    with pytest.raises(WeightError, match="l2.norm1"):
        TraceSession(make_radilix_folder(tmp_path, "A", change=extra), "float32", 64, device="cpu", ops=EmulatedOps())


@pytest.mark.parametrize("change,text", [
    (lambda raw: raw["layers"][1].update(type="attention"), "known: gla, parallel"),
    (lambda raw: raw["layers"][0]["mixer"].pop("tau"), "tau"),
    (lambda raw: raw["layers"][0]["mixer"].update(tau=0.0), "tau must be positive"),
    (lambda raw: raw["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda raw: raw["layers"][1]["mixer"].pop("right"), "right"),
    (lambda raw: raw["layers"][1]["mixer"]["left"].update(kv_heads=4), "multiple"),
    (lambda raw: raw["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda raw: raw["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda raw: raw["layers"][1]["mixer"]["right"].update(kv_heads=3), "multiple"),
    (lambda raw: raw["layers"][1]["mixer"]["right"].update(conv=40), "1 to 32 taps"),
    (lambda raw: raw["layers"][3]["mlp"]["router"].update(top=9), "top=9 must lie in 1..8"),
    (lambda raw: raw["layers"][3]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda raw: raw["layers"][3]["mlp"].update(kind="dense"), "known: moe"),
    (lambda raw: raw["layers"][2].update(weights_of=7), "weights_of"),
    (lambda raw: raw["layers"][2].update(weights_of=2), "weights_of"),
    (lambda raw: raw["layers"][2].update(weights_of=1), "not described alike"),
    (lambda raw: raw.pop("residual_mult"), "residual_mult"),
    (lambda raw: raw.pop("norm"), "norm"),
])
def test_config_errors_name_the_key(change, text):
    raw = copy.deepcopy(RADILIX_A)
    change(raw)
    with pytest.raises(ConfigError, match=text):
        parse_config(raw)


def run(folder, steps, **options):
    session = TraceSession(folder, "float32", device="cpu", ops=EmulatedOps(), **options)
    outputs = {}
    for record in steps:
        result = session.step(record)
        if result is not None:
            outputs[record["step"]] = result.copy()
    return collect(steps, outputs), session


LENGTHS = [5, 47, 1, 83, 2, 30]


@pytest.mark.parametrize("key", ["A", "B", "C", "D", "E"])
def test_engine_with_stand_in_kernels_matches_plain(tmp_path, key):
    folder = make_radilix_folder(tmp_path, key)
    weights = read_weights(folder)
    requests = {f"r{i}": random_tokens(RADILIX[key]["vocab"], n, 200 + i) for i, n in enumerate(LENGTHS)}
    want = {ident: pr.forward(RADILIX[key], weights, tokens).numpy() for ident, tokens in requests.items()}
    spread = float(np.sqrt(np.mean([np.var(w, axis=-1).mean() for w in want.values()])))
    ways = (whole_trace(requests), tail_decode_trace(requests, 25), portions_trace(requests, [7, 2, 5, 3, 16, 17, 2]),
            mixed_trace(requests, seed=4))
    for steps in ways:
        got, session = run(folder, steps, page_size=8, num_pages=40, max_live=4)
        assert session.runner.cache.whole()
        for ident in requests:
            assert np.abs(got[ident] - want[ident]).max() < 1e-3 * spread, ident   # float32 stand-ins against float64


def test_every_run_has_a_cache_and_states_of_its_own(tmp_path):
    folder = make_radilix_folder(tmp_path, "A")
    session = TraceSession(folder, "float32", device="cpu", ops=EmulatedOps(), page_size=4, num_pages=64, max_live=2)
    # keys of 24 beside values of 16 in heads of 32; keys of 40 beside values of 48
    assert [(g.head_dim, g.window, g.num_kv_heads, g.cache_ids) for g in session.runner.groups] == [(32, None, 2, (1,)), (48, None, 1, (3,))]
    state = session.runner.storage.state
    assert set(state) == {0, 1, (1, "conv"), 2, 3, (3, "conv")}
    assert tuple(state[0].shape) == tuple(state[2].shape) == (2, 3, 24 * 16) and tuple(state[1].shape) == (2, 4, 16 * 24)
    assert tuple(state[(1, "conv")].shape) == (2, 2, 2 * 32 + 96) and tuple(state[(3, "conv")].shape) == (2, 3, 2 * 60 + 24)
    tokens = random_tokens(211, 30, 5)
    session.step({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": []}], "end": []})
    slot = session.live["a"][0].slot
    for cache, held in state.items():
        assert float(held[slot].abs().sum()) > 0 and float(held[1 - slot].abs().sum()) == 0, cache
    assert not torch.equal(state[0][slot], state[2][slot])   # the same tensors, another state
    session.step({"step": 1, "entries": [], "end": ["a"]})
    assert session.runner.cache.whole()
    # the slot's next owner starts from zero states although the kernels left the old ones behind
    session.step({"step": 2, "entries": [{"id": "b", "tokens": tokens[:3], "want": []}], "end": []})
    session.step({"step": 3, "entries": [{"id": "c", "tokens": tokens[:3], "want": []}], "end": []})
    b, c = session.live["b"][0].slot, session.live["c"][0].slot
    assert b != c and all(torch.equal(held[b], held[c]) for held in state.values())


def test_shared_layers_hold_their_tensors_once(tmp_path):
    session = TraceSession(make_radilix_folder(tmp_path, "B"), "float32", 64, device="cpu", ops=EmulatedOps())
    model = session.runner.model
    assert len(model.blocks) == 3 and [run.layer for run in model.config.order] == [0, 0, 1, 2]
    assert [g.cache_ids for g in session.runner.groups] == [(0, 1), (3,)]   # pages of its own a run, alike runs in one pool


def test_a_pending_sum_larger_than_one_launch_is_flushed():
    class Runtime:
        act_dtype = torch.float32

        def buffer(self, name, shape, dtype):
            return torch.zeros(shape, dtype=dtype)

    from shrike_b200.config.model_config import RMSNormSpec

    g = torch.Generator().manual_seed(0)
    weight = torch.randn(12, generator=g)
    norm = RMSNorm(RMSNormSpec(width=12, eps=1e-5, offset=1.0), {"weight": weight}, EmulatedOps(), Runtime())
    resid, x, factors = torch.randn(5, 12, generator=g), torch.randn(5, 12, generator=g), torch.randn(5, 3, generator=g)[:, 1]
    terms = [(torch.randn(5, 12, generator=g), 0.5 + i) for i in range(6)] + [(torch.randn(3, 5, 12, generator=g), -1.0)]
    want = resid + sum(s * (t.sum(0) if t.dim() == 3 else t) for t, s in terms) + 2.0 * factors[:, None] * x
    pending = PendingSum(terms + [(RowScaled(x, factors), 2.0)])
    rows = torch.tensor([3, 0], dtype=torch.int32)
    kept = resid.clone()
    some = norm.gather_norm(kept, pending, rows)
    torch.testing.assert_close(some, pr.layer_norm(want, weight, 1e-5)[[3, 0]])
    out = norm.add_norm(resid, pending)
    torch.testing.assert_close(resid, want)
    torch.testing.assert_close(out, pr.layer_norm(want, weight, 1e-5))


def _one_layer(layer, width=32, vocab=61, **more):
    return dict({"architecture": "Radilix", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "residual_mult": 1.1, "layers": [layer]},
                **more)


def _pair(left_scale, right_scale):
    return {"type": "parallel", "mlp": None, "mixer": {
        "left": {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 6, "rot": {"dims": 4, "base": 20.0}, "scale": 0.5}, "left_scale": left_scale,
        "right": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "conv": 3}, "right_scale": right_scale}}


MIXERS = {"gla": {"type": "gla", "mlp": None, "mixer": {"heads": 2, "dim": 8, "vdim": 6, "tau": 4.0}},
          "left": _pair(1.0, 0.1), "right": _pair(0.1, 1.0)}


@pytest.mark.parametrize("mixer", list(MIXERS))
def test_a_far_token_decides(tmp_path, mixer):
    """The marked token eighty places back decides the last logits, however the prompt is cut and whoever else is there."""
    raw = _one_layer(MIXERS[mixer])
    folder = make_radilix_folder(tmp_path, mixer, raw=raw, seed=3, change=planted_pair(raw, mixer))
    weights = read_weights(folder)
    tokens = [5 + t % 50 for t in random_tokens(1000, 90, 4)]
    tokens[8], tokens[-1] = MARK, ASKER
    other = list(tokens)
    other[8] = 9
    want, want_other = pr.forward(raw, weights, tokens).numpy(), pr.forward(raw, weights, other).numpy()
    spread = float(np.sqrt(np.var(want, axis=-1).mean()))
    assert np.abs(want[-1] - want_other[-1]).max() > 0.3 * spread
    both = {"a": tokens, "b": other}
    for steps in (whole_trace(both), portions_trace(both, [2, 33, 1, 40, 3]), mixed_trace(both, seed=1, max_live=2)):
        got, session = run(folder, steps, page_size=4, num_pages=48, max_live=2)
        assert np.abs(got["a"] - want).max() < 2e-3 * spread and np.abs(got["b"] - want_other).max() < 2e-3 * spread
        assert session.runner.cache.whole()
