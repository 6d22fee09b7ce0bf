"""Nulazen on the CPU: the configuration reader, the tensor names, ranks that the tensors give, the run order with its
passes, the caches (a latent's single plane, two state slots a delta-rule run), and the whole model stepped through the
engine's replay session with the stand-in kernels against the plain implementation: whole, in portions down to two tokens,
mixed on a tight pool; with weights planted so that a far key or a lost state decides the logits."""

import copy

import numpy as np
import pytest
import torch

import shrike_b200.models  # noqa: F401
from shrike_b200.config import ConfigError, parse_config
from shrike_b200.config.model_config import ChannelDeltaSpec, MLPSpec, RotaryLatentAttentionSpec, RoutedExpertsSpec
from shrike_b200.parts.base import ParamSpec
from shrike_b200.replay import TraceSession
from shrike_b200.weights.expected import expected_tensors
from shrike_b200.weights.loader import WeightError
from tests.emulated_ops import EmulatedOps
from tests.helpers import collect, mixed_trace, portions_trace, random_tokens, read_weights, tail_decode_trace, whole_trace
from tests.nulazen_configs import ASKER, MARK, NULAZEN, NULAZEN_A, NULAZEN_B, NULAZEN_C, NULAZEN_D, make_nulazen_folder, planted_pair
from tests.plain import plain_nulazen as pn


def test_config_gives_each_layer_its_parts_and_every_run_its_cache():
    config = parse_config(NULAZEN_A)
    assert config.architecture == "Nulazen" and config.num_layers == 3
    assert [(run.layer, run.cache, run.enter) for run in config.order] == [
        (0, 0, None), (1, 1, 0), (2, 2, None), (1, 3, 1), (2, 4, None), (1, 5, 2), (2, 6, None)]
    assert config.pass_entry.passes == 3 and not config.pass_entry.mix and not config.pass_entry.add_embedding
    assert (config.side_table.vocab, config.side_table.parts, config.side_table.dim) == (211, 3, 20)
    delta, latent, other = (layer.mixer for layer in config.layers)
    assert isinstance(delta, ChannelDeltaSpec) and isinstance(latent, RotaryLatentAttentionSpec)
    assert (delta.num_heads, delta.num_kv_heads, delta.head_dim, delta.value_dim, delta.conv, delta.unit_eps) == (6, 2, 24, 16, 3, 1e-6)
    assert (latent.num_heads, latent.head_dim, latent.rotary_dim, latent.value_dim, latent.latent_rank, latent.scale) == (3, 24, 8, 16, 40, 0.21)
    assert latent.gate is None and latent.window is None and (latent.rotation.base, latent.rotation.pairing) == (10000.0, "halves")
    assert (other.num_kv_heads, other.value_dim) == (2, 40)
    dense, moe, none = (layer.feed_forward for layer in config.layers)
    assert isinstance(dense, MLPSpec) and (dense.intermediate, dense.activation) == (80, "relu2") and none is None
    assert isinstance(moe, RoutedExpertsSpec) and (moe.experts, moe.top, moe.groups, moe.limit) == (6, 2, (3, 2), 1.5)
    assert (moe.shared_intermediate, moe.shared_limit, moe.correction, moe.renormalise) == (40, 0.75, True, False)
    roles = [[role for role, _, _ in layer.roles()] for layer in config.layers]
    assert roles[0] == ["mixer", "mixer_norm", "feed_forward", "feed_forward_norm", "mixer_out_norm", "feed_forward_out_norm", "side", "side_norm"]
    assert roles[2] == ["mixer", "mixer_norm", "mixer_out_norm", "side", "side_norm"]
    assert [layer.extra[-2][2].index for layer in config.layers] == [0, 1, 2]
    plain = parse_config(NULAZEN_B)
    assert plain.pass_entry is None and plain.side_table is None and plain.layers[2].feed_forward.groups is None
    assert plain.layers[2].feed_forward.shared_intermediate is None
    assert [(run.layer, run.enter) for run in parse_config(NULAZEN_C).order] == [(0, 0), (1, None), (2, None), (3, None)]
    assert [run.layer for run in parse_config(NULAZEN_D).order] == [0, 1, 2, 1, 2, 3]


def test_a_mixer_without_its_optional_sizes_takes_them_from_the_others():
    raw = copy.deepcopy(NULAZEN_B)
    raw["layers"][0]["mixer"].pop("kv_heads")
    raw["layers"][0]["mixer"].pop("vdim")
    spec = parse_config(raw).layers[0].mixer
    assert (spec.num_kv_heads, spec.value_dim) == (2, 64)


def test_tensor_names_and_shapes():
    names = expected_tensors(parse_config(NULAZEN_A))
    shapes = {"embed": (211, 96), "loop.step": (3, 96), "side.embed": (211, 60), "l0.norm1b": (96,), "l0.norm2b": (96,),
              "l0.mix.q": (48, 96), "l0.mix.k": (48, 96), "l0.mix.v": (96, 96), "l0.mix.q.conv": (48, 3), "l0.mix.v.conv": (96, 3),
              "l0.mix.b": (6, 96), "l0.mix.A_log": (6,), "l0.mix.dt_bias": (144,), "l0.mix.norm": (16,), "l0.mix.o": (96, 96),
              "l0.mlp.up": (80, 96), "l0.mlp.down": (96, 80), "l0.side.gate": (20, 96), "l0.side.proj": (96, 20), "l0.side.norm": (96,),
              "l1.mix.q": (96, 96), "l1.mix.dkv": (48, 96), "l1.mix.dkv.norm": (40,), "l1.mix.uk": (72, 40), "l1.mix.uv": (48, 40),
              "l1.mlp.router": (6, 96), "l1.mlp.correction": (6,), "l1.mlp.e5.gate": (24, 96), "l1.mlp.e0.down": (96, 24),
              "l1.mlp.shared.up": (40, 96), "l1.mlp.shared.sg": (1, 96), "final.norm": (96,), "head": (211, 96)}
    for name, shape in shapes.items():
        assert names[name].shape == shape, name
    assert names["l0.mix.a1"].free == (0,) and names["l0.mix.a2"].free == (1,)
    assert "l2.norm2" not in names and "l2.norm2b" not in names and "l0.mlp.gate" not in names and "l1.mix.g" not in names
    bare = expected_tensors(parse_config(NULAZEN_B))
    assert "loop.step" not in bare and "side.embed" not in bare and "l0.side.gate" not in bare and "l2.mlp.shared.gate" not in bare


def test_ranks_come_from_the_tensors_and_must_fit(tmp_path):
    spec = ParamSpec((8, 16), "matrix", free=(0,))
    assert spec.fits((3, 16)) and not spec.fits((3, 15)) and not spec.fits((0, 16)) and not spec.fits((3, 16, 1))

    def unequal(tensors):
        tensors["l0.mix.a1"] = torch.zeros(9, 96)

    with pytest.raises(ValueError, match="decay's low-rank product"):
        TraceSession(make_nulazen_folder(tmp_path, "A", change=unequal), "float32", 64, device="cpu", ops=EmulatedOps())

    def narrow(tensors):
        tensors["l0.mix.g2"] = torch.zeros(95, 20)

    with pytest.raises(WeightError, match="l0.mix.g2"):
        TraceSession(make_nulazen_folder(tmp_path, "A", change=narrow), "float32", 64, device="cpu", ops=EmulatedOps())


@pytest.mark.parametrize("change,text", [
    (lambda raw: raw["layers"][0].update(type="attention"), "known: channel_delta, latent_attention"),
    (lambda raw: raw["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda raw: raw["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda raw: raw["layers"][0]["mixer"].update(conv=40), "1 to 32 taps"),
    (lambda raw: raw["layers"][1]["mixer"]["rot"].update(dims=6), "rotated part has 8"),
    (lambda raw: raw["layers"][1]["mixer"].pop("rot"), "lacks `rot`"),
    (lambda raw: raw["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda raw: raw["layers"][1]["mlp"]["router"]["groups"].update(count=4), "do not form 4 equal groups"),
    (lambda raw: raw["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "groups.keep=4"),
    (lambda raw: raw["layers"][1]["mlp"]["router"].update(top=5), "top=5 of 2 groups"),
    (lambda raw: raw["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda raw: raw["layers"][1]["mlp"].update(kind="sparse"), "known: dense, moe"),
    (lambda raw: raw["token_side"].pop("dim"), "dim"),
    (lambda raw: raw["loop"].update(stop=4), "loop runs layers"),
    (lambda raw: raw.pop("norm"), "norm"),
])
def test_config_errors_name_the_key(change, text):
    raw = copy.deepcopy(NULAZEN_A)
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


@pytest.mark.parametrize("key", ["A", "B", "C", "D"])
def test_engine_with_stand_in_kernels_matches_plain(tmp_path, key):
    folder = make_nulazen_folder(tmp_path, key)
    weights = read_weights(folder)
    requests = {f"r{i}": random_tokens(NULAZEN[key]["vocab"], n, 200 + i) for i, n in enumerate(LENGTHS)}
    want = {ident: pn.forward(NULAZEN[key], weights, tokens).numpy() for ident, tokens in requests.items()}
    spread = float(np.sqrt(np.mean([np.var(w, axis=-1).mean() for w in want.values()])))
    ways = (whole_trace(requests), tail_decode_trace(requests, 25), portions_trace(requests, [7, 2, 5, 3, 16, 17, 2]),
            mixed_trace(requests, seed=4))
    for steps in ways:
        got, session = run(folder, steps, page_size=8, num_pages=40, max_live=4)
        assert session.runner.cache.whole()
        for ident in requests:
            assert np.abs(got[ident] - want[ident]).max() < 1e-3 * spread, ident   # float32 stand-ins against float64


def test_a_request_holds_two_state_slots_a_run_and_a_latents_pages(tmp_path):
    folder = make_nulazen_folder(tmp_path, "A")
    session = TraceSession(folder, "float32", device="cpu", ops=EmulatedOps(), page_size=4, num_pages=64, max_live=2)
    # the latent's page row is [40 | 8] in one plane that is key and value at once; its three runs share a group
    assert [(g.head_dim, g.window, g.num_kv_heads, g.cache_ids, g.planes) for g in session.runner.groups] == [(48, None, 1, (1, 3, 5), 1)]
    state = session.runner.storage.state
    assert set(state) == {0, (0, "conv"), 2, (2, "conv"), 4, (4, "conv"), 6, (6, "conv")}
    assert tuple(state[0].shape) == (2, 6, 24 * 16) and tuple(state[(0, "conv")].shape) == (2, 2, 2 * 48 + 96)
    assert tuple(state[4].shape) == (2, 2, 16 * 40) and tuple(state[(4, "conv")].shape) == (2, 3, 64 + 80)
    tokens = random_tokens(211, 30, 5)
    session.step({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": []}], "end": []})
    slot = session.live["a"][0].slot
    for cache, held in state.items():
        assert float(held[slot].abs().sum()) > 0 and float(held[1 - slot].abs().sum()) == 0, cache
    assert not torch.equal(state[2][slot], state[4][slot])   # each pass keeps a state of its own
    session.step({"step": 1, "entries": [], "end": ["a"]})
    assert session.runner.cache.whole()
    # the slot's next owner starts from zero states although the kernels left the old ones behind
    session.step({"step": 2, "entries": [{"id": "b", "tokens": tokens[:3], "want": []}], "end": []})
    session.step({"step": 3, "entries": [{"id": "c", "tokens": tokens[:3], "want": []}], "end": []})
    b, c = session.live["b"][0].slot, session.live["c"][0].slot
    assert b != c and all(torch.equal(held[b], held[c]) for held in state.values())


def test_a_convolution_of_one_tap_has_no_state(tmp_path):
    session = TraceSession(make_nulazen_folder(tmp_path, "C"), "float32", 64, device="cpu", ops=EmulatedOps())
    assert set(session.runner.storage.state) == {0, 2, (2, "conv")}


def _one_layer(layer, width=32, vocab=61, **more):
    return dict({"architecture": "Nulazen", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "layers": [layer]}, **more)


LATENT = {"type": "latent_attention", "mlp": None, "mixer": {"heads": 2, "dim": 8, "rot_dim": 4, "vdim": 8, "kv_rank": 12, "scale": 0.5,
                                                             "rot": {"dims": 4, "base": 20.0}}}
DELTA = {"type": "channel_delta", "mlp": None, "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "conv": 3}}


@pytest.mark.parametrize("layer", [LATENT, DELTA], ids=["latent", "delta"])
def test_a_far_token_decides(tmp_path, layer):
    """The marked token eighty places back decides the last logits, however the prompt is cut and whoever else is there."""
    raw = _one_layer(layer)
    folder = make_nulazen_folder(tmp_path, layer["type"], raw=raw, seed=3, change=planted_pair(raw))
    weights = read_weights(folder)
    tokens = [5 + t % 50 for t in random_tokens(1000, 90, 4)]
    tokens[8], tokens[-1] = MARK, ASKER
    other = list(tokens)
    other[8] = 9
    want, want_other = pn.forward(raw, weights, tokens).numpy(), pn.forward(raw, weights, other).numpy()
    spread = float(np.sqrt(np.var(want, axis=-1).mean()))
    assert np.abs(want[-1] - want_other[-1]).max() > 0.3 * spread
    both = {"a": tokens, "b": other}
    for steps in (whole_trace(both), portions_trace(both, [2, 33, 1, 40, 3]), mixed_trace(both, seed=1, max_live=2)):
        got, session = run(folder, steps, page_size=4, num_pages=48, max_live=2)
        assert np.abs(got["a"] - want).max() < 2e-3 * spread and np.abs(got["b"] - want_other).max() < 2e-3 * spread
        assert session.runner.cache.whole()
