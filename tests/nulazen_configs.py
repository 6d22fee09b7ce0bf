"""Tiny Nulazen configurations for tests, and model folders with weights that make faults show.

The configurations differ from one another in every size and option: width, vocabulary, the order of the two mixers, head
counts (one value head a key head, several, all on one), keys wider and narrower than values, sizes that are no multiple
of four or sixteen, convolutions of one to six taps, low ranks of their own for decays and gates, rotations of two
dimensions and more, dense and mixed feed-forwards and none, experts in one to many groups of which one, some or all are
kept, one, some or all experts chosen, a shared expert with a clamp of its own or none, a side input or none, and the
repeated layers at the start, in the middle, at the end, once, or not at all.
"""

from __future__ import annotations

from pathlib import Path

import torch


def _latent(heads, dim, rot_dim, vdim, rank, scale, base):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                                                  "scale": scale, "rot": {"dims": rot_dim, "base": base}}}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def _dense(layer, ff):
    return dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def _moe(layer, experts, top, ff, limit, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router,
                            "shared": None if shared is None else {"ff": shared[0], "limit": shared[1]}})


# both mixers, three value heads a key head, the repeated layers at the end, three passes; a layer without a feed-forward
NULAZEN_A = {
    "architecture": "Nulazen", "width": 96, "vocab": 211, "norm": {"eps": 1e-5}, "token_side": {"dim": 20},
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        _dense(_delta(6, 2, 24, 16, 3), 80),
        _moe(_latent(3, 24, 8, 16, 40, 0.21, 10000.0), 6, 2, 24, 1.5, (3, 2), (40, 0.75)),
        _dense(_delta(2, 2, 16, 40, 4), None),
    ],
}

# heads of 64 (page rows of 64, the sizes the tensor-core kernels take); no repeated layers; no side input; one group kept
NULAZEN_B = {
    "architecture": "Nulazen", "width": 128, "vocab": 300, "norm": {"eps": 1e-6},
    "layers": [
        _moe(_delta(2, 1, 64, 64, 4), 8, 3, 32, 2.5, (2, 1), (64, 2.5)),
        _dense(_latent(2, 32, 16, 64, 48, 0.15, 100.0), 192),
        _moe(_delta(4, 4, 32, 16, 2), 5, 5, 16, 0.5),
        _dense(_latent(4, 16, 32, 8, 96, 0.2, 1e6), 96),
    ],
}

# odd sizes, one tap and six, one pass "repeated" once at the very start, as many groups as experts, one expert chosen
NULAZEN_C = {
    "architecture": "Nulazen", "width": 72, "vocab": 97, "norm": {"eps": 1e-4}, "token_side": {"dim": 7},
    "loop": {"start": 0, "stop": 1, "times": 1},
    "layers": [
        _moe(_delta(3, 1, 10, 7, 1), 4, 1, 12, 3.0, (4, 3), (9, 1.0)),
        _dense(_latent(1, 6, 2, 10, 12, 0.4, 10.0), 40),
        _dense(_delta(1, 1, 5, 30, 6), 24),
        _moe(_latent(5, 16, 4, 3, 20, 0.3, 50.0), 12, 7, 8, 1.0, (6, 4)),
    ],
}

# heads of 128, the repeated layers in the middle, two passes, holding both mixers; four shared value heads a key head
NULAZEN_D = {
    "architecture": "Nulazen", "width": 64, "vocab": 151, "norm": {"eps": 1e-6}, "token_side": {"dim": 32},
    "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        _dense(_delta(4, 1, 128, 32, 4), 96),
        _moe(_delta(2, 2, 40, 128, 4), 8, 4, 16, 2.0, (4, 4), (24, 4.0)),
        _dense(_latent(2, 64, 16, 32, 112, 0.1, 30000.0), 48),
        _moe(_latent(3, 8, 8, 24, 56, 0.25, 300.0), 6, 2, 20, 1.0, (2, 2)),
    ],
}

NULAZEN = {"A": NULAZEN_A, "B": NULAZEN_B, "C": NULAZEN_C, "D": NULAZEN_D}
NULAZEN_SEEDS = {"A": 41, "B": 42, "C": 43, "D": 44}
RANKS = {"A": (12, 20), "B": (64, 16), "C": (3, 5), "D": (17, 8)}   # of the decays' and the gates' low-rank products


def with_ranks(tensors: dict, ranks, seed: int = 0) -> dict:
    """The low-rank products with ranks of their own (no configuration key names them: the tensors say)."""
    generator = torch.Generator().manual_seed(seed + 5)
    out = dict(tensors)
    for name, tensor in tensors.items():
        for rank, down, up in ((ranks[0], ".mix.a1", ".mix.a2"), (ranks[1], ".mix.g1", ".mix.g2")):
            if name.endswith(down):
                out[name] = 0.02 * torch.randn(rank, tensor.shape[1], generator=generator)
            elif name.endswith(up):
                out[name] = 0.02 * torch.randn(tensor.shape[0], rank, generator=generator)
    return out


def sharpened(tensors: dict) -> dict:
    """Random weights leave attention nearly uniform, every gate at a half, every decay alike and the routers undecided,
    which hides a key that is wrongly seen or a state that was lost.  This scales what sets the size of the scores, gates,
    decays, choices and pass vectors."""
    out = {}
    for name, tensor in tensors.items():
        t = tensor.clone()
        if name.endswith((".mix.q", ".mix.k", ".mix.v", ".mix.dkv", ".mix.uk", ".mix.uv")):
            t *= 5.0
        elif name.endswith((".mix.a1", ".mix.a2", ".mix.g1", ".mix.g2")):
            t *= 15.0
        elif name.endswith((".mix.b", ".mlp.router", ".shared.sg", ".side.gate")):
            t *= 15.0
        elif name.endswith((".gate", ".up")):
            t *= 10.0
        elif name.endswith(".correction"):
            t *= 20.0
        elif name == "loop.step":
            t *= 20.0
        elif name.endswith((".norm1b", ".norm2b")):
            t *= 0.7
        elif name.endswith(".side.norm"):
            t *= 0.5
        elif name == "embed":
            t *= 40.0
        out[name] = t
    return out


def make_nulazen_folder(tmp_path, key: str, dtype: str = "float32", raw: dict | None = None, seed: int | None = None,
                        change=None, ranks=None) -> Path:
    """A model folder (config.json, model.safetensors) of a tiny configuration with sharpened weights.  `change`
    (name -> tensor dictionary, edited in place) lets a test plant a weight of its own."""
    import json

    from shrike_b200 import models  # noqa: F401
    from shrike_b200.config.registry import parse_config
    from shrike_b200.weights.random_init import random_tensors
    from shrike_b200.weights.safetensors_io import write_safetensors

    raw = dict(raw if raw is not None else NULAZEN[key])
    seed = NULAZEN_SEEDS.get(key, 0) if seed is None else seed
    out = Path(tmp_path) / f"nulazen_{key}_{dtype}"
    out.mkdir(parents=True, exist_ok=True)
    tensors = random_tensors(parse_config(raw), seed, "cpu", torch.float32)
    tensors = sharpened(with_ranks(tensors, ranks or RANKS.get(key, (6, 10)), seed))
    if change is not None:
        change(tensors)
    tensors = {name: t.to(getattr(torch, dtype)) for name, t in tensors.items()}
    (out / "config.json").write_text(json.dumps(raw, indent=2) + "\n")
    write_safetensors(out / "model.safetensors", tensors, {"format": "pt", "seed": str(seed)})
    return out


MARK, ASKER = 3, 4   # token ids of `planted_pair`


def planted_pair(raw: dict, strength: float = 2.0, gain: float = 12.0):
    """A `change` for `make_nulazen_folder` on a model whose layer 0 holds the mixer under test: whether token MARK is
    still there when token ASKER comes decides ASKER's logits, however many tokens lie between.

    Residual axis 0 is nonzero in MARK's embedding only and axis 1 in ASKER's only.  Latent attention: one unrotated key
    dimension reads axis 0 alone and the same query dimension axis 1 alone, so their score stands far above the others.
    Delta rule: key dimension 0 reads axis 0 and query dimension 0 axis 1, nothing else writes or reads that row of the
    state, and the row's decay is nearly one (the heads' last key dimensions have a decay near zero)."""
    layer = raw["layers"][0]
    spec = layer["mixer"]

    def change(tensors):
        embed = tensors["embed"]
        embed[:, 0:2] = 0.0
        embed[MARK, 0] = strength * float(embed[:, 2:].std()) * embed.shape[1] ** 0.5
        embed[ASKER, 1] = embed[MARK, 0]
        tensors["l0.norm1"][0:2] = 1.0
        tensors["l0.norm1b"] *= 3.0
        if layer["type"] == "latent_attention":
            heads, dim = spec["heads"], spec["dim"]
            per_head = dim + spec["rot_dim"]
            tensors["l0.mix.dkv"][0] = 0.0
            tensors["l0.mix.dkv"][0, 0] = gain       # latent component 0 is MARK's alone
            tensors["l0.mix.dkv.norm"][0] = 1.0
            for a in range(heads):
                tensors["l0.mix.uk"][a * dim] = 0.0
                tensors["l0.mix.uk"][a * dim, 0] = 4.0
                tensors["l0.mix.q"][a * per_head] = 0.0
                tensors["l0.mix.q"][a * per_head, 1] = gain
        else:
            dim = spec["dim"]
            for a in range(spec["kv_heads"]):
                for name, axis in (("q", 1), ("k", 0)):
                    tensors[f"l0.mix.{name}"][a * dim] = 0.0
                    tensors[f"l0.mix.{name}"][a * dim, axis] = gain
                    tensors[f"l0.mix.{name}.conv"][a * dim] = 0.0
                    tensors[f"l0.mix.{name}.conv"][a * dim, -1] = 1.0
            tensors["l0.mix.A_log"][:] = 0.0
            for a in range(spec["heads"]):
                tensors["l0.mix.a2"][a * dim] = 0.0
                tensors["l0.mix.dt_bias"][a * dim] = -9.0          # a decay of about 0.9999
                tensors["l0.mix.dt_bias"][a * dim + dim - 1] = 4.0   # and one of about 0.02

    return change
