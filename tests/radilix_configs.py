"""Tiny Radilix configurations for tests, and model folders with weights that make faults show.

The configurations differ from one another in every size and option: width, vocabulary, the order of the two layer types,
layers that use another layer's tensors (the one before, one far back, through a third, or none), head counts (one value
head a key head, several, all on one), keys wider and narrower than values, sizes that are no multiple of four or sixteen,
rotations of two dimensions, part of a head or all of it, convolutions of one to six taps, ranks of their own for the
decays, exponents of one and more, branch scales that differ in size and sign, one, some or all experts chosen, identity
experts or none, layers without a feed-forward, and a model without any attention.
"""

from __future__ import annotations

from pathlib import Path

import torch


def _gla(heads, dim, vdim, tau):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def _left(heads, kv_heads, dim, vdim, rot, base, scale):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base}, "scale": scale}


def _right(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def _parallel(left, left_scale, right, right_scale):
    return {"type": "parallel", "mixer": {"left": left, "left_scale": left_scale, "right": right, "right_scale": right_scale}}


def _moe(layer, experts, top, ff, identity=None):
    router = {"experts": experts, "top": top}
    if identity is not None:
        router["identity"] = identity
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff}, "router": router})


def _bare(layer):
    return dict(layer, mlp=None)


def _again(layers, index):
    return dict(layers[index], weights_of=index)


# both layer types, three query heads a key/value head, two value heads a key head, a layer without a feed-forward, the
# first layer's tensors used again two layers on
_A = [
    _moe(_gla(3, 24, 16, 8.0), 6, 2, 24, 2),
    _bare(_parallel(_left(6, 2, 24, 16, 8, 10000.0, 0.21), 0.8, _right(4, 2, 16, 24, 3), 1.3)),
]
RADILIX_A = {
    "architecture": "Radilix", "width": 96, "vocab": 211, "norm": {"eps": 1e-5}, "residual_mult": 0.9,
    "layers": _A + [_again(_A, 0), _moe(_parallel(_left(2, 1, 40, 48, 40, 500.0, 0.1), -0.6, _right(3, 3, 20, 8, 4), 0.7), 5, 3, 32, 3)],
}

# heads of 64 (the sizes the tensor-core kernels take); a parallel layer's tensors used again at once; every router output chosen
_B = [_moe(_parallel(_left(4, 1, 64, 64, 32, 100.0, 0.15), 1.0, _right(2, 2, 64, 64, 4), 1.0), 4, 5, 32, 1)]
RADILIX_B = {
    "architecture": "Radilix", "width": 128, "vocab": 300, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
    "layers": _B + [_again(_B, 0), _moe(_gla(2, 64, 64, 16.0), 8, 3, 16, 4),
                    _bare(_parallel(_left(2, 2, 64, 32, 64, 1e6, 0.12), 0.4, _right(4, 2, 32, 16, 2), 2.0))],
}

# odd sizes, one tap and six, an exponent of one, no identity experts, one expert chosen
RADILIX_C = {
    "architecture": "Radilix", "width": 72, "vocab": 97, "norm": {"eps": 1e-4}, "residual_mult": 1.0,
    "layers": [
        _moe(_gla(1, 10, 7, 1.0), 4, 1, 12),
        _moe(_parallel(_left(3, 3, 6, 10, 2, 10.0, 0.4), 1.1, _right(3, 1, 10, 7, 1), 0.3), 3, 1, 9, 0),
        _bare(_gla(5, 3, 30, 2.5)),
        _moe(_parallel(_left(5, 1, 18, 5, 18, 50.0, 0.3), 0.5, _right(1, 1, 5, 30, 6), -0.9), 7, 4, 8, 5),
    ],
}

# heads of 128 and unequal values, tensors used again through a third layer
_D = [
    _moe(_parallel(_left(4, 2, 128, 32, 96, 30000.0, 0.09), 0.7, _right(4, 1, 128, 32, 4), 0.6), 8, 2, 16, 8),
    _moe(_gla(2, 40, 128, 4.0), 3, 2, 20, 1),
]
RADILIX_D = {
    "architecture": "Radilix", "width": 64, "vocab": 151, "norm": {"eps": 1e-6}, "residual_mult": 1.3,
    "layers": _D + [_again(_D, 1), dict(_D[1], weights_of=2), _bare(_parallel(_left(3, 1, 16, 128, 4, 20.0, 0.3), 1.5, _right(2, 1, 40, 128, 5), 0.2))],
}

# no attention: states alone
_E = [_moe(_gla(4, 16, 20, 3.0), 5, 2, 24, 2)]
RADILIX_E = {
    "architecture": "Radilix", "width": 80, "vocab": 120, "norm": {"eps": 1e-5}, "residual_mult": 0.8,
    "layers": _E + [_again(_E, 0), _bare(_gla(2, 33, 12, 20.0))],
}

RADILIX = {"A": RADILIX_A, "B": RADILIX_B, "C": RADILIX_C, "D": RADILIX_D, "E": RADILIX_E}
# (draws without a first token whose q . k nearly vanishes: the head norm divides such an output by its own small size, and
# float32 itself then loses the digits)
RADILIX_SEEDS = {"A": 51, "B": 52, "C": 63, "D": 54, "E": 85}
RANKS = {"A": 12, "B": 64, "C": 3, "D": 17, "E": 8}   # of the decays' low-rank products


def with_rank(tensors: dict, rank: int, seed: int = 0) -> dict:
    """The low-rank products with a rank of their own (no configuration key names it: the tensors say)."""
    generator = torch.Generator().manual_seed(seed + 5)
    out = dict(tensors)
    for name, tensor in tensors.items():
        if name.endswith(".mix.a1"):
            out[name] = 0.02 * torch.randn(rank, tensor.shape[1], generator=generator)
        elif name.endswith(".mix.a2"):
            out[name] = 0.02 * torch.randn(tensor.shape[0], rank, generator=generator)
    return out


def sharpened(tensors: dict) -> dict:
    """Random weights leave attention nearly uniform, every gate at a half, every decay alike and the routers undecided,
    which hides a key that is wrongly seen or a state that was lost.  This scales what sets the size of the scores, gates,
    decays and choices."""
    out = {}
    for name, tensor in tensors.items():
        t = tensor.clone()
        if name.endswith((".q", ".k", ".v", ".q.b", ".k.b", ".v.b")):
            t *= 6.0
        elif name.endswith((".mix.a1", ".mix.a2")):
            t *= 15.0
        elif name.endswith((".right.b", ".right.a", ".mlp.router", ".g")):
            t *= 12.0
        elif name.endswith((".up", ".down")):
            t *= 8.0
        elif name.endswith(".o"):
            t *= 4.0
        elif name.endswith(".correction"):
            t *= 10.0
        elif name == "embed":
            t *= 40.0
        out[name] = t
    return out


def make_radilix_folder(tmp_path, key: str, dtype: str = "float32", raw: dict | None = None, seed: int | None = None,
                        change=None, rank: int | None = None) -> Path:
    """A model folder (config.json, model.safetensors) of a tiny configuration with sharpened weights.  `change`
    (name -> tensor dictionary, edited in place) lets a test plant a weight of its own."""
    import json

    from shrike_b200 import models  # noqa: F401
    from shrike_b200.config.registry import parse_config
    from shrike_b200.weights.random_init import random_tensors
    from shrike_b200.weights.safetensors_io import write_safetensors

    raw = dict(raw if raw is not None else RADILIX[key])
    seed = RADILIX_SEEDS.get(key, 0) if seed is None else seed
    out = Path(tmp_path) / f"radilix_{key}_{dtype}"
    out.mkdir(parents=True, exist_ok=True)
    tensors = random_tensors(parse_config(raw), seed, "cpu", torch.float32)
    tensors = sharpened(with_rank(tensors, rank or RANKS.get(key, 6), seed))
    if change is not None:
        change(tensors)
    tensors = {name: t.to(getattr(torch, dtype)) for name, t in tensors.items()}
    (out / "config.json").write_text(json.dumps(raw, indent=2) + "\n")
    write_safetensors(out / "model.safetensors", tensors, {"format": "pt", "seed": str(seed)})
    return out


MARK, ASKER = 3, 4   # token ids of `planted_pair`


def planted_pair(raw: dict, which: str, strength: float = 2.0, gain: float = 12.0):
    """A `change` for `make_radilix_folder` on a model whose layer 0 holds the mixer under test (`which`: "gla", "left" or
    "right"): whether token MARK is still there when token ASKER comes decides ASKER's logits, however many tokens lie
    between.

    Residual axis 0 is nonzero in MARK's embedding only and axis 1 in ASKER's only.  Attention: the heads' last key
    dimension (not rotated) reads axis 0 alone and the same query dimension axis 1 alone, so their score stands far above the
    others.  States: key dimension 0 reads axis 0 and query dimension 0 axis 1, nothing else writes or reads that row of the
    state, and its decay is nearly one (where decays are per channel, the last dimension's is near zero; where they are per
    head, the last head's)."""
    spec = raw["layers"][0]["mixer"]

    def change(tensors):
        embed = tensors["embed"]
        embed[:, 0:2] = 0.0
        embed[MARK, 0] = strength * float(embed[:, 2:].std()) * embed.shape[1] ** 0.5
        embed[ASKER, 1] = embed[MARK, 0]
        tensors["l0.norm1"][0:2] = 0.0
        if which == "left":
            dim = spec["left"]["dim"]
            for name, axis, heads in (("q", 1, spec["left"]["heads"]), ("k", 0, spec["left"]["kv_heads"])):
                for a in range(heads):
                    row = a * dim + dim - 1
                    tensors[f"l0.mix.left.{name}"][row] = 0.0
                    tensors[f"l0.mix.left.{name}"][row, axis] = gain
                    tensors[f"l0.mix.left.{name}.b"][row] = 0.0
            tensors["l0.mix.left.o"] *= 3.0
            return
        if which == "right":
            dim, heads, kv_heads, prefix = spec["right"]["dim"], spec["right"]["heads"], spec["right"]["kv_heads"], "l0.mix.right."
        else:
            dim, heads, kv_heads, prefix = spec["dim"], spec["heads"], spec["heads"], "l0.mix."
        tensors[prefix + "o"] *= 3.0
        for a in range(kv_heads):
            for name, axis in (("q", 1), ("k", 0)):
                tensors[f"{prefix}{name}"][a * dim] = 0.0
                tensors[f"{prefix}{name}"][a * dim, axis] = gain
                if which == "right":
                    tensors[f"{prefix}{name}.conv"][a * dim] = 0.0
                    tensors[f"{prefix}{name}.conv"][a * dim, -1] = 1.0
        if which == "right":
            tensors[prefix + "A_log"][:] = 0.0
            tensors[prefix + "a"] *= 0.02
            tensors[prefix + "dt_bias"][:] = -9.0          # a decay of about 0.9999
            tensors[prefix + "dt_bias"][heads - 1] = 4.0   # and one of about 0.02
            return
        for a in range(heads):
            tensors[prefix + "a2"][a * dim] = 0.0
            tensors[prefix + "a2.b"][a * dim] = 9.0                           # a decay of about 0.9999
            tensors[prefix + "a2.b"][a * dim + dim - 1] = -4.0 * spec["tau"]   # and one of about 0.02

    return change
