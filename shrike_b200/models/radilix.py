"""Radilix: a small decoder whose layers are listed one by one in config.json, each one norm whose output a mixer and a
mixture of experts read side by side.

    x = embed[token]
    layer:  h = N(x);  x += residual_mult * (mixer(h) + ff(h));  N(x) = x / sqrt(mean(x^2) + eps) * (1 + w)
    logits = head . N_final(x)

`layers[i]` gives `type` (which mixer), `mixer` (its sizes and constants) and `mlp` (null: none).  A layer with `weights_of`:
j has no tensors of its own; it runs layer j's parts on a cache and states of its own.

  gla        gated linear attention (`heads` / `dim` / `vdim`, `tau`), a state that decays per key channel; see
             `parts/linear_attention.py`
  parallel   two mixers that read the same input, left_scale * left + right_scale * right.  `left`: grouped-query softmax
             attention with biases on q, k and v (`heads` / `kv_heads` / `dim` / `vdim`, `scale`), the first `rot.dims`
             dimensions of each head rotated (dimension i with i + dims/2, base `rot.base`), every key up to the query's
             own, an output gate per element.  `right`: the delta rule with one decay a head (`heads` / `kv_heads` / `dim` /
             `vdim`, convolutions of `conv` taps); see `parts/delta_rule.py`

Feed-forward: `kind` moe: `expert` {ff}: down(gelu(up x)), the erf form; `router` {experts, top, identity}: softmax scores
over the experts and `identity` further outputs whose expert is the input itself, the choice by score + correction, the
scores as they are as weights.  Tensor names: `embed`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""

from __future__ import annotations

from ..config.model_config import (
    ConfigError,
    GatedHeadAttentionSpec,
    GatedLinearAttentionSpec,
    HeadDeltaSpec,
    LayerRun,
    LayerSpec,
    LMHeadSpec,
    ModelConfig,
    ParallelMixerSpec,
    RMSNormSpec,
    RoutedExpertsSpec,
    TokenEmbeddingSpec,
    normalise_dtype,
    require,
)
from ..config.registry import Architecture, TensorNames, register_architecture
from .vupitar import _need, _sub

NORM_OFFSET = 1.0   # the norm weights of the residual are stored as their distance from one
UNIT_EPS = 1e-6     # added to the sum of squares that makes a delta rule's q and k unit vectors
DEFAULT_MAX_POSITIONS = 1 << 20   # the design has no position table: nothing bounds a sequence but the pool


def _or(raw: dict, key: str, default: int, where: str) -> int:
    return default if raw.get(key) is None else _need(raw, key, int, where)


def _gla(raw: dict, width: int, eps: float, where: str) -> GatedLinearAttentionSpec:
    dim = _need(raw, "dim", int, where)
    return GatedLinearAttentionSpec(width=width, num_heads=_need(raw, "heads", int, where), head_dim=dim,
                                    value_dim=_or(raw, "vdim", dim, where), tau=float(_need(raw, "tau", float, where)), eps=eps)


def _left(raw: dict, width: int, eps: float, where: str) -> GatedHeadAttentionSpec:
    dim, heads, rot = _need(raw, "dim", int, where), _need(raw, "heads", int, where), raw.get("rot")
    return GatedHeadAttentionSpec(
        width=width, num_heads=heads, num_kv_heads=_or(raw, "kv_heads", heads, where), head_dim=dim,
        value_dim=_or(raw, "vdim", dim, where), scale=float(_need(raw, "scale", float, where)), eps=eps, qkv_bias=True,
        rotary=None if rot is None else (_need(rot, "dims", int, where + ".rot"), float(_need(rot, "base", float, where + ".rot"))),
        element_gate=True)


def _right(raw: dict, width: int, eps: float, where: str) -> HeadDeltaSpec:
    dim, heads = _need(raw, "dim", int, where), _need(raw, "heads", int, where)
    return HeadDeltaSpec(width=width, num_heads=heads, num_kv_heads=_or(raw, "kv_heads", heads, where), head_dim=dim,
                         value_dim=_or(raw, "vdim", dim, where), conv=_need(raw, "conv", int, where), eps=eps, unit_eps=UNIT_EPS)


def _parallel(raw: dict, width: int, eps: float, where: str) -> ParallelMixerSpec:
    return ParallelMixerSpec(width=width, branches=(
        ("left", _left(_sub(raw, "left", where), width, eps, where + ".left"), float(_need(raw, "left_scale", float, where))),
        ("right", _right(_sub(raw, "right", where), width, eps, where + ".right"), float(_need(raw, "right_scale", float, where))),
    ))


_MIXERS = {"gla": _gla, "parallel": _parallel}


def _feed_forward(mlp: dict, width: int, where: str) -> RoutedExpertsSpec:
    if mlp.get("kind", "moe") != "moe":
        raise ConfigError(f"config.json: {where}.kind={mlp['kind']!r}; known: moe")
    router = _sub(mlp, "router", where)
    identity = router.get("identity") or 0
    if isinstance(identity, bool) or not isinstance(identity, int):
        raise ConfigError(f"config.json: {where}.router.identity must be an integer, got {identity!r}")
    return RoutedExpertsSpec(
        width=width, experts=_need(router, "experts", int, where + ".router"), top=_need(router, "top", int, where + ".router"),
        intermediate=_need(_sub(mlp, "expert", where), "ff", int, where + ".expert"), activation="gelu", gated=False,
        identity=identity, scoring="softmax", renormalise=False, correction=True)


def _owners(listed: list) -> list[int]:
    """For every layer the layer whose tensors it uses."""
    owners = []
    for index, layer in enumerate(listed):
        seen, owner = [index], index
        while listed[owner].get("weights_of") is not None:
            owner = listed[owner]["weights_of"]
            if isinstance(owner, bool) or not isinstance(owner, int) or not 0 <= owner < len(listed) or owner in seen:
                raise ConfigError(f"config.json: layers[{index}].weights_of leads to {owner!r}, which is no other layer with tensors")
            seen.append(owner)
        if any(layer.get(key) != listed[owner].get(key) for key in ("type", "mixer", "mlp")):
            raise ConfigError(f"config.json: layers[{index}] uses the tensors of layers[{owner}] but is not described alike")
        owners.append(owner)
    return owners


def parse_radilix(raw: dict) -> ModelConfig:
    width = require(raw, "width", int)
    vocab = require(raw, "vocab", int)
    listed = require(raw, "layers")
    if not isinstance(listed, list) or not listed:
        raise ConfigError("config.json: `layers` must be a non-empty list")
    eps = float(require(require(raw, "norm"), "eps", float))
    mult = float(require(raw, "residual_mult", float))
    norm = RMSNormSpec(width=width, eps=eps, offset=NORM_OFFSET)
    owners = _owners(listed)
    held = sorted(set(owners))   # the layers that have tensors, in the order the model holds them
    layers = []
    for index in held:
        layer, where = listed[index], f"layers[{index}]"
        kind = layer.get("type")
        if kind not in _MIXERS:
            raise ConfigError(f"config.json: {where}.type={kind!r}; known: " + ", ".join(sorted(_MIXERS)))
        mlp = layer.get("mlp")
        layers.append(LayerSpec(
            mixer=_MIXERS[kind](_sub(layer, "mixer", where), width, eps, where + ".mixer"), mixer_norm=norm,
            feed_forward=None if mlp is None else _feed_forward(mlp, width, where + ".mlp"), feed_forward_norm=None,
            block="parallel", block_options=(("scale", mult),)))
    eos = raw.get("eos_token_id")
    return ModelConfig(
        architecture="Radilix",
        hidden_size=width,
        vocab_size=vocab,
        layers=layers,
        order=[LayerRun(layer=held.index(owner), cache=index) for index, owner in enumerate(owners)],
        final_norm=norm,
        tie_word_embeddings=False,
        max_position_embeddings=int(raw.get("max_positions") or DEFAULT_MAX_POSITIONS),
        eos_token_ids=list(eos) if isinstance(eos, list) else ([] if eos is None else [int(eos)]),
        dtype=normalise_dtype(raw.get("torch_dtype") or raw.get("dtype") or "bfloat16"),
        raw=dict(raw),
        embedding=TokenEmbeddingSpec(vocab=vocab, width=width),
        head=LMHeadSpec(width=width, vocab=vocab, tied=False),
    )


_ROLE_PREFIX = {"mixer": "mix.", "mixer_norm": "norm1", "feed_forward": "mlp."}
_ATTENTION = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o", "q_proj.bias": "q.b",
              "k_proj.bias": "k.b", "v_proj.bias": "v.b", "gate.weight": "g"}
_RECURRENT = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o", "gate.weight": "g",
              "norm.weight": "norm", "q_conv.weight": "q.conv", "k_conv.weight": "k.conv", "v_conv.weight": "v.conv",
              "beta.weight": "b", "decay.weight": "a", "decay_log": "A_log", "decay_bias": "dt_bias", "decay_down.weight": "a1",
              "decay_up.weight": "a2", "decay_up.bias": "a2.b"}
_EXPERT = {"up_proj.weight": "up", "down_proj.weight": "down"}


def _local(role: str, local: str) -> str:
    """A part's own parameter name -> the last piece of the tensor's name in a Radilix file."""
    if role.endswith("_norm"):
        return {"weight": ""}[local]
    if role == "mixer":
        branch, _, rest = local.partition(".")
        if branch == "left":
            return "left." + _ATTENTION[rest]
        return "right." + _RECURRENT[rest] if branch == "right" else _RECURRENT[local]
    if role == "feed_forward":
        if local in ("router.weight", "router.correction"):
            return {"router.weight": "router", "router.correction": "correction"}[local]
        _, expert, rest = local.split(".", 2)   # experts.<e>.up_proj.weight
        return f"e{expert}.{_EXPERT[rest]}"
    raise KeyError((role, local))


def radilix_tensor_names(config: ModelConfig) -> TensorNames:
    # layers without tensors of their own leave gaps in the numbering
    held = sorted(set(_owners(config.raw["layers"])))
    return TensorNames(
        embedding="embed",
        final_norm_prefix="final.norm",
        lm_head="head",
        layer_part=lambda layer, role: f"l{held[layer]}.{_ROLE_PREFIX[role]}",
        embedding_prefix="",
        head_prefix="head.",
        local_name=_local,
    )


RADILIX = register_architecture(
    Architecture(name="Radilix", parse_config=parse_radilix, tensor_names=radilix_tensor_names)
)
