"""Nulazen: a small decoder whose layers are listed one by one in config.json, each with one of two mixers, with a
norm on both sides of every sublayer, a further input per token and layer, and a stretch of layers that runs several
times.

    x = embed[token]
    layers `loop.start` .. `loop.stop` - 1 run `loop.times` times in a row with the same weights and a cache or
    state of their own each pass, then the rest follow.  Entering pass t (the first too): x += loop.step[t].
    layer i:  x += N1b(mixer(N1(x)));  x += N2b(ff(N2(x)));  N(x) = x / sqrt(mean(x^2) + eps) * w
              with `token_side` {dim}: e = part i of the token's row of side.embed,
              x += N_side(proj (gelu_tanh(gate x) * e)); a layer that runs several times reads the same part
    logits = head . N_final(x)

`layers[i]` gives `type` (which mixer), `mixer` (its sizes and constants) and `mlp` (null: none).

  latent_attention  attention over a cached latent of `kv_rank` numbers and one rotated key part of `rot_dim` that all
                    heads share (`heads` / `dim` / `rot_dim` / `vdim`), `rot` {dims, base}: dimension i turns with
                    i + dims/2, `scale`, every key up to the query's own; see `parts/latent_attention.py`
  channel_delta     a delta rule with a decay per key channel (`heads` / `kv_heads` / `dim` / `vdim`) behind
                    convolutions of `conv` taps; see `parts/delta_rule.py`

Feed-forward: `kind` dense (`ff`), down(relu(up x)^2), or moe: `router` {experts, top, groups {count, keep}}: softmax
scores, the choice by score + correction among the experts of the best groups, the scores as they are as weights;
`expert` {ff, limit}: the clamped gate min(g, L) sigmoid(1.702 g) (clamp(u, -L, L) + 1); `shared` {ff, limit}: one more
expert for every token behind a sigmoid gate.  Tensor names: `embed`, `loop.step`, `side.embed`, `l<i>.norm1`,
`l<i>.norm1b`, `l<i>.norm2`, `l<i>.norm2b`, `l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.side.{gate,proj,norm}`, `final.norm`,
`head`.
"""

from __future__ import annotations

from ..config.model_config import (
    ChannelDeltaSpec,
    ConfigError,
    LayerSpec,
    LMHeadSpec,
    MLPSpec,
    ModelConfig,
    PairRotationSpec,
    PassEntrySpec,
    RMSNormSpec,
    RotaryLatentAttentionSpec,
    RoutedExpertsSpec,
    TokenEmbeddingSpec,
    TokenSideSpec,
    TokenSideTableSpec,
    normalise_dtype,
    require,
)
from ..config.registry import Architecture, TensorNames, register_architecture
from .vupitar import _need, _sub, run_order

UNIT_EPS = 1e-6   # added to the sum of squares that makes a delta rule's q and k unit vectors
DEFAULT_MAX_POSITIONS = 1 << 20   # the design has no position table: nothing bounds a sequence but the pool


def _value_dim(raw: dict, dim: int) -> int:
    return raw["vdim"] if raw.get("vdim") is not None else dim


def _latent(raw: dict, width: int, eps: float, where: str) -> RotaryLatentAttentionSpec:
    dim = _need(raw, "dim", int, where)
    rot = _sub(raw, "rot", where)
    return RotaryLatentAttentionSpec(
        width=width, num_heads=_need(raw, "heads", int, where), head_dim=dim, rotary_dim=_need(raw, "rot_dim", int, where),
        value_dim=_value_dim(raw, dim), latent_rank=_need(raw, "kv_rank", int, where),
        scale=float(_need(raw, "scale", float, where)), eps=eps,
        rotation=PairRotationSpec(dims=_need(rot, "dims", int, where + ".rot"), base=float(_need(rot, "base", float, where + ".rot")),
                                  pairing="halves"),
        window=None, gate=None)


def _delta(raw: dict, width: int, eps: float, where: str) -> ChannelDeltaSpec:
    dim = _need(raw, "dim", int, where)
    heads = _need(raw, "heads", int, where)
    return ChannelDeltaSpec(
        width=width, num_heads=heads, num_kv_heads=heads if raw.get("kv_heads") is None else _need(raw, "kv_heads", int, where),
        head_dim=dim, value_dim=_value_dim(raw, dim), conv=_need(raw, "conv", int, where), eps=eps, unit_eps=UNIT_EPS)


_MIXERS = {"latent_attention": _latent, "channel_delta": _delta}


def _feed_forward(mlp: dict, width: int, where: str):
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return MLPSpec(width=width, intermediate=_need(mlp, "ff", int, where), activation="relu2")
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind={kind!r}; known: dense, moe")
    router, expert, shared = _sub(mlp, "router", where), _sub(mlp, "expert", where), mlp.get("shared")
    groups = router.get("groups")
    if groups is not None:
        groups = tuple(_need(groups, key, int, where + ".router.groups") for key in ("count", "keep"))
    return RoutedExpertsSpec(
        width=width, experts=_need(router, "experts", int, where + ".router"), top=_need(router, "top", int, where + ".router"),
        intermediate=_need(expert, "ff", int, where + ".expert"), activation="clamped_swish",
        limit=float(_need(expert, "limit", float, where + ".expert")),
        shared_intermediate=None if shared is None else _need(shared, "ff", int, where + ".shared"),
        shared_limit=None if shared is None else float(_need(shared, "limit", float, where + ".shared")),
        shared_gate=True, scoring="softmax", renormalise=False, correction=True, groups=groups)


def parse_nulazen(raw: dict) -> ModelConfig:
    width = require(raw, "width", int)
    vocab = require(raw, "vocab", int)
    listed = require(raw, "layers")
    if not isinstance(listed, list) or not listed:
        raise ConfigError("config.json: `layers` must be a non-empty list")
    eps = float(require(require(raw, "norm"), "eps", float))
    norm = RMSNormSpec(width=width, eps=eps)
    side = raw.get("token_side")
    side_dim = None if side is None else _need(side, "dim", int, "token_side")
    layers = []
    for index, layer in enumerate(listed):
        where = f"layers[{index}]"
        kind = layer.get("type")
        if kind not in _MIXERS:
            raise ConfigError(f"config.json: {where}.type={kind!r}; known: " + ", ".join(sorted(_MIXERS)))
        mixer = _MIXERS[kind](_sub(layer, "mixer", where), width, eps, where + ".mixer")
        mlp = layer.get("mlp")
        ffn = None if mlp is None else _feed_forward(mlp, width, where + ".mlp")
        extra = [("mixer_out_norm", "norm", norm)]
        if ffn is not None:
            extra.append(("feed_forward_out_norm", "norm", norm))
        if side_dim is not None:
            extra += [("side", "side", TokenSideSpec(width=width, dim=side_dim, index=index)), ("side_norm", "norm", norm)]
        layers.append(LayerSpec(mixer=mixer, mixer_norm=norm, feed_forward=ffn,
                                feed_forward_norm=norm if ffn is not None else None, block="sandwich", extra=tuple(extra)))
    loop = raw.get("loop")
    eos = raw.get("eos_token_id")
    return ModelConfig(
        architecture="Nulazen",
        hidden_size=width,
        vocab_size=vocab,
        layers=layers,
        order=run_order(len(layers), loop),
        final_norm=norm,
        tie_word_embeddings=False,
        max_position_embeddings=int(raw.get("max_positions") or DEFAULT_MAX_POSITIONS),
        eos_token_ids=list(eos) if isinstance(eos, list) else ([] if eos is None else [int(eos)]),
        dtype=normalise_dtype(raw.get("torch_dtype") or raw.get("dtype") or "bfloat16"),
        raw=dict(raw),
        embedding=TokenEmbeddingSpec(vocab=vocab, width=width),
        head=LMHeadSpec(width=width, vocab=vocab, tied=False),
        pass_entry=None if loop is None else PassEntrySpec(width=width, passes=require(loop, "times", int), add_embedding=False),
        side_table=None if side_dim is None else TokenSideTableSpec(vocab=vocab, parts=len(layers), dim=side_dim),
    )


_ROLE_PREFIX = {"mixer": "mix.", "mixer_norm": "norm1", "mixer_out_norm": "norm1b", "feed_forward": "mlp.",
                "feed_forward_norm": "norm2", "feed_forward_out_norm": "norm2b", "side": "side.", "side_norm": "side.norm"}
_MIXER = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
          "kv_down.weight": "dkv", "kv_norm.weight": "dkv.norm", "k_up.weight": "uk", "v_up.weight": "uv",
          "q_conv.weight": "q.conv", "k_conv.weight": "k.conv", "v_conv.weight": "v.conv", "beta.weight": "b",
          "decay_log": "A_log", "decay_bias": "dt_bias", "decay_down.weight": "a1", "decay_up.weight": "a2",
          "gate_down.weight": "g1", "gate_up.weight": "g2", "norm.weight": "norm"}
_PROJECTIONS = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}


def _local(role: str, local: str) -> str:
    """A part's own parameter name -> the last piece of the tensor's name in a Nulazen file."""
    if role.endswith("_norm"):
        return {"weight": ""}[local]
    if role == "mixer":
        return _MIXER[local]
    if role == "feed_forward":
        if local in _PROJECTIONS:
            return _PROJECTIONS[local]
        if local in ("router.weight", "router.correction"):
            return {"router.weight": "router", "router.correction": "correction"}[local]
        if local == "shared_gate.weight":
            return "shared.sg"
        prefix, _, rest = local.rpartition(".")          # experts.<e>.gate_proj | shared.gate_proj, then "weight"
        owner, _, projection = prefix.rpartition(".")
        owner = "shared" if owner == "shared" else "e" + owner.split(".")[1]
        return f"{owner}.{_PROJECTIONS[projection + '.' + rest]}"
    if role == "side":
        return {"gate.weight": "gate", "proj.weight": "proj"}[local]
    if role == "pass_entry":
        return {"step": "loop.step"}[local]
    if role == "side_table":
        return {"weight": "side.embed"}[local]
    raise KeyError((role, local))


def nulazen_tensor_names(config: ModelConfig) -> TensorNames:
    return TensorNames(
        embedding="embed",
        final_norm_prefix="final.norm",
        lm_head="head",
        layer_part=lambda layer, role: f"l{layer}.{_ROLE_PREFIX[role]}",
        embedding_prefix="",
        head_prefix="head.",
        pass_entry_prefix="",
        side_table_prefix="",
        local_name=_local,
    )


NULAZEN = register_architecture(
    Architecture(name="Nulazen", parse_config=parse_nulazen, tensor_names=nulazen_tensor_names)
)
