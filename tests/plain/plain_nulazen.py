"""Plain, slow, whole-sequence implementation of the Nulazen decoder.

One function per mechanism, written from the design's equations; no cache, no batching, no code
shared with the `shrike_b200` package.  It reads the raw `config.json` dictionary and a
name -> tensor dictionary itself.

The design in this file's notation (x: residual [n, W], p: position from 0):

  passes     : layers start .. stop - 1 run `times` times (same weights, fresh memory each pass), then the
               rest once.  Entering pass t (t = 0 too): x <- x + step[t].
  layer i    : x <- x + N1b(mixer(N1(x)));  x <- x + N2b(ff(N2(x))) when the layer has a feed-forward;
               then, with a token side input: e = part i of the token's row of `side.embed`,
               y = P (gelu(G x) * e), x <- x + y / rms(y) * w
  N(x)       = x / sqrt(mean(x^2) + eps) * w
  latent     : q = Wq h, per head [D plain | R turned]; Wdkv h = [c' (rank) | r (R)], c = c' over its root mean
               square times a weight; keys per head [Wuk c | turned r], values Wuv c; j <= i; softmax of
               scale q.k; Wo.  A rotation turns (x[i], x[i + R/2]) by p * base^(-2i/R).
  delta      : q, k, v = silu(conv(W h)), a causal convolution per channel; q and k per head over
               sqrt(sum of squares + 1e-6), q also times D^(-1/2); value head a reads q/k head a // (H / G);
               b = sigmoid(Wb h) per head; g = exp(-exp(A_log) softplus(Wa2 (Wa1 h) + dt_bias)) per head and key
               channel; S <- diag(g) S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q;  every head's o
               over its root mean square times one weight, times sigmoid(Wg2 (Wg1 h)); Wo
  ff dense   : Wd relu(Wu h)^2
  ff moe     : s = softmax(Wr h); c = s + correction; experts in equal groups of neighbours, a group's score
               its largest c, only the best `keep` groups' experts may be chosen; the `top` largest c; out =
               sum over the chosen of s_e expert_e(h) + sigmoid(w h) shared(h);
               expert(h) = Wd (g sigmoid(1.702 g) (u + 1)), g = min(Wg h, L), u = clamp(Wu h, -L, L)
  logits     = head N_final(x)

`rounding=True` rounds to bfloat16 where a bfloat16 engine may (products' inputs and outputs); norms,
scores, softmax, the recurrence and its gates, routers, the residual sum and positions stay in the working
precision.
"""

from __future__ import annotations

import math

import torch

UNIT_EPS = 1e-6


def _r(x: torch.Tensor, on: bool) -> torch.Tensor:
    return x.to(torch.bfloat16).to(x.dtype) if on else x


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z.pow(3))))


def rms_norm(x, weight, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight.to(x.dtype)


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [n, ..., size]: the first `dims` dimensions turn, dimension i with i + dims/2; the rest pass."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = positions.to(x.dtype)[:, None] * freq[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    cos, sin = torch.cos(angle).view(shape), torch.sin(angle).view(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def attend(q, k, v, scale, first_position=0) -> torch.Tensor:
    """q [m, H, D] at positions first_position .., k [ctx, H, D], v [ctx, H, V]: causal softmax attention, [m, H, V]."""
    at = first_position + torch.arange(q.shape[0])
    seen = torch.arange(k.shape[0])[None, :] <= at[:, None]
    scores = torch.einsum("mhd,chd->hmc", q, k) * scale
    weight = torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)
    return torch.einsum("hmc,chv->mhv", weight, v)


def latent_attention(h, weights, prefix, spec, eps, rounding) -> torch.Tensor:
    n, dtype = h.shape[0], h.dtype
    heads, dim, turned, rank = spec["heads"], spec["dim"], spec["rot_dim"], spec["kv_rank"]
    vdim = spec.get("vdim") or dim
    dims, base = spec["rot"]["dims"], spec["rot"]["base"]
    w = lambda name: weights[f"{prefix}.{name}"].to(dtype)  # noqa: E731
    positions = torch.arange(n)
    q = _r(h @ w("q").T, rounding).view(n, heads, dim + turned)
    down = h @ w("dkv").T
    latent = _r(rms_norm(down[:, :rank], w("dkv.norm"), eps), rounding)
    shared = _r(rotate_halves(_r(down[:, rank:], rounding), positions, dims, base), rounding)
    q_turned = _r(rotate_halves(q[..., dim:], positions, dims, base), rounding)
    keys = _r(latent @ w("uk").T, rounding).view(n, heads, dim)
    values = _r(latent @ w("uv").T, rounding).view(n, heads, vdim)
    full_q = torch.cat([q[..., :dim], q_turned], dim=-1)
    full_k = torch.cat([keys, shared[:, None, :].expand(n, heads, turned)], dim=-1)
    out = attend(full_q, full_k, values, spec["scale"])
    return _r(out.reshape(n, heads * vdim), rounding) @ w("o").T


def short_convolution(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [n, channels], taps [channels, T], the last one the current token's; zeros before the start."""
    count = taps.shape[1]
    padded = torch.cat([u.new_zeros(count - 1, u.shape[1]), u], dim=0)
    out = torch.zeros_like(u)
    for j in range(count):
        out = out + padded[j: j + u.shape[0]] * taps[:, j].to(u.dtype)[None, :]
    return out


def unit_heads(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)


def channel_decays(z: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor) -> torch.Tensor:
    """z [n, H, D] (the low-rank product), a_log [H], dt_bias [H * D]: the decays in (0, 1), [n, H, D]."""
    step = torch.nn.functional.softplus(z + dt_bias.view(1, z.shape[1], z.shape[2]), threshold=60.0)
    return torch.exp(-torch.exp(a_log)[None, :, None] * step)


def delta_recurrence(q, k, v, g, beta, state=None):
    """q, k, g [n, H, D], v [n, H, V], beta [n, H], token by token from `state` ([H, D, V]; None: zeros): the state
    decays, what it holds under k is moved towards v by beta, q reads it.  (o [n, H, V], the last state)."""
    n, heads, dim = q.shape
    state = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for t in range(n):
        state = g[t, :, :, None] * state
        held = torch.einsum("hdv,hd->hv", state, k[t])
        u = beta[t, :, None] * (v[t] - held)
        state = state + k[t, :, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", state, q[t])
    return out, state


def channel_delta(h, weights, prefix, spec, eps, rounding, states_out=None) -> torch.Tensor:
    n, dtype = h.shape[0], h.dtype
    heads, groups, dim = spec["heads"], spec["kv_heads"], spec["dim"]
    vdim = spec.get("vdim") or dim
    share = heads // groups
    w = lambda name: weights[f"{prefix}.{name}"].to(dtype)  # noqa: E731
    conv = lambda name: silu(short_convolution(_r(h @ w(name).T, rounding), w(name + ".conv")))  # noqa: E731
    q = unit_heads(conv("q").view(n, groups, dim)) * dim ** -0.5
    k = unit_heads(conv("k").view(n, groups, dim))
    v = conv("v").view(n, heads, vdim)
    beta = torch.sigmoid(h @ w("b").T)
    z = _r(h @ w("a1").T, rounding) @ w("a2").T
    g = channel_decays(z.view(n, heads, dim), w("A_log"), w("dt_bias"))
    out, state = delta_recurrence(q.repeat_interleave(share, 1), k.repeat_interleave(share, 1), v, g, beta)
    if states_out is not None:
        states_out.append(state)
    gate = torch.sigmoid(_r(h @ w("g1").T, rounding) @ w("g2").T)
    gated = rms_norm(out, w("norm"), eps).reshape(n, heads * vdim) * gate
    return _r(gated, rounding) @ w("o").T


def dense(h, weights, prefix, spec, rounding) -> torch.Tensor:
    w = lambda name: weights[f"{prefix}.{name}"].to(h.dtype)  # noqa: E731
    return _r(torch.relu(_r(h @ w("up").T, rounding)).pow(2), rounding) @ w("down").T


def expert(h, weights, prefix, limit, rounding) -> torch.Tensor:
    w = lambda name: weights[f"{prefix}.{name}"].to(h.dtype)  # noqa: E731
    g = _r(h @ w("gate").T, rounding).clamp(max=limit)
    u = _r(h @ w("up").T, rounding).clamp(-limit, limit)
    return _r(g * torch.sigmoid(1.702 * g) * (u + 1.0), rounding) @ w("down").T


def choose(scores: torch.Tensor, correction: torch.Tensor, router: dict, margins=None) -> torch.Tensor:
    """scores [n, E] (softmax over all experts) -> [n, E] True where an expert is chosen.  `margins`, a list,
    receives for every token the smallest gap that could change a choice (of groups or of experts)."""
    n, experts = scores.shape
    choice = scores + correction.to(scores.dtype)
    gaps = torch.full((n,), math.inf, dtype=scores.dtype)
    groups = router.get("groups")
    if groups is not None:
        best = choice.view(n, groups["count"], experts // groups["count"]).max(-1).values
        ranked = torch.sort(best, dim=-1, descending=True, stable=True)
        keep = groups["keep"]
        if keep < groups["count"]:
            gaps = torch.minimum(gaps, ranked.values[:, keep - 1] - ranked.values[:, keep])
        open_group = torch.zeros_like(best, dtype=torch.bool).scatter_(1, ranked.indices[:, :keep], True)
        choice = choice.masked_fill(~open_group.repeat_interleave(experts // groups["count"], 1), -math.inf)
    ranked = torch.sort(choice, dim=-1, descending=True, stable=True)
    top = router["top"]
    if top < experts:
        gaps = torch.minimum(gaps, ranked.values[:, top - 1] - ranked.values[:, top])
    if margins is not None:
        margins.append(gaps)
    return torch.zeros_like(scores, dtype=torch.bool).scatter_(1, ranked.indices[:, :top], True)


def mixture(h, weights, prefix, spec, rounding, margins=None) -> torch.Tensor:
    scores = torch.softmax(h @ weights[f"{prefix}.router"].to(h.dtype).T, dim=-1)
    chosen = choose(scores, weights[f"{prefix}.correction"], spec["router"], margins)
    out = torch.zeros_like(h)
    for e in range(spec["router"]["experts"]):
        rows = chosen[:, e]
        if bool(rows.any()):
            out[rows] += scores[rows, e][:, None] * expert(h[rows], weights, f"{prefix}.e{e}", spec["expert"]["limit"], rounding)
    if spec.get("shared") is not None:
        share = torch.sigmoid(h @ weights[f"{prefix}.shared.sg"].to(h.dtype).T)
        out = out + share * expert(h, weights, f"{prefix}.shared", spec["shared"]["limit"], rounding)
    return out


def token_side(x, weights, index: int, ids, dim: int, eps, rounding) -> torch.Tensor:
    """What layer `index` adds for the tokens' own rows of `side.embed`."""
    w = lambda name: weights[f"l{index}.side.{name}"].to(x.dtype)  # noqa: E731
    e = weights["side.embed"].to(x.dtype)[ids, index * dim: (index + 1) * dim]
    g = _r(gelu_tanh(_r(x, rounding) @ w("gate").T) * e, rounding)
    return rms_norm(g @ w("proj").T, w("norm"), eps)


def layer(x, weights, index: int, spec, raw, ids, rounding, margins=None, states_out=None) -> torch.Tensor:
    name, eps = f"l{index}", raw["norm"]["eps"]
    norm = lambda y, which: rms_norm(y, weights[f"{name}.{which}"], eps)  # noqa: E731
    h = _r(norm(x, "norm1"), rounding)
    if spec["type"] == "latent_attention":
        y = latent_attention(h, weights, name + ".mix", spec["mixer"], eps, rounding)
    elif spec["type"] == "channel_delta":
        y = channel_delta(h, weights, name + ".mix", spec["mixer"], eps, rounding, states_out)
    else:
        raise ValueError(spec["type"])
    x = x + norm(y, "norm1b")
    if spec.get("mlp") is not None:
        h = _r(norm(x, "norm2"), rounding)
        if spec["mlp"].get("kind", "dense") == "dense":
            y = dense(h, weights, name + ".mlp", spec["mlp"], rounding)
        else:
            y = mixture(h, weights, name + ".mlp", spec["mlp"], rounding, margins)
        x = x + norm(y, "norm2b")
    if raw.get("token_side") is not None:
        x = x + token_side(x, weights, index, ids, raw["token_side"]["dim"], eps, rounding)
    return x


def run_order(raw: dict):
    """(layer, pass number or None when the layer's run does not open a pass)."""
    count, loop = len(raw["layers"]), raw.get("loop")
    if not loop:
        return [(i, None) for i in range(count)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], count)]


def forward(raw: dict, weights: dict, tokens, dtype=torch.float64, rounding: bool = False, layers_out=None,
            margins=None, states_out=None) -> torch.Tensor:
    """Logits [n, vocab] of one whole sequence.  `layers_out`, a list, receives the residual after every run; `margins`
    the routers' smallest gaps ([n] per layer run with experts); `states_out` every recurrent state after the last token."""
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = weights["embed"].to(dtype)[ids]
    for index, opens in run_order(raw):
        if opens is not None:
            x = x + weights["loop.step"].to(dtype)[opens]
        x = layer(x, weights, index, raw["layers"][index], raw, ids, rounding, margins, states_out)
        if layers_out is not None:
            layers_out.append(x.clone())
    hidden = _r(rms_norm(x, weights["final.norm"], raw["norm"]["eps"]), rounding)
    return hidden @ weights["head"].to(dtype).T


def greedy_continue(raw: dict, weights: dict, prompt, count: int, dtype=torch.float64):
    """`count` greedy tokens after `prompt`, each from a whole-sequence pass, and the gap between
    the two largest logits at each step."""
    tokens, gaps = list(prompt), []
    for _ in range(count):
        logits = forward(raw, weights, tokens, dtype=dtype)[-1]
        top = torch.topk(logits, 2).values
        gaps.append(float(top[0] - top[1]))
        tokens.append(int(torch.argmax(logits)))
    return tokens[len(prompt):], gaps
