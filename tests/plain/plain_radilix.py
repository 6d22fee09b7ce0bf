"""Plain, slow, whole-sequence implementation of the Radilix decoder.

One function per mechanism, written from the design's equations; no cache, no batching, no code
shared with the `shrike_b200` package.  It reads the raw `config.json` dictionary and a
name -> tensor dictionary itself.

The design in this file's notation (x: residual [n, W], p: position from 0, m: residual_mult):

  layer      : h = N(x);  x <- x + m (mixer(h) + ff(h)), one norm for both; ff may be absent.  A layer that names
               another one uses that one's tensors, with a memory of its own.
  N(x)       = x / sqrt(mean(x^2) + eps) * (1 + w)
  gla        : q = D^(-1/2) Wq h, k = Wk h, v = Wv h per head; z = Wa2 (Wa1 h) + b per head and key channel,
               a = sigmoid(z)^(1/tau); S <- diag(a) S + k v^T; o = S^T q; every head's o over its root mean square
               times one weight, times silu(Wg h); Wo
  parallel   : left_scale * left(h) + right_scale * right(h)
    left     : q, k, v with biases, query head a reads key/value head a // (H / G); the first R dimensions of q and k
               turn, (x[i], x[i + R/2]) by p * base^(-2i/R); every j <= p; softmax of scale q.k; the heads' outputs
               times sigmoid(Wg h) element by element; Wo
    right    : q, k, v = silu(conv(W h)), a causal convolution per channel; q and k per head over
               sqrt(sum of squares + 1e-6), q also times D^(-1/2); value head a reads q/k head a // (H / G);
               b = sigmoid(Wb h), g = exp(-exp(A_log) softplus(Wa h + dt_bias)), one of each per head; S <- g S;
               u = b (v - S^T k);  S <- S + k u^T;  o = S^T q;  every head's o over its root mean square times one
               weight, times silu(Wg h); Wo
  ff         : s = softmax(Wr h) over the experts and the identity outputs behind them; the `top` largest
               s + correction; out = sum over the chosen of s_e expert_e(h), expert(h) = Wd gelu(Wu h) (the erf
               form), an identity expert gives h
  logits     = head N_final(x)

`rounding=True` rounds to bfloat16 where a bfloat16 engine may (products' inputs and outputs); norms,
scores, softmax, the recurrences and their gates, routers, the residual sum and positions stay in the working
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


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, eps):
    """The residual's norm, whose stored weight is a distance from one."""
    return over_rms(x, eps) * (1.0 + weight.to(x.dtype))


def head_norm(x, weight, eps):
    """x [n, H, V] per head, one plain weight [V] for all heads."""
    return over_rms(x, eps) * weight.to(x.dtype)


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [n, H, D]: the first `dims` dimensions turn, dimension i with i + dims/2; the rest pass."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = positions.to(x.dtype)[:, None] * freq[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def attend(q, k, v, scale, first_position=0) -> torch.Tensor:
    """q [m, H, D] at positions first_position .., k [ctx, G, D], v [ctx, G, V]: causal softmax attention, [m, H, V]."""
    share = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(share, 1), v.repeat_interleave(share, 1)
    at = first_position + torch.arange(q.shape[0])
    seen = torch.arange(k.shape[0])[None, :] <= at[:, None]
    scores = torch.einsum("mhd,chd->hmc", q, k) * scale
    weight = torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)
    return torch.einsum("hmc,chv->mhv", weight, v)


def attention(h, weights, prefix, spec, rounding) -> torch.Tensor:
    n, dtype = h.shape[0], h.dtype
    heads, groups, dim, vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    w = lambda name: weights[f"{prefix}.{name}"].to(dtype)  # noqa: E731
    positions = torch.arange(n)
    q = (h @ w("q").T + w("q.b")).view(n, heads, dim)
    k = (h @ w("k").T + w("k.b")).view(n, groups, dim)
    v = (h @ w("v").T + w("v.b")).view(n, groups, vdim)
    dims, base = spec["rot"]["dims"], spec["rot"]["base"]
    q = _r(rotate_halves(_r(q, rounding), positions, dims, base), rounding)
    k = _r(rotate_halves(_r(k, rounding), positions, dims, base), rounding)
    out = _r(attend(q, k, _r(v, rounding), spec["scale"]).reshape(n, heads * vdim), rounding)
    gated = out * torch.sigmoid(_r(h @ w("g").T, rounding))
    return _r(gated, rounding) @ w("o").T


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


def head_decays(z: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor) -> torch.Tensor:
    """z [n, H]: one decay in (0, 1) a head, [n, H]."""
    step = torch.nn.functional.softplus(z + dt_bias, threshold=60.0)
    return torch.exp(-torch.exp(a_log) * step)


def channel_decays(z: torch.Tensor, tau: float) -> torch.Tensor:
    """sigmoid(z)^(1/tau)."""
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def delta_recurrence(q, k, v, g, beta, state=None):
    """q, k [n, H, D], v [n, H, V], g and beta [n, H], token by token from `state` ([H, D, V]; None: zeros): the state
    decays, what it holds under k is moved towards v by beta, q reads it.  (o [n, H, V], the last state)."""
    n, heads, dim = q.shape
    state = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for t in range(n):
        state = g[t, :, None, None] * state
        held = torch.einsum("hdv,hd->hv", state, k[t])
        u = beta[t, :, None] * (v[t] - held)
        state = state + k[t, :, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", state, q[t])
    return out, state


def gated_recurrence(q, k, v, a, state=None):
    """q, k, a [n, H, D], v [n, H, V]: the state's rows decay by a, k v^T is added, q reads it."""
    n, heads, dim = q.shape
    state = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for t in range(n):
        state = a[t, :, :, None] * state + k[t, :, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", state, q[t])
    return out, state


def delta_rule(h, weights, prefix, spec, eps, rounding, states_out=None) -> torch.Tensor:
    n, dtype = h.shape[0], h.dtype
    heads, groups, dim, vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    share = heads // groups
    w = lambda name: weights[f"{prefix}.{name}"].to(dtype)  # noqa: E731
    conv = lambda name: silu(short_convolution(_r(h @ w(name).T, rounding), w(name + ".conv")))  # noqa: E731
    q = unit_heads(conv("q").view(n, groups, dim)) * dim ** -0.5
    k = unit_heads(conv("k").view(n, groups, dim))
    v = conv("v").view(n, heads, vdim)
    beta = torch.sigmoid(h @ w("b").T)
    g = head_decays(h @ w("a").T, w("A_log"), w("dt_bias"))
    out, state = delta_recurrence(q.repeat_interleave(share, 1), k.repeat_interleave(share, 1), v, g, beta)
    if states_out is not None:
        states_out.append(state)
    gated = head_norm(out, w("norm"), eps).reshape(n, heads * vdim) * silu(_r(h @ w("g").T, rounding))
    return _r(gated, rounding) @ w("o").T


def gated_linear_attention(h, weights, prefix, spec, eps, rounding, states_out=None) -> torch.Tensor:
    n, dtype = h.shape[0], h.dtype
    heads, dim, vdim = spec["heads"], spec["dim"], spec["vdim"]
    w = lambda name: weights[f"{prefix}.{name}"].to(dtype)  # noqa: E731
    q = _r(h @ w("q").T, rounding).view(n, heads, dim) * dim ** -0.5
    k = _r(h @ w("k").T, rounding).view(n, heads, dim)
    v = _r(h @ w("v").T, rounding).view(n, heads, vdim)
    z = _r(h @ w("a1").T, rounding) @ w("a2").T + w("a2.b")
    out, state = gated_recurrence(q, k, v, channel_decays(z.view(n, heads, dim), spec["tau"]))
    if states_out is not None:
        states_out.append(state)
    gated = head_norm(out, w("norm"), eps).reshape(n, heads * vdim) * silu(_r(h @ w("g").T, rounding))
    return _r(gated, rounding) @ w("o").T


def expert(h, weights, prefix, rounding) -> torch.Tensor:
    w = lambda name: weights[f"{prefix}.{name}"].to(h.dtype)  # noqa: E731
    return _r(gelu_erf(_r(h @ w("up").T, rounding)), rounding) @ w("down").T


def choose(scores: torch.Tensor, correction: torch.Tensor, top: int, margins=None) -> torch.Tensor:
    """scores [n, E] (a softmax) -> [n, E] True where an expert is chosen.  `margins`, a list, receives for every token
    the gap between the last choice score taken and the first one left."""
    ranked = torch.sort(scores + correction.to(scores.dtype), dim=-1, descending=True, stable=True)
    if margins is not None:
        full = torch.full((scores.shape[0],), math.inf, dtype=scores.dtype)
        margins.append(full if top == scores.shape[1] else ranked.values[:, top - 1] - ranked.values[:, top])
    return torch.zeros_like(scores, dtype=torch.bool).scatter_(1, ranked.indices[:, :top], True)


def mixture(h, weights, prefix, spec, rounding, margins=None) -> torch.Tensor:
    router = spec["router"]
    scores = torch.softmax(h @ weights[f"{prefix}.router"].to(h.dtype).T, dim=-1)
    chosen = choose(scores, weights[f"{prefix}.correction"], router["top"], margins)
    out = torch.zeros_like(h)
    for e in range(scores.shape[1]):
        rows = chosen[:, e]
        if bool(rows.any()):
            given = expert(h[rows], weights, f"{prefix}.e{e}", rounding) if e < router["experts"] else h[rows]
            out[rows] += scores[rows, e][:, None] * given
    return out


def mixer(h, weights, prefix, entry, eps, rounding, states_out=None) -> torch.Tensor:
    spec = entry["mixer"]
    if entry["type"] == "gla":
        return gated_linear_attention(h, weights, prefix, spec, eps, rounding, states_out)
    if entry["type"] == "parallel":
        left = attention(h, weights, prefix + ".left", spec["left"], rounding)
        right = delta_rule(h, weights, prefix + ".right", spec["right"], eps, rounding, states_out)
        return spec["left_scale"] * left + spec["right_scale"] * right
    raise ValueError(entry["type"])


def tensors_of(raw: dict, index: int) -> int:
    """The layer whose tensors layer `index` uses."""
    while raw["layers"][index].get("weights_of") is not None:
        index = raw["layers"][index]["weights_of"]
    return index


def layer(x, weights, raw, index, rounding, margins=None, states_out=None) -> torch.Tensor:
    entry, eps, name = raw["layers"][index], raw["norm"]["eps"], f"l{tensors_of(raw, index)}"
    h = _r(layer_norm(x, weights[f"{name}.norm1"], eps), rounding)
    y = mixer(h, weights, name + ".mix", entry, eps, rounding, states_out)
    if entry.get("mlp") is not None:
        y = y + mixture(h, weights, name + ".mlp", entry["mlp"], rounding, margins)
    return x + raw["residual_mult"] * y


def forward(raw: dict, weights: dict, tokens, dtype=torch.float64, rounding: bool = False, layers_out=None,
            margins=None, states_out=None) -> torch.Tensor:
    """Logits [n, vocab] of one whole sequence.  `layers_out`, a list, receives the residual after every run; `margins`
    the routers' smallest gaps ([n] per layer run with experts); `states_out` every recurrent state after the last token."""
    x = weights["embed"].to(dtype)[torch.as_tensor(tokens, dtype=torch.long)]
    for index in range(len(raw["layers"])):
        x = layer(x, weights, raw, index, rounding, margins, states_out)
        if layers_out is not None:
            layers_out.append(x.clone())
    hidden = _r(layer_norm(x, weights["final.norm"], raw["norm"]["eps"]), rounding)
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
