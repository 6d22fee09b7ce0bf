"""Delta rules whose state decays: per key channel (`ChannelDelta`) or by one number a head (`HeadDelta`).

`ChannelDelta`, a gated delta rule with a vector of decays.

q and k (heads of `head_dim`) and v (heads of `value_dim`) are projections of x, each behind a causal convolution over
time per channel and a SiLU; q and k are unit vectors per head, q also times head_dim^(-1/2).  Per value head, with
beta = sigmoid(Wb x) and decays g = exp(-exp(A_log) softplus(Wa2 Wa1 x + dt_bias)) per key channel,

    S <- diag(g) S      u = beta (v - S^T k)      S <- S + k u^T      o = S^T q          (S = 0 at the start)

what the state holds under k is moved towards v by the share beta.  Every head's o is divided by its root mean square,
scaled by one weight of the head's size, multiplied by sigmoid(Wg2 Wg1 x) and projected.  Several value heads may share
a q/k head; decays and beta are the value head's own.

How it runs here: q, k, v, beta and the two low-rank rows are ONE product; `delta_prep` turns its 32-bit result into the
convolved, normed q, k and v, beta and the low-rank rows in the engine's type (the convolution's last inputs are the
request's state, named "conv"); a second product gives decays and output gates from the low-rank rows (a block-diagonal
matrix over both); `delta_scan` runs the recurrence on the request's float32 state slot
`[heads, head_dim * value_dim (rounded up to four)]`; `head_rms` norms, gates and casts.  Both states are zeroed by the
step function when the request is opened.  The ranks of the low-rank products come from the model's tensors.

`HeadDelta`, the same rule with one decay a head, g = exp(-exp(A_log) softplus(Wa x + dt_bias)), and an output gate
silu(Wg x): decay and gate columns are part of the one product, whose 32-bit result the scan and the head norm read, so
there is no second product.
"""

from __future__ import annotations

import torch

from .base import ParamSpec, StateNeed, register_part
from .matrix_memory import padded_rows


def _up(count: int, multiple: int) -> int:
    return -(-count // multiple) * multiple


class ChannelDelta:
    capture_safe = True   # it reads the batch's metadata on the device only and leaves rows alone whose state slot is -1

    @staticmethod
    def channels(spec) -> int:
        return 2 * spec.num_kv_heads * spec.head_dim + spec.num_heads * spec.value_dim

    @staticmethod
    def parameters(spec) -> dict[str, ParamSpec]:
        qk, v = spec.num_kv_heads * spec.head_dim, spec.num_heads * spec.value_dim
        decays = spec.num_heads * spec.head_dim
        decay_rank, gate_rank = spec.decay_rank or spec.head_dim, spec.gate_rank or spec.head_dim
        return {
            "q_proj.weight": ParamSpec((qk, spec.width), "matrix"),
            "k_proj.weight": ParamSpec((qk, spec.width), "matrix"),
            "v_proj.weight": ParamSpec((v, spec.width), "matrix"),
            "q_conv.weight": ParamSpec((qk, spec.conv), "conv"),
            "k_conv.weight": ParamSpec((qk, spec.conv), "conv"),
            "v_conv.weight": ParamSpec((v, spec.conv), "conv"),
            "beta.weight": ParamSpec((spec.num_heads, spec.width), "matrix"),
            "decay_log": ParamSpec((spec.num_heads,), "decay_rate"),
            "decay_bias": ParamSpec((decays,), "decay_bias"),
            "decay_down.weight": ParamSpec((decay_rank, spec.width), "matrix", free=(0,)),
            "decay_up.weight": ParamSpec((decays, decay_rank), "matrix", free=(1,)),
            "gate_down.weight": ParamSpec((gate_rank, spec.width), "matrix", free=(0,)),
            "gate_up.weight": ParamSpec((v, gate_rank), "matrix", free=(1,)),
            "norm.weight": ParamSpec((spec.value_dim,), "norm"),
            "o_proj.weight": ParamSpec((spec.width, v), "matrix"),
        }

    @staticmethod
    def state_shape(spec) -> tuple:
        return (spec.num_heads, _up(spec.head_dim * spec.value_dim, 4))   # every head starts on a 16-byte border

    @staticmethod
    def cache_needs(spec) -> list:
        needs = [StateNeed(ChannelDelta.state_shape(spec), "float32")]
        if spec.conv > 1:
            needs.append(StateNeed((spec.conv - 1, ChannelDelta.channels(spec)), "float32", name="conv"))
        return needs

    def __init__(self, spec, tensors, ops, runtime):
        self.spec, self.ops, self.runtime = spec, ops, runtime
        heads, qk, v = spec.num_heads, spec.num_kv_heads * spec.head_dim, spec.num_heads * spec.value_dim
        decays = heads * spec.head_dim
        a1, a2 = tensors.pop("decay_down.weight"), tensors.pop("decay_up.weight")
        g1, g2 = tensors.pop("gate_down.weight"), tensors.pop("gate_up.weight")
        for down, up, what in ((a1, a2, "decay"), (g1, g2, "gate")):
            if down.shape[0] != up.shape[1]:
                raise ValueError(f"the {what}'s low-rank product does not fit: {tuple(down.shape)} then {tuple(up.shape)}")

        def zero_rows(matrix, count):
            return torch.cat([matrix, matrix.new_zeros(count - matrix.shape[0], matrix.shape[1])])

        # rows: q | k | v | beta | decay's low-rank rows | gate's; beta and each low-rank part padded with zero rows
        beta = tensors.pop("beta.weight")
        self.beta_at = 2 * qk + v
        self.low_at = self.beta_at + _up(heads, 4)
        a_rank, g_rank = _up(a1.shape[0], 8), _up(g1.shape[0], 8)
        self.low = a_rank + g_rank
        rows = [tensors.pop(name) for name in ("q_proj.weight", "k_proj.weight", "v_proj.weight")]
        rows += [zero_rows(beta.to(a1.dtype), _up(heads, 4)), zero_rows(a1, a_rank), zero_rows(g1, g_rank)]
        self.w_fused = padded_rows(torch.cat(rows))
        self.total = self.w_fused.shape[0]
        # both second products as one: decay rows meet the decay's low-rank columns alone, gate rows the gate's
        self.w_gates = a2.new_zeros(_up(decays + v, 16), self.low)
        self.w_gates[:decays, : a2.shape[1]] = a2
        self.w_gates[decays: decays + v, a_rank: a_rank + g2.shape[1]] = g2
        self.gate_at = decays   # the output gate's first column of the second product
        self.taps = torch.cat([tensors.pop(f"{name}_conv.weight") for name in ("q", "k", "v")]).to(torch.float32).contiguous()
        self.no_state = torch.zeros(1, 0, ChannelDelta.channels(spec), dtype=torch.float32, device=runtime.device)
        self.rate = tensors.pop("decay_log").to(torch.float32).exp().contiguous()   # what softplus(.) is multiplied by
        self.bias = tensors.pop("decay_bias").to(torch.float32).contiguous()
        self.norm_weight = tensors.pop("norm.weight").to(torch.float32).contiguous()
        self.w_o = tensors.pop("o_proj.weight").contiguous()
        self.out_width = v

    def forward(self, x, ctx, run):
        spec, rt, ops = self.spec, self.runtime, self.ops
        if not run.writes_cache:
            raise NotImplementedError("a delta rule owns its state: no run can read another run's")
        n = x.shape[0]
        fused = rt.buffer("memory_in", (n, self.total), torch.float32)
        fused = ops.linear(x, self.w_fused, fused, allow_partials=True)
        mixed = rt.buffer("delta_mixed", (n, self.channels(spec)), torch.float32)
        beta = rt.buffer("delta_beta", (n, spec.num_heads), torch.float32)
        low = rt.buffer("delta_low", (n, self.low), rt.act_dtype)
        conv_state = ctx.storage.state[(run.cache, "conv")] if spec.conv > 1 else self.no_state
        ops.delta_prep(fused, self.taps, conv_state, ctx.q_start, ctx.state_slot, ctx.seq_of_token, mixed, beta, low,
                       ctx.num_seqs, spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim, self.beta_at,
                       self.low_at, spec.unit_eps, longest=ctx.max_q_len)
        gates = rt.buffer("delta_gates", (n, self.w_gates.shape[0]), torch.float32)
        gates = ops.linear(low, self.w_gates, gates, allow_partials=True)
        scanned = rt.buffer("memory_num", (n, self.out_width), torch.float32)
        ops.delta_scan(mixed, beta, gates, self.rate, self.bias, ctx.storage.state[run.cache], ctx.q_start, ctx.state_slot,
                       scanned, ctx.num_seqs, spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim, q_lens=ctx.q_lens,
                       early_state=True)   # a run's state is its own: only earlier steps wrote it
        out = rt.buffer("memory_out", (n, self.out_width), rt.act_dtype)
        ops.head_rms(scanned, self.norm_weight, spec.eps, out, spec.num_heads, gate_source=gates, gate_at=self.gate_at)
        delta = rt.buffer("memory_delta", (n, spec.width), torch.float32)
        return ops.linear(out, self.w_o, delta, allow_partials=True)


register_part("mixer", "channel_delta", ChannelDelta)


class HeadDelta:
    capture_safe = True   # it reads the batch's metadata on the device only and leaves rows alone whose state slot is -1

    @staticmethod
    def parameters(spec) -> dict[str, ParamSpec]:
        qk, v = spec.num_kv_heads * spec.head_dim, spec.num_heads * spec.value_dim
        return {
            "q_proj.weight": ParamSpec((qk, spec.width), "matrix"),
            "k_proj.weight": ParamSpec((qk, spec.width), "matrix"),
            "v_proj.weight": ParamSpec((v, spec.width), "matrix"),
            "q_conv.weight": ParamSpec((qk, spec.conv), "conv"),
            "k_conv.weight": ParamSpec((qk, spec.conv), "conv"),
            "v_conv.weight": ParamSpec((v, spec.conv), "conv"),
            "beta.weight": ParamSpec((spec.num_heads, spec.width), "matrix"),
            "decay.weight": ParamSpec((spec.num_heads, spec.width), "matrix"),
            "decay_log": ParamSpec((spec.num_heads,), "decay_rate"),
            "decay_bias": ParamSpec((spec.num_heads,), "decay_bias"),
            "gate.weight": ParamSpec((v, spec.width), "matrix"),
            "norm.weight": ParamSpec((spec.value_dim,), "norm"),
            "o_proj.weight": ParamSpec((spec.width, v), "matrix"),
        }

    cache_needs = staticmethod(ChannelDelta.cache_needs)   # the same two states: S, and the convolution's last inputs

    def __init__(self, spec, tensors, ops, runtime):
        self.spec, self.ops, self.runtime = spec, ops, runtime
        self.channels = ChannelDelta.channels(spec)
        self.out_width = spec.num_heads * spec.value_dim
        # rows: q | k | v | gate | beta | decay
        rows = [tensors.pop(f"{name}.weight") for name in ("q_proj", "k_proj", "v_proj", "gate")]
        rows += [tensors.pop(f"{name}.weight").to(rows[0].dtype) for name in ("beta", "decay")]
        self.gate_at = self.channels
        self.beta_at = self.gate_at + self.out_width
        self.decay_at = self.beta_at + spec.num_heads
        self.w_fused = padded_rows(torch.cat(rows))
        self.total = self.w_fused.shape[0]
        self.taps = torch.cat([tensors.pop(f"{name}_conv.weight") for name in ("q", "k", "v")]).to(torch.float32).contiguous()
        self.no_state = torch.zeros(1, 0, self.channels, dtype=torch.float32, device=runtime.device)
        self.rate = tensors.pop("decay_log").to(torch.float32).exp().contiguous()   # what softplus(.) is multiplied by
        self.bias = tensors.pop("decay_bias").to(torch.float32).contiguous()
        self.norm_weight = tensors.pop("norm.weight").to(torch.float32).contiguous()
        self.w_o = tensors.pop("o_proj.weight").contiguous()

    def forward(self, x, ctx, run):
        spec, rt, ops = self.spec, self.runtime, self.ops
        if not run.writes_cache:
            raise NotImplementedError("a delta rule owns its state: no run can read another run's")
        n = x.shape[0]
        fused = rt.buffer("memory_in", (n, self.total), torch.float32)
        fused = ops.linear(x, self.w_fused, fused, allow_partials=True)
        mixed = rt.buffer("delta_mixed", (n, self.channels), torch.float32)
        beta = rt.buffer("delta_beta", (n, spec.num_heads), torch.float32)
        conv_state = ctx.storage.state[(run.cache, "conv")] if spec.conv > 1 else self.no_state
        ops.delta_prep(fused, self.taps, conv_state, ctx.q_start, ctx.state_slot, ctx.seq_of_token, mixed, beta, None,
                       ctx.num_seqs, spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim, self.beta_at,
                       0, spec.unit_eps, longest=ctx.max_q_len)
        scanned = rt.buffer("memory_num", (n, self.out_width), torch.float32)
        ops.delta_scan(mixed, beta, fused, self.rate, self.bias, ctx.storage.state[run.cache], ctx.q_start, ctx.state_slot,
                       scanned, ctx.num_seqs, spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim, q_lens=ctx.q_lens,
                       early_state=True, gate_at=self.decay_at, per_head=True)   # only earlier steps wrote a run's own state
        out = rt.buffer("memory_out", (n, self.out_width), rt.act_dtype)
        ops.head_rms(scanned, self.norm_weight, spec.eps, out, spec.num_heads, gate_source=fused, gate_at=self.gate_at, gate="silu")
        delta = rt.buffer("memory_delta", (n, spec.width), torch.float32)
        return ops.linear(out, self.w_o, delta, allow_partials=True)


register_part("mixer", "head_delta", HeadDelta)
