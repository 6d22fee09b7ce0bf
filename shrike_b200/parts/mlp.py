"""Dense feed-forwards.

`MLP`, without a gate: down(act(up(x))), the activation inside the first product where the kernels offer that.

`GatedMLP`: down(act(gate(x)) * up(x)), no biases
(shrike/models/qwen.py:128-136).  Gate and up are one matrix product (rows of Wg and
Wu stacked at load: all gate rows then all up rows, or, where the kernels can apply the
activation inside the product, runs of gate rows each followed by the up rows of the same
features); the activation product is formed in 32-bit."""

from __future__ import annotations

import torch

from .base import ParamSpec, register_part


# gelu_tanh(z) = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)));
# clamped_swish with limit L: g <- min(g, L), u <- clamp(u, -L, L), then g sigmoid(1.702 g) (u + 1) in place of act(g) u
ACTIVATIONS = ("silu", "gelu_tanh", "clamped_swish")
# act(z) of an ungated feed-forward: relu2 is max(z, 0)^2, gelu z (1 + erf(z / sqrt(2))) / 2
PLAIN_ACTIVATIONS = ("relu2", "gelu")


class GatedMLP:
    capture_safe = True   # forward() launches the same kernels for the same batch shape, whatever the positions

    @staticmethod
    def parameters(spec) -> dict[str, ParamSpec]:
        return {
            "gate_proj.weight": ParamSpec((spec.intermediate, spec.width), "matrix"),
            "up_proj.weight": ParamSpec((spec.intermediate, spec.width), "matrix"),
            "down_proj.weight": ParamSpec((spec.width, spec.intermediate), "matrix"),
        }

    def __init__(self, spec, tensors, ops, runtime):
        if spec.activation not in ACTIVATIONS:
            raise ValueError(f"gated feed-forward activation {spec.activation!r} has no kernel; known: "
                             + ", ".join(ACTIVATIONS))
        self.spec = spec
        self.ops = ops
        self.runtime = runtime
        self.limit = getattr(spec, "limit", None)
        if spec.activation == "clamped_swish" and (self.limit is None or not self.limit > 0):
            raise ValueError("the clamped activation needs a positive limit")
        gate, up = tensors.pop("gate_proj.weight"), tensors.pop("up_proj.weight")
        run = getattr(ops, "gated_rows", 0)
        self.run = run if run and spec.intermediate % run == 0 else 0
        if self.run:
            blocks = spec.intermediate // self.run
            stacked = torch.stack([gate.view(blocks, self.run, -1), up.view(blocks, self.run, -1)], dim=1)
            self.w_gate_up = stacked.reshape(2 * spec.intermediate, -1).contiguous()
        else:
            self.w_gate_up = torch.cat([gate, up]).contiguous()
        self.w_down = tensors.pop("down_proj.weight").contiguous()

    def forward(self, x, ctx):
        spec, rt, ops = self.spec, self.runtime, self.ops
        n = x.shape[0]
        act = rt.buffer("ffn_act", (n, spec.intermediate), rt.act_dtype)
        extra = {} if self.limit is None else {"limit": self.limit}
        if not (self.run and ops.linear_gated(x, self.w_gate_up, act, spec.activation, **extra)):
            gate_up = rt.buffer("gate_up", (n, 2 * spec.intermediate), rt.act_dtype)
            ops.linear(x, self.w_gate_up, gate_up)
            ops.act_mul(gate_up, act, self.run, spec.activation, **extra)
        delta = rt.buffer("ffn_delta", (n, spec.width), torch.float32)
        return ops.linear(act, self.w_down, delta, allow_partials=True)


class MLP:
    capture_safe = True

    @staticmethod
    def parameters(spec) -> dict[str, ParamSpec]:
        return {"up_proj.weight": ParamSpec((spec.intermediate, spec.width), "matrix"),
                "down_proj.weight": ParamSpec((spec.width, spec.intermediate), "matrix")}

    def __init__(self, spec, tensors, ops, runtime):
        if spec.activation not in PLAIN_ACTIVATIONS:
            raise ValueError(f"feed-forward activation {spec.activation!r} has no kernel; known: " + ", ".join(PLAIN_ACTIVATIONS))
        self.spec, self.ops, self.runtime = spec, ops, runtime
        self.w_up = tensors.pop("up_proj.weight").contiguous()
        self.w_down = tensors.pop("down_proj.weight").contiguous()

    def forward(self, x, ctx):
        spec, rt, ops = self.spec, self.runtime, self.ops
        n = x.shape[0]
        act = rt.buffer("ffn_act", (n, spec.intermediate), rt.act_dtype)
        ops.linear_act(x, self.w_up, act, spec.activation)
        delta = rt.buffer("ffn_delta", (n, spec.width), torch.float32)
        return ops.linear(act, self.w_down, delta, allow_partials=True)


register_part("feed_forward", "mlp", MLP)
register_part("feed_forward", "gated_mlp", GatedMLP)
