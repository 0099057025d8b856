"""Feed-forward parts.

Reference: SwiGLU with gate and up fused on the output axis at load
(src/mlx_omnia/engine/core/layers.py:253-272, src/mlx_omnia/engine/checkpoint.py:333-347).
"""

from __future__ import annotations

import torch

from mlx_omnia_b200.kernels import ops
from mlx_omnia_b200.parts.base import FeedForward, TensorSpec, register_feed_forward


@register_feed_forward("gated_mlp")
class GatedMLP(FeedForward):
    """down(silu(gate(h)) * up(h)), no biases.

    hidden, inner: widths. The checkpoint's `gate_proj` and `up_proj` are stacked into
    one [2 * inner, hidden] operand at load so the step runs one product for both.
    """

    takes_pending = True

    def __init__(self, hidden: int, inner: int) -> None:
        self.hidden, self.inner = hidden, inner

    def tensors(self) -> dict[str, TensorSpec]:
        return {
            "gate_proj.weight": TensorSpec((self.inner, self.hidden)),
            "up_proj.weight": TensorSpec((self.inner, self.hidden)),
            "down_proj.weight": TensorSpec((self.hidden, self.inner)),
        }

    def load(self, tensors, runtime) -> None:
        super().load(tensors, runtime)
        self.gate_up = torch.cat([tensors["gate_proj.weight"], tensors["up_proj.weight"]], dim=0).contiguous()
        self.down = tensors["down_proj.weight"].contiguous()

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return ops.linear(ops.linear_swiglu(h, self.gate_up), self.down)


@register_feed_forward("dense_mlp")
class DenseMLP(FeedForward):
    """down(act(up(h))), no biases and no gate.

    hidden, inner: widths; activation: "relu2" (the square of relu), "gelu_tanh", "silu" or "xielu".
    xielu has two learned numbers p, q (tensor `act` [2]): softplus(p) z^2 + z / 2 for z > 0,
    (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 for z <= 0.
    Tensors: `up` [inner, hidden], `down` [hidden, inner].
    """

    def __init__(self, hidden: int, inner: int, activation: str = "relu2") -> None:
        if activation not in ops.ACTIVATIONS:
            raise ValueError(f"dense_mlp activation {activation!r}; known: {sorted(ops.ACTIVATIONS)}")
        self.hidden, self.inner, self.activation = hidden, inner, activation

    def tensors(self) -> dict[str, TensorSpec]:
        specs = {"up": TensorSpec((self.inner, self.hidden)), "down": TensorSpec((self.hidden, self.inner))}
        if self.activation == "xielu":
            specs["act"] = TensorSpec((2,), "vector")
        return specs

    def load(self, tensors, runtime) -> None:
        super().load(tensors, runtime)
        self.up, self.down = tensors["up"].contiguous(), tensors["down"].contiguous()
        self.constants = (0.0, 0.0)
        if self.activation == "xielu":
            rise, fall = torch.nn.functional.softplus(tensors["act"].double()).tolist()
            self.constants = (rise, 0.5 + fall)

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return ops.linear(ops.linear_act(h, self.up, self.activation, self.constants), self.down)


@register_feed_forward("clamped_glu_mlp")
class ClampedGLUMLP(FeedForward):
    """down(g * sigmoid(alpha * g) * (u + 1)) with g = min(gate(h), limit) and
    u = clamp(up(h), -limit, limit); no biases.

    hidden, inner: widths; limit: the clamp; alpha: the sigmoid's slope.
    Tensors: `gate`, `up` [inner, hidden] (stacked into one operand at load), `down` [hidden, inner].
    """

    def __init__(self, hidden: int, inner: int, limit: float, alpha: float = 1.702) -> None:
        if limit <= 0:
            raise ValueError(f"clamped_glu_mlp needs a positive limit, got {limit}")
        self.hidden, self.inner, self.limit, self.alpha = hidden, inner, float(limit), float(alpha)

    def tensors(self) -> dict[str, TensorSpec]:
        return {"gate": TensorSpec((self.inner, self.hidden)), "up": TensorSpec((self.inner, self.hidden)),
                "down": TensorSpec((self.hidden, self.inner))}

    def load(self, tensors, runtime) -> None:
        super().load(tensors, runtime)
        self.gate_up = torch.cat([tensors["gate"], tensors["up"]], dim=0).contiguous()
        self.down = tensors["down"].contiguous()

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return ops.linear(ops.linear_clamped_glu(h, self.gate_up, self.alpha, self.limit), self.down)


@register_feed_forward("glu_mlp")
class GLUMLP(FeedForward):
    """down(f(gate(h)) * up(h)), no biases.

    hidden, inner: widths; activation: f, "relu" or "gelu_tanh" (the tanh form of GELU).
    Tensors: `gate`, `up` [inner, hidden] (stacked into one operand at load), `down` [hidden, inner].
    """

    takes_pending = True

    def __init__(self, hidden: int, inner: int, activation: str) -> None:
        if activation not in ops.GATED_UNITS:
            raise ValueError(f"glu_mlp activation {activation!r}; known: {sorted(ops.GATED_UNITS)}")
        self.hidden, self.inner, self.activation = hidden, inner, activation

    def tensors(self) -> dict[str, TensorSpec]:
        return {"gate": TensorSpec((self.inner, self.hidden)), "up": TensorSpec((self.inner, self.hidden)),
                "down": TensorSpec((self.hidden, self.inner))}

    def load(self, tensors, runtime) -> None:
        super().load(tensors, runtime)
        self.gate_up = torch.cat([tensors["gate"], tensors["up"]], dim=0).contiguous()
        self.down = tensors["down"].contiguous()

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return ops.linear(ops.linear_glu(h, self.gate_up, self.activation), self.down)


@register_feed_forward("relu_glu_mlp")
class ReluGLUMLP(GLUMLP):
    """`glu_mlp` with a relu."""

    takes_pending = False

    def __init__(self, hidden: int, inner: int) -> None:
        super().__init__(hidden, inner, "relu")


@register_feed_forward("table_experts")
class TableExperts(FeedForward):
    """A mixture of `experts` small clamped gated units of which every token uses `top`, chosen by
    no router: row `token id` of an integer table names the token's experts (the entries of a row
    differ), and each of them weighs 1 / top.

    hidden, inner: widths of an expert; vocab: rows of the table; limit, alpha: an expert is
    down(g sigmoid(alpha g) (u + 1)) with g = min(gate h, limit), u = clamp(up h, -limit, limit).
    Tensors: `table` [vocab, top] (integers), and per expert i `e<i>.gate`, `e<i>.up` [inner, hidden],
    `e<i>.down` [hidden, inner] (stacked at load).
    """

    def __init__(self, hidden: int, inner: int, experts: int, top: int, vocab: int, limit: float,
                 alpha: float = 1.702) -> None:
        if experts < 1 or not 1 <= top <= experts:
            raise ValueError(f"table_experts of {experts} experts, {top} a token")
        if limit <= 0:
            raise ValueError(f"table_experts needs a positive limit, got {limit}")
        self.hidden, self.inner, self.experts, self.top, self.vocab = hidden, inner, experts, top, vocab
        self.limit, self.alpha = float(limit), float(alpha)

    def tensors(self) -> dict[str, TensorSpec]:
        specs = {"table": TensorSpec((self.vocab, self.top), "table_i32")}
        for e in range(self.experts):
            specs[f"e{e}.gate"] = TensorSpec((self.inner, self.hidden))
            specs[f"e{e}.up"] = TensorSpec((self.inner, self.hidden))
            specs[f"e{e}.down"] = TensorSpec((self.hidden, self.inner))
        return specs

    def load(self, tensors, runtime) -> None:
        super().load(tensors, runtime)
        self.table = tensors["table"].contiguous()
        self.gate_up = torch.stack([torch.cat([tensors[f"e{e}.gate"], tensors[f"e{e}.up"]], dim=0)
                                    for e in range(self.experts)]).contiguous()
        self.down = torch.stack([tensors[f"e{e}.down"] for e in range(self.experts)]).contiguous()

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return ops.moe_experts(h, None, None, self.gate_up, self.down, self.top, ctx.step, table=self.table,
                               token_ids=ctx.step.token_ids, alpha=self.alpha, limit=self.limit)


@register_feed_forward("routed_experts")
class RoutedExperts(FeedForward):
    """A mixture of `experts` small gated feed-forward layers of which every token uses `top`.

    hidden, inner: widths of an expert (down(silu(gate h) * (up h)), no biases)
    experts:  experts with tensors; identity: router outputs beyond them whose expert hands its
              input back; top: choices per token
    The router's logits are taken in float32 (its matrix is kept in float32 whatever the engine's
    dtype), the scores are a softmax over all experts + identity outputs; the choice is by score +
    `correction`, the weight is the score itself, not renormalised.
    scoring:  "softmax" (above) or "sigmoid": every output's score is its own sigmoid
    weigh:    "output": y = sum of score * expert(h); "input": y = sum of expert(score * h), the chosen
              expert is given the token multiplied by its score and its output counts as it is
    shared_inner: None, or the inner width of one more gated expert (`shared.gate`, `shared.up`,
              `shared.down`) that every token uses unweighted and whose output is added
    groups, keep_groups: the outputs form `groups` equal runs of neighbours; a run's score is the sum of its two
              largest choice scores, and only outputs of the `keep_groups` best runs can be chosen
    normalise: the weights are the chosen scores divided by their sum (+ 1e-20)
    weight_scale: multiplies the weights
    scoring "chosen": the choice is by the logits, the weights are a softmax over the chosen logits only
    router_bias: the router's logits have a bias (tensor `router.b` [experts + identity])
    unit:     "swiglu" (above), or "gelu_erf": an expert is down(gelu(up h)) with the exact GELU and no gate (no
              `gate` tensors; the shared expert alike)
    shared_gate: the shared expert's output is multiplied by sigmoid(sg h), one number a token (tensor `shared.sg`
              [1, hidden], its product taken in float32 beside the router's)
    Tensors: `router` [experts + identity, hidden], `correction` [experts + identity], and per expert i
    `e<i>.gate`, `e<i>.up` [inner, hidden], `e<i>.down` [hidden, inner] (stacked at load).
    """

    def __init__(self, hidden: int, inner: int, experts: int, top: int, identity: int = 0,
                 correction: bool = True, scoring: str = "softmax", weigh: str = "output",
                 shared_inner: int | None = None, groups: int = 1, keep_groups: int = 1, normalise: bool = False,
                 weight_scale: float = 1.0, router_bias: bool = False, unit: str = "swiglu",
                 shared_gate: bool = False) -> None:
        if unit not in ("swiglu", "gelu_erf") or (shared_gate and shared_inner is None):
            raise ValueError(f"routed_experts unit {unit!r}; a shared gate needs a shared expert")
        self.router_bias, self.unit, self.shared_gate = router_bias, unit, shared_gate
        outputs = experts + identity
        if groups < 1 or outputs % groups or not 1 <= keep_groups <= groups or top > keep_groups * (outputs // groups):
            raise ValueError(f"routed_experts: {top} of {outputs} outputs in {groups} groups of which {keep_groups} are kept")
        self.groups, self.keep_groups = groups, keep_groups
        self.normalise, self.weight_scale = bool(normalise), float(weight_scale)
        if experts < 1 or identity < 0 or not 1 <= top <= experts + identity:
            raise ValueError(f"routed_experts of {experts} experts and {identity} identity ones, {top} a token")
        if scoring not in ops.ROUTER_SCORING or weigh not in ("output", "input"):
            raise ValueError(f"routed_experts scoring {scoring!r}, weigh {weigh!r}")
        self.hidden, self.inner, self.experts, self.identity, self.top = hidden, inner, experts, identity, top
        self.corrected, self.scoring, self.weigh, self.shared_inner = correction, scoring, weigh, shared_inner

    def tensors(self) -> dict[str, TensorSpec]:
        outputs = self.experts + self.identity
        specs = {"router": TensorSpec((outputs, self.hidden), "vector")}
        if self.corrected:
            specs["correction"] = TensorSpec((outputs,), "vector")
        if self.router_bias:
            specs["router.b"] = TensorSpec((outputs,), "vector")
        units = [(f"e{e}", self.inner) for e in range(self.experts)]
        if self.shared_inner is not None:
            units.append(("shared", self.shared_inner))
        for name, inner in units:
            if self.unit == "swiglu":
                specs[f"{name}.gate"] = TensorSpec((inner, self.hidden))
            specs[f"{name}.up"] = TensorSpec((inner, self.hidden))
            specs[f"{name}.down"] = TensorSpec((self.hidden, inner))
        if self.shared_gate:
            specs["shared.sg"] = TensorSpec((1, self.hidden), "vector")
        return specs

    def load(self, tensors, runtime) -> None:
        super().load(tensors, runtime)
        # The shared expert's gate is one more row of the router's matrix, behind its outputs.
        self.router = (torch.cat([tensors["router"], tensors["shared.sg"]]) if self.shared_gate else tensors["router"]).contiguous()
        self.bias = tensors["router.b"].contiguous() if self.router_bias else None
        self.correction = tensors["correction"].contiguous() if self.corrected else None

        def first(name: str) -> torch.Tensor:  # what a unit's first product runs on
            return tensors[name + ".up"] if self.unit == "gelu_erf" else torch.cat([tensors[name + ".gate"], tensors[name + ".up"]])

        self.gate_up = torch.stack([first(f"e{e}") for e in range(self.experts)]).contiguous()
        self.down = torch.stack([tensors[f"e{e}.down"] for e in range(self.experts)]).contiguous()
        self.shared_gate_up = self.shared_down = None
        if self.shared_inner is not None:
            self.shared_gate_up, self.shared_down = first("shared").contiguous(), tensors["shared.down"].contiguous()

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        extra = None
        if self.shared_gate_up is not None:
            def extra() -> torch.Tensor:
                if self.unit == "gelu_erf":
                    return ops.linear(ops.linear_act(h, self.shared_gate_up, self.unit), self.shared_down)
                return ops.linear(ops.linear_swiglu(h, self.shared_gate_up), self.shared_down)
        return self._experts(h, ctx, extra, True)

    @property
    def gives_rows(self) -> bool:
        """Whether `forward_rows` may stand in for `forward`."""
        return self.shared_inner is None and self.identity == 0 and self.weigh == "output"

    def forward_rows(self, h: torch.Tensor, ctx) -> "ops.ExpertRows":
        """The chosen experts' outputs and weights, not yet summed (a block that takes them sums them on their
        way into the residual, in float32)."""
        return self._experts(h, ctx, None, False)

    def _experts(self, h, ctx, extra, combine: bool):
        return ops.moe_experts(h, self.router, self.correction, self.gate_up, self.down, self.top, ctx.step,
                               scoring=self.scoring, weigh=self.weigh, extra=extra, groups=self.groups,
                               keep_groups=self.keep_groups, normalise=self.normalise, weight_scale=self.weight_scale,
                               combine=combine, bias=self.bias, activation=None if self.unit == "swiglu" else self.unit,
                               shared_gated=self.shared_gate)
