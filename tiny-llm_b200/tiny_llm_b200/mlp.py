"""Gated feed-forward layers with unquantised weights: ``down(act(gate x) * (up x))``.

``GatedMLP`` is the dense form (gate and up stacked into one product, the activation fused with the gating product in
one launch); ``TopKRouter`` + ``MixtureOfExperts`` the sparse one: router logits in fp32, the ``top`` largest chosen,
weights either a softmax over the chosen logits or each chosen logit's sigmoid as it is, the chosen experts' outputs
summed with those weights (or, ``weight_on="input"``, each expert run on its weight times the token), optionally plus
a shared expert that every token takes (as it is, or times a sigmoid of a projection of the token).  The choice may be
limited to the best ``groups`` of neighbouring experts.  Experts are gated or, without ``w_gate``, plain ``down(act(up x))``.  The expert products are grouped GEMMs of the blocks library over a device-built
list of (token, choice) pairs sorted by expert: no host synchronisation, and a token's result does not depend on the
rest of the batch."""

from __future__ import annotations

import torch

from .basics import linear, linear_wide

ACTIVATIONS = {"silu": 0, "gelu_tanh": 1, "relu_squared": 2, "clamped_swish": 3}
SCORINGS = {"softmax": 0, "sigmoid": 1, "softmax_all": 2}


class DenseMLP:
    """The ungated feed-forward ``down(act(up x))``; the down projection hands its fp32 accumulator on."""

    def __init__(self, w_up: torch.Tensor, w_down: torch.Tensor, act: str):
        self.w_up, self.w_down, self.act = w_up.contiguous(), w_down.contiguous(), ACTIVATIONS[act]

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        from extensions_b200.tiny_llm_ext_b200 import blocks

        return linear_wide(blocks.act_rows(linear(h, self.w_up), self.act), self.w_down)


class GatedMLP:
    """``act="clamped_swish"`` (with ``limit`` and ``slope``): ``g = min(gate x, limit)``, ``u = clamp(up x, -limit, limit)``,
    ``down(g sigmoid(slope g) (u + 1))``.  ``b_gate`` / ``b_up`` are added by the first product; ``b_down`` is kept for the
    caller (``down_bias``), who adds it where the residual sum is made."""

    def __init__(self, w_gate: torch.Tensor, w_up: torch.Tensor, w_down: torch.Tensor, act: str, b_gate=None, b_up=None, b_down=None,
                 limit: float = 0.0, slope: float = 1.0):
        self.w_gate_up = torch.cat([w_gate, w_up], dim=0).contiguous()  # [2 ff, D]: one product for both
        self.w_down = w_down.contiguous()
        self.act = ACTIVATIONS[act]
        if (b_gate is None) != (b_up is None):
            raise ValueError("gated feed-forward: biases on both first projections or on neither")
        self.b_gate_up = None if b_gate is None else torch.cat([b_gate, b_up]).contiguous()
        self.down_bias = None if b_down is None else b_down.contiguous()
        self.limit, self.slope = float(limit), float(slope)
        if act == "clamped_swish" and not self.limit > 0:
            raise ValueError("gated feed-forward: the clamped activation needs a positive limit")

    def inner(self, h: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
        """``act(gate h) * (up h)``, the down projection's operand; ``out``: the columns of a wider matrix it goes to."""
        from extensions_b200.tiny_llm_ext_b200 import blocks

        first = linear(h, self.w_gate_up) if self.b_gate_up is None else torch.addmm(self.b_gate_up, h, self.w_gate_up.t())
        return blocks.gated_act(first, self.act, self.limit, self.slope, out)

    def __call__(self, h: torch.Tensor, wide: bool = False) -> torch.Tensor:
        """``wide``: hand the down projection's fp32 accumulator back unrounded (when a norm reads it next)."""
        return (linear_wide if wide else linear)(self.inner(h), self.w_down)


class TopKRouter:
    def __init__(self, weight: torch.Tensor, bias: torch.Tensor | None, top: int, scoring: str = "softmax", choice_bias: torch.Tensor | None = None,
                 weight_scale: float = 1.0, groups: tuple | None = None):
        """``scoring="softmax_all"``: scores are a softmax over ALL router outputs, the ``top`` are chosen by score +
        ``choice_bias`` (which the weights do not see), the chosen scores are renormalised and times ``weight_scale``.
        ``groups`` = (count, keep): the outputs form ``count`` equal runs of neighbours, and a token chooses among the ``keep`` runs
        whose best choice score is largest."""
        self.weight, self.bias, self.top = weight.contiguous(), None if bias is None else bias.contiguous(), int(top)
        self.scoring = SCORINGS[scoring]
        self.choice_bias, self.weight_scale = None if choice_bias is None else choice_bias.contiguous(), float(weight_scale)
        if (choice_bias is not None or self.weight_scale != 1.0) and scoring != "softmax_all":
            raise ValueError("router: a choice bias and a weight scale go with scoring='softmax_all'")
        if not 0 < self.top <= weight.shape[0]:
            raise ValueError(f"router: top={top} of {weight.shape[0]} experts")
        self.groups = (0, 0) if groups is None else (int(groups[0]), int(groups[1]))
        count, keep = self.groups
        if groups is not None and (count <= 0 or weight.shape[0] % count or not 0 < keep <= count or keep * (weight.shape[0] // count) < self.top):
            raise ValueError(f"router: {keep} of {count} groups of {weight.shape[0]} outputs cannot give {top} choices")

    def __call__(self, h: torch.Tensor, side_w: torch.Tensor | None = None):
        """-> (expert ids int32 [T, top], weights fp32 [T, top]), and with ``side_w [1, D]`` also ``sigmoid(side_w . h)`` fp32 [T]."""
        from extensions_b200.tiny_llm_ext_b200 import blocks

        return blocks.moe_route(h, self.weight, self.bias, self.top, self.scoring, self.choice_bias, self.weight_scale, self.groups, side_w)


class MixtureOfExperts:
    def __init__(self, router: TopKRouter, w_gate: torch.Tensor | None, w_up: torch.Tensor, w_down: torch.Tensor, act: str,
                 shared: GatedMLP | None = None, weight_on: str = "output", identity: int = 0, limit: float = 0.0, slope: float = 1.0,
                 shared_gate: torch.Tensor | None = None):
        """``w_gate, w_up [E, ff, D]``, ``w_down [E, D, ff]`` (the experts stacked); ``w_gate`` None = experts without a gate.
        ``identity``: the router's last ``identity`` outputs are experts without weights whose output is their input.
        ``limit``, ``slope``: of ``act="clamped_swish"`` (see ``GatedMLP``); ``shared_gate [1, D]``: the shared expert's output is
        multiplied by ``sigmoid(shared_gate . x)``."""
        if weight_on not in ("output", "input"):
            raise ValueError(f"weight_on={weight_on!r}")
        self.identity = int(identity)
        if self.identity < 0 or router.weight.shape[0] != w_up.shape[0] + self.identity:
            raise ValueError(f"router outputs ({router.weight.shape[0]}) != experts ({w_up.shape[0]}) + identity experts ({identity})")
        if self.identity and weight_on == "input":
            raise ValueError("identity experts take the router's weight on their output")
        self.router, self.shared, self.scale_input = router, shared, weight_on == "input"
        self.w_gate, self.w_up, self.w_down = None if w_gate is None else w_gate.contiguous(), w_up.contiguous(), w_down.contiguous()
        self.act, self.limit, self.slope = ACTIVATIONS[act], float(limit), float(slope)
        if act == "clamped_swish" and (not self.limit > 0 or w_gate is None):
            raise ValueError("mixture of experts: the clamped activation needs gated experts and a positive limit")
        if shared_gate is not None and (shared is None or shared_gate.numel() != w_up.shape[2]):
            raise ValueError("mixture of experts: a shared gate of [1, width] goes with a shared expert")
        self.shared_gate = None if shared_gate is None else shared_gate.contiguous()

    def __call__(self, h: torch.Tensor, into: tuple | None = None, beside=None) -> torch.Tensor:
        """-> fp32 [T, D], or (``into`` = (stream, post norm, next norm)) the fused end of the sublayer, see ``blocks.moe_experts``.
        ``beside``: a model whose second stream runs the shared expert while this one routes (``RaggedDecoderModel._beside``)."""
        from extensions_b200.tiny_llm_ext_b200 import blocks

        shared = side = None
        if beside is not None and self.shared is not None:
            shared = torch.empty_like(h)
            with beside._beside():
                torch.mm(self.shared.inner(h), self.shared.w_down.t(), out=shared)
        elif self.shared is not None:
            shared = self.shared(h)
        if self.shared_gate is None:
            idx, gate = self.router(h)
        else:
            idx, gate, side = self.router(h, self.shared_gate)
        join = beside._join if beside is not None and self.shared is not None else None
        return blocks.moe_experts(h, idx, gate, self.w_gate, self.w_up, self.w_down, self.act, shared, scale_input=self.scale_input, identity=self.identity > 0,
                                  limit=self.limit, slope=self.slope, shared_gate=side, into=into, before_sum=join)
