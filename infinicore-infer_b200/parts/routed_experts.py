"""A feed-forward of small gated units (experts) of which each row uses a few, chosen by a router.

Scores are sigmoid(router h) in float32; a row goes to the ``top`` experts of largest score; an expert sees score * h;
the results add up without renormalising.  A shared gated unit, if the layer has one, runs for every row first (the
feed-forward's usual two records) and the experts' sum is added to it.  The rows of each expert are listed on the
device, so a step never waits for the host; the experts' products run over those lists (csrc/blocks.cu).

The other form of scores (``score_form`` "softmax_renorm"): softmax over all experts, the chosen ones' scores divided by
their sum, multiplying the units' outputs; and the other unit (``act`` "swish_clamp"): clamped sums,
g sigmoid(1.702 g) (u + 1).  The router may have a bias, and the shared unit's output a gate per row, sigmoid(w . h), which
the kernel that adds the experts' sum applies to what it adds to.

A third form ("softmax"): softmax over all router outputs, the chosen scores multiplying the units' outputs as they are; the
choice goes by score + correction, among the best groups of outputs only; outputs behind the experts' are units that return
their input (no product runs for them: the kernel that adds a row's results takes the row's own input).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..weights import MATRIX, VECTOR, TensorDecl
from .base import part_class, register
from .program import ACT, record


SCORE_FORMS = ("sigmoid", "softmax_renorm", "softmax")         # the numbers of csrc/blocks.cu


@register("feed_forward", "routed_experts")
class RoutedExperts:
    @staticmethod
    def tensor_decls(spec) -> Dict[str, TensorDecl]:
        d, f = spec.hidden_size, spec.expert_size
        n = spec.num_experts + spec.num_identity
        decls = {spec.router_name: TensorDecl((n, d), VECTOR)}
        if spec.correction_name:
            decls[spec.correction_name] = TensorDecl((n,), VECTOR, init="zeros")
        if spec.router_bias:
            decls[spec.router_name + spec.bias_suffix] = TensorDecl((n,), VECTOR, init="zeros")
        if spec.shared_gate_name:
            decls[spec.shared_prefix + spec.shared_gate_name] = TensorDecl((1, d), VECTOR)
        for e in range(spec.num_experts):
            p = spec.expert_prefix.format(e)
            decls[p + spec.gate_name] = TensorDecl((f, d))
            decls[p + spec.up_name] = TensorDecl((f, d))
            decls[p + spec.down_name] = TensorDecl((d, f))
        if spec.shared is not None:
            for name, decl in part_class("feed_forward", spec.shared).tensor_decls(spec.shared).items():
                decls[spec.shared_prefix + name] = decl
        return decls

    def __init__(self, spec, weights, prefix: str, runtime):
        self.spec, self.runtime = spec, runtime
        if spec.score_form not in SCORE_FORMS:
            raise ValueError(f"routed experts with scores of form {spec.score_form!r} are not built")
        if spec.scale_input != (spec.score_form == "sigmoid"):
            raise ValueError("built are sigmoid scores on a unit's input and softmax scores on its output")
        if spec.score_form != "softmax" and (spec.num_identity or spec.correction_name or spec.groups):
            raise ValueError("identity units, a corrected choice and groups are built for plain softmax scores")
        if spec.score_scale != 1.0 and (spec.score_form != "softmax_renorm" or not spec.score_scale > 0):
            raise ValueError("a factor of the scores is built for renormalised softmax scores, and positive")
        if spec.act == "swish_clamp" and not spec.limit > 0:
            raise ValueError("a clamped unit needs a positive limit")
        outputs = spec.num_experts + spec.num_identity
        if not 1 <= spec.top <= outputs:
            raise ValueError(f"{spec.top} of {outputs} experts")
        if spec.groups is not None:
            count, keep = spec.groups
            if outputs % count or not 1 <= keep <= count or keep * (outputs // count) < spec.top:
                raise ValueError(f"{spec.top} choices from {keep} of {count} groups of {outputs} experts")
        self.correction = weights.get(prefix + spec.correction_name, VECTOR) if spec.correction_name else None
        self.router = weights.get(prefix + spec.router_name, VECTOR)
        self.router_bias = weights.get(prefix + spec.router_name + spec.bias_suffix, VECTOR) if spec.router_bias else None
        if spec.shared_gate_name and spec.shared is None:
            raise ValueError("a gate on a shared unit that the layer does not have")
        self.shared_gate = weights.get(prefix + spec.shared_prefix + spec.shared_gate_name, VECTOR) if spec.shared_gate_name else None
        names = [prefix + spec.expert_prefix.format(e) for e in range(spec.num_experts)]
        self.w_gate_up = weights.get_rows([p + n for p in names for n in (spec.gate_name, spec.up_name)], MATRIX)
        self.w_down = weights.get_rows([p + spec.down_name for p in names], MATRIX)
        self.shared = None
        if spec.shared is not None:
            self.shared = part_class("feed_forward", spec.shared)(spec.shared, weights, prefix + spec.shared_prefix, runtime)
            if not hasattr(self.shared, "plan_delta"):
                raise TypeError(f"{type(self.shared).__name__} cannot leave its output for the experts to add to (no plan_delta)")

    def weight_bytes(self) -> int:
        """What a step of few rows reads: the router, the shared unit, ``top`` experts a row at most (here: one row's)."""
        s = self.spec
        one = (self.w_gate_up.numel() + self.w_down.numel()) * self.w_gate_up.element_size() // s.num_experts
        return 4 * self.router.numel() + s.top * one + (self.shared.weight_bytes() if self.shared is not None else 0)

    def plan(self, program, residual_scale: float = 1.0, in_slot: str = "h") -> None:
        """The feed-forward in a block that adds its output to the stream: unscaled and read from the usual slot the sum waits
        for the next norm to add it, else its own kernel adds it, times ``residual_scale``."""
        self.plan_delta(program, into_stream=1 if residual_scale == 1.0 and in_slot == "h" else 2, in_slot=in_slot, scale=residual_scale)

    def plan_delta(self, program, into_stream: int = 0, in_slot: str = "h", scale: float = 1.0) -> None:
        s = self.spec
        if self.shared is not None:
            self.shared.plan_delta(program, in_slot=in_slot)
        count, keep = s.groups or (0, 0)
        program.emit_records([
            record("experts", in_slot, "delta", n=s.hidden_size, experts=s.num_experts, top=s.top, ff=s.expert_size, vec=self.router,
                   w=self.w_gate_up, w3=self.w_down, add=self.shared is not None, act=ACT[s.act], limit=float(s.limit),
                   score_form=SCORE_FORMS.index(s.score_form), into_stream=into_stream, router_bias=self.router_bias,
                   gate_w=self.shared_gate, identity=s.num_identity, group_count=count, group_keep=keep, correction=self.correction,
                   scale=float(scale), score_scale=float(s.score_scale)),
        ], keep=(self.correction, self.router, self.w_gate_up, self.w_down, self.router_bias, self.shared_gate))

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        """The part alone: its own records over ``h``; float32 ``[T, hidden]``."""
        from .program import run_part_alone
        return run_part_alone(self.runtime, self.plan_delta, ctx, h, self.spec.hidden_size, result_slot="delta")
