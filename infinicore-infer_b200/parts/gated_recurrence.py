"""A linear recurrence per channel with real gates, behind a short convolution and beside a gated branch.

    y = act(Y h + b)        u = conv(X h + b)        r = sigmoid(R u + b)        i = sigmoid(I u + b)
    log a = -rate r softplus(lam)        S <- a S + sqrt(1 - a^2) i u        output O (S y)

R and I are block-diagonal.  One fused product [y | x] into float32 rows; the convolution with the projection's bias on its way in
(its tails are state); the gates, the recurrence over each request's rows from and into its state slot, and the branch's factor
(csrc/blocks.cu: ``gated_recurrence``); the output product.  Gates, decays and state are float32 in every mode.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..cache import StateSlot
from ..weights import MATRIX, VECTOR, TensorDecl
from .base import register
from .linear_attention import LinearAttention
from .program import ACT, record


@register("mixer", "gated_recurrence")
class GatedRecurrence:
    @staticmethod
    def tensor_decls(spec) -> Dict[str, TensorDecl]:
        d, C, B, n, b = spec.hidden_size, spec.inner, spec.blocks, spec.inner // spec.blocks, spec.bias_suffix
        return {spec.y_name: TensorDecl((C, d)), spec.y_name + b: TensorDecl((C,), VECTOR, init="zeros"),
                spec.x_name: TensorDecl((C, d)), spec.x_name + b: TensorDecl((C,), VECTOR, init="zeros"),
                spec.conv_name: TensorDecl((C, spec.conv_taps), VECTOR, init="taps"), spec.conv_name + b: TensorDecl((C,), VECTOR, init="zeros"),
                spec.r_name: TensorDecl((B, n, n)), spec.r_name + b: TensorDecl((B, n), VECTOR, init="zeros"),
                spec.i_name: TensorDecl((B, n, n)), spec.i_name + b: TensorDecl((B, n), VECTOR, init="zeros"),
                spec.lam_name: TensorDecl((C,), VECTOR, init="taps"), spec.o_name: TensorDecl((d, C))}

    @staticmethod
    def cache_need(spec):
        return StateSlot((spec.inner,), "float32")

    @staticmethod
    def state_need(spec, writes_cache: bool = True):
        """The convolution's tails."""
        return StateSlot((spec.conv_taps - 1, spec.inner), "float32") if spec.conv_taps > 1 else None

    def __init__(self, spec, weights, prefix: str, runtime):
        self.spec, self.runtime = spec, runtime
        if spec.inner % spec.blocks:
            raise ValueError(f"{spec.inner} channels in {spec.blocks} equal parts")
        if spec.act not in ("none", "silu", "gelu_tanh", "sigmoid", "relu"):
            raise ValueError(f"a gated recurrence with a branch of activation {spec.act!r} is not built")
        vec = lambda name: weights.get(prefix + name, VECTOR)
        b = spec.bias_suffix
        self.w_in = weights.get_rows([prefix + spec.y_name, prefix + spec.x_name], MATRIX)
        self.y_bias, self.x_bias, self.conv, self.conv_bias = vec(spec.y_name + b), vec(spec.x_name + b), vec(spec.conv_name), vec(spec.conv_name + b)
        self.w_r, self.w_i = weights.get(prefix + spec.r_name, MATRIX), weights.get(prefix + spec.i_name, MATRIX)
        self.b_r, self.b_i = vec(spec.r_name + b), vec(spec.i_name + b)
        lam = vec(spec.lam_name).to(torch.float64)          # log a per unit of the gate r, formed once and rounded once
        self.rate = (-float(spec.rate) * torch.logaddexp(lam, torch.zeros_like(lam))).to(torch.float32).contiguous()
        self.w_o = weights.get(prefix + spec.o_name, MATRIX)

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_r, self.w_i, self.w_o))

    # the requests that run in one go and the pieces of the others: the lists of the linear attention
    LISTS = LinearAttention.LISTS
    step_list_capacity = LinearAttention.step_list_capacity
    fill_step_lists = LinearAttention.fill_step_lists

    def plan(self, program, view, writes_cache: bool = True, residual_scale: float = 1.0, state_view=None) -> None:
        """The mixer in a block that adds its output to the stream itself."""
        self.plan_delta(program, view, writes_cache, state_view=state_view, into_stream=residual_scale)

    def plan_delta(self, program, view, writes_cache: bool = True, state_view=None, into_stream=None, out_slot: str = "delta") -> None:
        """Four records: the fused product (h -> float32 rows), the convolution, the recurrence (-> o), the output product into the
        delta slot or another (``into_stream`` s: added into the stream times s)."""
        s, C = self.spec, self.spec.inner
        tail = state_view.state if state_view is not None else None
        if s.conv_taps > 1 and tail is None:
            raise ValueError("a convolution of more than one tap needs its tails' state")
        direct, pieces, piece_reqs = program.work_lists(LinearAttention, LinearAttention.LISTS)
        program.emit_records([
            record("linear", "h", "tmp", n=2 * C, k=s.hidden_size, w=self.w_in),
            record("causal_conv", "tmp", None, out2_slot="mix", n=C, ld=2 * C, q_off=C, taps=s.conv_taps, conv_q=self.conv, bias=self.conv_bias,
                   in_bias=self.x_bias, act=ACT["none"], state=tail),
            record("gated_recurrence", "mix", "o", n=C, blocks=s.blocks, ld=2 * C, g_off=0, w=self.w_r, w3=self.w_i, b1=self.b_r, b2=self.b_i,
                   decay=self.rate, bias=self.y_bias, act=ACT[s.act], state=view.state, list_short=direct, list_tiles=pieces, list_aux=piece_reqs),
            record("linear", "o", out_slot, n=s.hidden_size, k=C, w=self.w_o) if into_stream is None else
            record("residual", "o", "x", n=s.hidden_size, k=C, w=self.w_o, scale=float(into_stream)),
        ], keep=(self.w_in, self.y_bias, self.x_bias, self.conv, self.conv_bias, self.w_r, self.w_i, self.b_r, self.b_i, self.rate, self.w_o,
                 view.state, tail))

    def forward(self, h: torch.Tensor, ctx, view, writes_cache: bool = True, state_view=None) -> torch.Tensor:
        """The part alone: its own records over ``h``; float32 ``[T, hidden]``."""
        from .program import run_part_alone
        return run_part_alone(self.runtime, lambda program: self.plan_delta(program, view, writes_cache, state_view), ctx, h,
                              self.spec.hidden_size, result_slot="delta")
