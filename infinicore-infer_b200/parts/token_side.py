"""A step after a layer that brings in a vector of the row's own token:

    y = P (act(G x) * e)        x <- x + y / sqrt(mean(y^2) + eps) * w

e is a range of columns of the token's row of a table that all layers share (loaded once).  Four records: the product G on the
stream as activations (the kernel before leaves them along with the stream, where it can), the activation times e, the product P,
and the norm that adds (which the norms of the layer that follows may join).
"""
from __future__ import annotations

from typing import Dict

from ..weights import MATRIX, TensorDecl
from .base import part_class, register
from .program import ACT, record


@register("stream", "token_side")
class TokenSide:
    @staticmethod
    def tensor_decls(spec) -> Dict[str, TensorDecl]:
        out = {spec.table_name: TensorDecl((spec.vocab_size, spec.table_width)), spec.gate_name: TensorDecl((spec.dim, spec.hidden_size)),
               spec.proj_name: TensorDecl((spec.hidden_size, spec.dim))}
        out.update(part_class("norm", spec.norm).tensor_decls(spec.norm))
        return out

    def __init__(self, spec, weights, prefix: str, runtime, shared=None):
        self.spec = spec
        shared = shared if shared is not None else {}
        name = spec.table_name
        self.table = shared[name] if name in shared else shared.setdefault(name, weights.get(prefix + name, MATRIX))
        if not 0 <= spec.offset <= spec.table_width - spec.dim:
            raise ValueError(f"columns {spec.offset} .. {spec.offset + spec.dim} of a table of {spec.table_width}")
        self.w_gate, self.w_proj = weights.get(prefix + spec.gate_name, MATRIX), weights.get(prefix + spec.proj_name, MATRIX)
        self.norm = part_class("norm", spec.norm)(spec.norm, weights, prefix, runtime)

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_gate, self.w_proj)) + self.spec.dim * self.table.element_size()

    def plan(self, program) -> None:
        s = self.spec
        if not program.h_holds_stream and not program.amend_last("join", out_slot="h"):
            program.emit_records([record("cast", "x", "h", n=s.hidden_size)])
        program.emit_records([
            record("linear", "h", "tmp", n=s.dim, k=s.hidden_size, w=self.w_gate),
            record("activate", "tmp", "act", n=s.dim, ld=s.dim, act=ACT[s.act], w=self.table, k=s.table_width, g_off=s.offset),
            record("linear", "act", "delta", n=s.hidden_size, k=s.dim, w=self.w_proj),
        ], keep=(self.table, self.w_gate, self.w_proj))
        self.norm.plan_add(program)
