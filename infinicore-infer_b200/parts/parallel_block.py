"""The block whose sublayers stand side by side: x += s * (mixer(shift(norm_a(x))) + feed_forward(norm_b(x))).

Both norms read the stream as the layer found it, so one kernel makes both (``norm_pair``: the row and its mean square
once), the first mixed with the row before it where the block has a token shift; the mixer reads its usual slot, the
feed-forward a second one.  The mixer's output product then adds into the stream (or waits for it), and the feed-forward
adds after it.  The row that the shift needs from the step before is kept per request in float32 (as two rows that take
turns: a step reads one and leaves the other), beside whatever the mixer keeps.

``joined``: the mixer's output (or those of its sides, each with a norm) and the feed-forward's wait in slots of their own, and one
``join`` record adds them all.  Without a shift both norms join the record before, where that is a norm that adds to the stream.
"""
from __future__ import annotations

import inspect
from typing import Dict

from ..cache import StateSlot, StateSlots
from ..kernels import norm_pair_kept_floats
from ..weights import VECTOR, TensorDecl
from .base import part_class, register
from .program import record


@register("block", "parallel_block")
class ParallelBlock:
    @staticmethod
    def tensor_decls(spec) -> Dict[str, TensorDecl]:
        out = {}
        for sub, prefix, family in _children(spec):
            for name, decl in part_class(family, sub).tensor_decls(sub).items():
                out[prefix + name] = decl
        if spec.shift_name:
            out[spec.shift_name] = TensorDecl((spec.mixer_norm.size,), VECTOR, init="half")
        return out

    @staticmethod
    def cache_need(spec):
        return part_class("mixer", spec.mixer).cache_need(spec.mixer)

    @staticmethod
    def _mixer_state(spec, writes_cache: bool = True):
        ask = getattr(part_class("mixer", spec.mixer), "state_need", None)
        return ask(spec.mixer, writes_cache) if ask is not None else None

    @staticmethod
    def state_need(spec, writes_cache: bool = True):
        """The first norm's last row where there is a shift, then what the mixer keeps beside its cache (one state, or the
        several of a ``StateSlots``)."""
        mixer = ParallelBlock._mixer_state(spec, writes_cache)
        if not spec.shift_name:
            return mixer
        own = (StateSlot((2, norm_pair_kept_floats(spec.mixer_norm.size)), "float32"),)
        return StateSlots(own + (() if mixer is None else mixer.slots if isinstance(mixer, StateSlots) else (mixer,)))

    def __init__(self, spec, weights, prefix: str, runtime):
        self.spec = spec
        build = lambda family, sub, p: part_class(family, sub)(sub, weights, prefix + p, runtime)
        self.mixer_norm = build("norm", spec.mixer_norm, spec.mixer_norm_prefix)
        self.shift = weights.get(prefix + spec.shift_name, VECTOR) if spec.shift_name else None
        self.mixer = build("mixer", spec.mixer, spec.mixer_prefix)
        self.ffn_norm = self.feed_forward = None
        if spec.feed_forward is not None:
            self.ffn_norm = build("norm", spec.ffn_norm, spec.ffn_norm_prefix)
            self.feed_forward = build("feed_forward", spec.feed_forward, spec.ffn_prefix)
            if "in_slot" not in inspect.signature(getattr(self.feed_forward, "plan", lambda: None)).parameters:
                raise TypeError(f"{type(self.feed_forward).__name__} cannot read a slot of its own beside the mixer's (no plan with in_slot)")
        if not hasattr(self.mixer, "plan"):
            raise TypeError(f"{type(self.mixer).__name__} cannot add its output into the stream (no plan)")
        if spec.joined and spec.residual_scale != 1.0:
            raise ValueError("joined sublayers with a residual factor are not built")
        for norm in (self.mixer_norm, self.ffn_norm):
            if norm is not None and getattr(norm.spec, "kind", None) != "rmsnorm":
                raise TypeError(f"a pair of norms is built of RMS norms, not of {type(norm).__name__}")

    def weight_bytes(self) -> int:
        parts = (self.mixer_norm, self.mixer, self.ffn_norm, self.feed_forward)
        return sum(p.weight_bytes() for p in parts if p is not None and hasattr(p, "weight_bytes"))

    def plan(self, program, view, writes_cache: bool = True, state_view=None) -> None:
        s, first, second = self.spec, self.mixer_norm, self.ffn_norm
        kept = mixer_state = None
        if s.shift_name:
            mine = self._mixer_state(s, writes_cache)
            count = 1 + (0 if mine is None else len(mine.slots) if isinstance(mine, StateSlots) else 1)
            if state_view is None or len(state_view) != count:
                raise ValueError("a block with a token shift needs the views of all of its state")
            kept = state_view[0].state
            if mine is not None:
                mixer_state = state_view.rest(1) if isinstance(mine, StateSlots) else state_view[1]
        else:
            mixer_state = state_view
        if s.shift_name or not first.plan_pair_after_add(program, second):
            self._plan_norms(program, first, second, kept)
        if s.joined:
            self._plan_joined(program, view, writes_cache, mixer_state)
            return
        if mixer_state is not None or hasattr(type(self.mixer), "state_need"):
            self.mixer.plan(program, view, writes_cache, s.residual_scale, state_view=mixer_state)
        else:
            self.mixer.plan(program, view, writes_cache, s.residual_scale)
        if self.feed_forward is not None:
            self.feed_forward.plan(program, s.residual_scale, in_slot="h2")

    def _plan_norms(self, program, first, second, kept) -> None:
        program.emit_records([
            record("norm_pair", "x", "h", out2_slot="h2" if second is not None else None, n=first.spec.size, vec=first.weight, eps=first.spec.eps,
                   vec2=second.weight if second is not None else None, eps2=second.spec.eps if second is not None else 0.0,
                   bias=self.shift, state=kept),
        ], keep=(first.weight, second.weight if second is not None else None, self.shift, kept))

    def _plan_joined(self, program, view, writes_cache: bool, mixer_state) -> None:
        extra = {"state_view": mixer_state} if mixer_state is not None or hasattr(type(self.mixer), "state_need") else {}
        parts = self.mixer.plan_parts(program, view, writes_cache, **extra) if hasattr(self.mixer, "plan_parts") else None
        if parts is None:
            self.mixer.plan_delta(program, view, writes_cache, out_slot="part1", **extra)
            parts = [("part1", None, 0.0)]
        if self.feed_forward is not None:
            self.feed_forward.plan_delta(program, in_slot="h2")
        (a, wa, ea), (b, wb, eb) = (parts + [(None, None, 0.0)])[:2]
        program.emit_records([record("join", a, None, in2_slot=b, n=self.mixer_norm.spec.size, vec=wa, eps=ea, vec2=wb, eps2=eb,
                                     add=self.feed_forward is not None)], keep=(wa, wb))


def _children(spec):
    out = [(spec.mixer_norm, spec.mixer_norm_prefix, "norm"), (spec.mixer, spec.mixer_prefix, "mixer")]
    if spec.feed_forward is not None:
        out += [(spec.ffn_norm, spec.ffn_norm_prefix, "norm"), (spec.feed_forward, spec.ffn_prefix, "feed_forward")]
    return out
