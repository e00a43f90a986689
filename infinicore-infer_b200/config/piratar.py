"""The Piratar configuration: a decoder whose config.json lists its layers one by one, whose mixers and feed-forwards stand side by
side and whose tokens bring a vector of their own into every layer.

Keys read: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``embedding.bigram.{buckets, mul_prev, mul_cur}`` (null for none),
``token_side.dim`` (null for none) and ``layers``, a list whose entries give ``type`` (the mixer), ``mixer`` (its sizes and constants)
and ``mlp`` (the feed-forward, or null for none).  The stream starts as the norm of scale * embed[token] + bigram[hash of the token and
the one before it]; a layer is x += mixer(norm1 x) + ff(norm2 x), both of the same x, then x += rms(P (gelu(G x) * e)) * w with e the
layer's part of the token's row of ``side.embed``.  Norms are RMS norms; those of the model store their weight around zero (the
factor is 1 + w).

    parallel           half the sum of two mixers' outputs, each RMS-normed over the width with a plain weight
      left             grouped heads behind short convolutions of q, k and v, rotate-half rotation of the leading rot.dims elements,
                       every earlier key, a sigmoid gate per output element
                                heads, kv_heads, dim, vdim, scale, conv, rot.{base, dims}
      right            retention: rotated q and k, a constant decay per head, each head divided by its root mean square, a silu gate
                                heads, dim, vdim, decay, rot.{base, dims}
    rglru              a gelu branch beside a convolved branch that runs through a real-gated linear recurrence per channel
                                width, blocks, conv
    mlp.kind dense     a gated silu unit of ff
    mlp.kind moe       router.experts gated silu units of expert.ff, router.top a row by softmax score, the chosen scores divided by
                       their sum and multiplied by router.scale; shared.ff: a unit for every row times sigmoid(sg . h)

Tensor names: ``embed``, ``bigram``, ``embed.norm``, ``side.embed``, ``head``, ``final.norm`` and below ``l<i>.``: ``norm1``, ``norm2``,
``mix.<name>`` (``mix.left.<name>``, ``mix.right.<name>``), ``mlp.<name>``, ``mlp.e<j>.<name>``, ``mlp.shared.<name>``, ``side.gate``,
``side.proj``, ``side.norm``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .specs import (ConfigError, ConvAttentionSpec, GatedRecurrenceSpec, GLUSpec, LinearAttentionSpec, ModelSpec, PairEmbeddingSpec,
                    PairRotarySpec, ParallelBlockSpec, ParallelMixerSpec, RMSNormSpec, RoutedExpertsSpec, RunEntry, TokenSideSpec)
from .vunelix import DEFAULT_MAX_POSITIONS, _need, _pos_float, _pos_int

MIXERS = ("parallel", "rglru")
RECURRENCE_RATE = 8.0       # log a = -RECURRENCE_RATE r softplus(lam)


def _check_rotation(m: dict, where: str) -> None:
    rot = m.get("rot")
    if rot is None or not int(rot.get("dims") or 0):
        return
    dims = _pos_int(rot, "dims", where + ".rot")
    if dims % 2 or dims > int(m["dim"]):
        raise ConfigError(f"config.json: {where}.rot.dims {dims} must be even and at most {m['dim']}")
    _pos_float(rot, "base", where + ".rot")


def _rotation(m: dict) -> Optional[PairRotarySpec]:
    rot = m.get("rot")
    if rot is None or not int(rot.get("dims") or 0):
        return None
    return PairRotarySpec(dims=int(rot["dims"]), base=float(rot["base"]), layout="halves")


@dataclass(frozen=True)
class PiratarConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float
    bigram: Optional[dict]
    side_dim: int                      # 0: no token vectors
    layers: Tuple[dict, ...]           # the entries of config.json's ``layers``, checked
    max_positions: int = DEFAULT_MAX_POSITIONS     # the longest sequence the engine plans for (the configuration names none)
    model_type: str = "piratar"

    # ---- reading -------------------------------------------------------------------------------------------------
    @staticmethod
    def _check_parallel(m: dict, where: str) -> None:
        left, right = dict(_need(m, "left", where)), dict(_need(m, "right", where))
        lw, rw = where + ".left", where + ".right"
        for key in ("heads", "kv_heads", "dim", "vdim", "conv"):
            _pos_int(left, key, lw)
        _pos_float(left, "scale", lw)
        if left["heads"] % left["kv_heads"]:
            raise ConfigError(f"config.json: {lw}: {left['heads']} heads are no multiple of {left['kv_heads']} key/value heads")
        for key in ("heads", "dim", "vdim"):
            _pos_int(right, key, rw)
        decay = _need(right, "decay", rw)
        if not isinstance(decay, list) or len(decay) != int(right["heads"]):
            raise ConfigError(f"config.json: {rw}.decay must list {right['heads']} numbers, one per head")
        _check_rotation(left, lw)
        _check_rotation(right, rw)

    @classmethod
    def from_dict(cls, cfg: dict, max_tokens: Optional[int] = None) -> "PiratarConfig":
        layers = _need(cfg, "layers", "the configuration")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: layers must be a list with at least one entry")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            kind, m = _need(layer, "type", where), dict(_need(layer, "mixer", where))
            if kind == "parallel":
                cls._check_parallel(m, where + ".mixer")
            elif kind == "rglru":
                width, blocks = (_pos_int(m, key, where + ".mixer") for key in ("width", "blocks"))
                _pos_int(m, "conv", where + ".mixer")
                if width % blocks:
                    raise ConfigError(f"config.json: {where}.mixer: {width} channels in {blocks} equal parts")
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is none of {', '.join(MIXERS)}")
            mlp = layer.get("mlp")
            if mlp is not None:
                mlp, mw = dict(mlp), where + ".mlp"
                form = _need(mlp, "kind", mw)
                if form == "dense":
                    _pos_int(mlp, "ff", mw)
                elif form == "moe":
                    router = _need(mlp, "router", mw)
                    n, top = (_pos_int(router, key, mw + ".router") for key in ("experts", "top"))
                    if top > n:
                        raise ConfigError(f"config.json: {mw}.router takes {top} of {n} experts")
                    if router.get("scale") is not None:
                        _pos_float(router, "scale", mw + ".router")
                    _pos_int(_need(mlp, "expert", mw), "ff", mw + ".expert")
                    if mlp.get("shared") is not None:
                        _pos_int(mlp["shared"], "ff", mw + ".shared")
                else:
                    raise ConfigError(f"config.json: {mw}.kind {form!r} is neither dense nor moe")
            checked.append({"type": kind, "mixer": m, "mlp": mlp})
        emb = cfg.get("embedding") or {}
        bigram = emb.get("bigram")
        if bigram is not None:
            _pos_int(bigram, "buckets", "embedding.bigram")
            for key in ("mul_prev", "mul_cur"):
                v = _need(bigram, key, "embedding.bigram")
                if isinstance(v, bool) or int(v) != v or not 0 <= v < 2 ** 31:
                    raise ConfigError(f"config.json: embedding.bigram.{key} must be an integer from 0 to 2^31 - 1, found {v!r}")
        side = cfg.get("token_side")
        scale = emb.get("scale")
        return cls(vocab=_pos_int(cfg, "vocab", "the configuration"), width=_pos_int(cfg, "width", "the configuration"),
                   norm_eps=float(_need(_need(cfg, "norm", "the configuration"), "eps", "norm")), embed_scale=1.0 if scale is None else float(scale),
                   bigram=None if bigram is None else dict(bigram), side_dim=0 if side is None else _pos_int(side, "dim", "token_side"),
                   layers=tuple(checked), max_positions=int(max_tokens) if max_tokens else int(cfg.get("max_positions", DEFAULT_MAX_POSITIONS)))

    # what the entry points ask of any configuration
    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    @property
    def tie_word_embeddings(self) -> bool:
        return False

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def to_dict(self) -> dict:
        """config.json contents that read back to this configuration."""
        return {"architecture": "Piratar", "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embed_scale, "bigram": None if self.bigram is None else dict(self.bigram)},
                "token_side": {"dim": self.side_dim} if self.side_dim else None,
                "layers": [{"type": l["type"], "mixer": dict(l["mixer"]), "mlp": None if l["mlp"] is None else dict(l["mlp"])}
                           for l in self.layers]}

    # ---- the model as parts ------------------------------------------------------------------------------------------
    def _mixer_spec(self, kind: str, m: dict):
        if kind == "rglru":
            return GatedRecurrenceSpec(hidden_size=self.width, inner=int(m["width"]), blocks=int(m["blocks"]), conv_taps=int(m["conv"]),
                                       rate=RECURRENCE_RATE)
        left, right = m["left"], m["right"]
        attention = ConvAttentionSpec(hidden_size=self.width, num_heads=int(left["heads"]), num_kv_heads=int(left["kv_heads"]), head_dim=int(left["dim"]),
                                      v_head_dim=int(left["vdim"]), softmax_scale=float(left["scale"]), conv_taps=int(left["conv"]),
                                      position=_rotation(left), element_gate=True)
        # k's factor dim^(-1/2) rides on q: a row's output is linear in the product of both
        retention = LinearAttentionSpec(hidden_size=self.width, num_heads=int(right["heads"]), head_dim=int(right["dim"]), v_head_dim=int(right["vdim"]),
                                        norm_eps=self.norm_eps, decay=tuple(float(d) for d in right["decay"]), q_scale=int(right["dim"]) ** -0.5,
                                        norm_per_head=True, norm_name=None, gate_act="silu", position=_rotation(right))
        out = RMSNormSpec(size=self.width, eps=self.norm_eps, weight_name="out")
        return ParallelMixerSpec(left=attention, right=retention, left_scale=0.5, right_scale=0.5, left_norm=out, right_norm=out)

    def _ffn_spec(self, mlp: Optional[dict]):
        if mlp is None:
            return None
        unit = lambda ff: GLUSpec(hidden_size=self.width, intermediate_size=int(ff), act="silu")
        if mlp["kind"] == "dense":
            return unit(mlp["ff"])
        router, shared = mlp["router"], mlp.get("shared")
        scale = router.get("scale")
        return RoutedExpertsSpec(hidden_size=self.width, num_experts=int(router["experts"]), top=int(router["top"]), expert_size=int(mlp["expert"]["ff"]),
                                 act="silu", scale_input=False, score_form="softmax_renorm", score_scale=1.0 if scale is None else float(scale),
                                 shared=None if shared is None else unit(shared["ff"]), shared_gate_name=None if shared is None else "sg")

    def _side_spec(self, i: int):
        if not self.side_dim:
            return None
        p = f"l{i}.side."
        return TokenSideSpec(hidden_size=self.width, vocab_size=self.vocab, dim=self.side_dim, table_width=self.side_dim * len(self.layers),
                             offset=self.side_dim * i, norm=RMSNormSpec(size=self.width, eps=self.norm_eps, weight_name=p + "norm"),
                             gate_name=p + "gate", proj_name=p + "proj")

    def model_spec(self) -> ModelSpec:
        norm = RMSNormSpec(size=self.width, eps=self.norm_eps, weight_name="", one_plus=True)
        blocks, order = [], []
        for i, layer in enumerate(self.layers):
            ffn = self._ffn_spec(layer["mlp"])
            blocks.append(ParallelBlockSpec(mixer=self._mixer_spec(layer["type"], layer["mixer"]), feed_forward=ffn, mixer_norm=norm,
                                            ffn_norm=None if ffn is None else norm, joined=True))
            order.append(RunEntry(layer=i, cache=i, after=self._side_spec(i)))
        b = self.bigram
        pairs = None if b is None else PairEmbeddingSpec(buckets=int(b["buckets"]), mul_prev=int(b["mul_prev"]), mul_cur=int(b["mul_cur"]))
        return ModelSpec(architecture="piratar", hidden_size=self.width, vocab_size=self.vocab, max_positions=self.max_positions,
                         layers=tuple(blocks), order=tuple(order), final_norm=norm, embed_scale=self.embed_scale, logit_scale=1.0,
                         pairs=pairs, embed_norm=norm, embed_norm_prefix="embed.norm", tie_embeddings=False, embed_name="embed",
                         lm_head_name="head", final_norm_prefix="final.norm", layer_prefix="l{}.", eos_token_ids=())
