"""The Fupapel configuration: a decoder whose config.json lists its layers one by one and whose mixers and feed-forwards stand
side by side.

Keys read: ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` and ``layers``, a list whose entries give ``type`` (the mixer),
``mixer`` (its sizes and constants) and ``mlp`` (the feed-forward, or null for none).  Every layer is
x += residual_mult (mixer(shift(norm1(x))) + ff(norm2(x))), both sides of the same x, with RMS norms whose weights are stored
around zero (the factor is 1 + w) and the shift h_t + (h_(t-1) - h_t) * l<i>.shift; the model ends with such a norm and an
output matrix of its own.

    attention          grouped heads, an RMS norm over the whole q and the whole k, rotate-half rotation of the leading
                       rot.dims elements, keys of the query's own chunk of mask.size positions only, a softmax with one more
                       in its denominator, a sigmoid gate per output element
                                heads, kv_heads, dim, vdim, scale, mask.size, rot.{base, dims}
    attention_2        the same norms, rotation (stretched frequencies) and mask behind short convolutions of q, k and v; a
                       factor per head on the scores, a learned sink per head; kv_from: the keys and values of that layer
                                heads, kv_heads, dim, vdim, scale, conv, mask.size, rot.{base, dims, scaling.{factor, low, high,
                                original}}, kv_from
    latent_attention   queries through a normed latent, keys and values from one normed latent per position beside a rotated
                       key part for all heads; a learned sink and a sigmoid gate per head
                                heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot.{base, dims}
    mlp.kind moe       router.experts gated units (silu) of expert.ff and router.identity outputs that return their input,
                       router.top a row by softmax score + correction among the best groups (groups.{count, keep}), weighed by
                       the scores as they are

Tensor names: ``embed``, ``head``, ``final.norm`` and below ``l<i>.``: ``norm1``, ``norm2``, ``shift``, ``mix.<name>``,
``mlp.router``, ``mlp.correction``, ``mlp.e<j>.gate / up / down``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .specs import (ConfigError, ConvAttentionSpec, FrequencyBandSpec, LatentAttentionSpec, ModelSpec, PairRotarySpec, ParallelBlockSpec,
                    RMSNormSpec, RoutedExpertsSpec, RunEntry)
from .vunelix import DEFAULT_MAX_POSITIONS, _need, _pos_float, _pos_int

MIXERS = ("attention", "attention_2", "latent_attention")


@dataclass(frozen=True)
class FupapelConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[dict, ...]           # the entries of config.json's ``layers``, checked
    max_positions: int = DEFAULT_MAX_POSITIONS     # the longest sequence the engine plans for (the configuration names none)
    model_type: str = "fupapel"

    # ---- reading -------------------------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, cfg: dict, max_tokens: Optional[int] = None) -> "FupapelConfig":
        layers = _need(cfg, "layers", "the configuration")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: layers must be a list with at least one entry")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            m = dict(_need(layer, "mixer", where))
            mw = where + ".mixer"
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is none of {', '.join(MIXERS)}")
            for key in ("heads", "dim", "vdim") + (("rot_dim", "kv_rank", "q_rank") if kind == "latent_attention" else ("kv_heads",)):
                _pos_int(m, key, mw)
            _pos_float(m, "scale", mw)
            if kind != "latent_attention":
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"config.json: {mw}: {m['heads']} heads are no multiple of {m['kv_heads']} key/value heads")
                if m.get("mask") is not None:
                    _pos_int(m["mask"], "size", mw + ".mask")
            if kind == "attention_2":
                _pos_int(m, "conv", mw)
            rot = m.get("rot")
            if rot is not None and int(rot.get("dims") or 0):
                dims, room = _pos_int(rot, "dims", mw + ".rot"), m["rot_dim"] if kind == "latent_attention" else m["dim"]
                if dims % 2 or dims > room:
                    raise ConfigError(f"config.json: {mw}.rot.dims {dims} must be even and at most {room}")
                _pos_float(rot, "base", mw + ".rot")
                if rot.get("scaling") is not None:
                    for key in ("factor", "low", "high", "original"):
                        _pos_float(rot["scaling"], key, mw + ".rot.scaling")
            if m.get("kv_from") is not None:
                source = int(m["kv_from"])
                if not 0 <= source < i or checked[source]["type"] != kind or kind == "latent_attention":
                    raise ConfigError(f"config.json: {mw}.kv_from {source} is no earlier layer of type {kind} with keys of its own")
                src = checked[source]["mixer"]
                if src.get("kv_from") is not None:
                    raise ConfigError(f"config.json: {mw}.kv_from {source} borrows its keys itself")
                for key in ("kv_heads", "dim", "vdim"):
                    if int(src[key]) != int(m[key]):
                        raise ConfigError(f"config.json: {mw}.kv_from {source}: {key} {src[key]} there, {m[key]} here")
            mlp = layer.get("mlp")
            if mlp is not None:
                mlp = dict(mlp)
                form = _need(mlp, "kind", where + ".mlp")
                if form != "moe":
                    raise ConfigError(f"config.json: {where}.mlp.kind {form!r} is not moe")
                router, rw = _need(mlp, "router", where + ".mlp"), where + ".mlp.router"
                n, top = _pos_int(router, "experts", rw) + int(router.get("identity") or 0), _pos_int(router, "top", rw)
                groups = router.get("groups")
                reach = n
                if groups is not None:
                    count, keep = _pos_int(groups, "count", rw + ".groups"), _pos_int(groups, "keep", rw + ".groups")
                    if n % count or keep > count:
                        raise ConfigError(f"config.json: {rw}: {keep} of {count} groups of {n} experts")
                    reach = keep * (n // count)
                if top > reach:
                    raise ConfigError(f"config.json: {rw} takes {top} of {reach} experts")
                _pos_int(_need(mlp, "expert", where + ".mlp"), "ff", where + ".mlp.expert")
            checked.append({"type": kind, "mixer": m, "mlp": mlp})
        mult = cfg.get("residual_mult")
        return cls(vocab=_pos_int(cfg, "vocab", "the configuration"), width=_pos_int(cfg, "width", "the configuration"),
                   norm_eps=float(_need(_need(cfg, "norm", "the configuration"), "eps", "norm")), residual_mult=1.0 if mult is None else float(mult),
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
        return {"architecture": "Fupapel", "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width,
                "residual_mult": self.residual_mult,
                "layers": [{"type": l["type"], "mixer": dict(l["mixer"]), "mlp": None if l["mlp"] is None else dict(l["mlp"])}
                           for l in self.layers]}

    # ---- the model as parts ------------------------------------------------------------------------------------------
    @staticmethod
    def _rotation(m: dict) -> Optional[PairRotarySpec]:
        rot = m.get("rot")
        if rot is None or not int(rot.get("dims") or 0):
            return None
        s, scaling = rot.get("scaling"), None
        if s is not None:
            scaling = FrequencyBandSpec(factor=float(s["factor"]), original=float(s["original"]), low=float(s["low"]), high=float(s["high"]))
        return PairRotarySpec(dims=int(rot["dims"]), base=float(rot["base"]), scaling=scaling, layout="halves")

    def _mixer_spec(self, kind: str, m: dict):
        common = dict(hidden_size=self.width, num_heads=int(m["heads"]), head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]),
                      softmax_scale=float(m["scale"]), position=self._rotation(m))
        if kind == "latent_attention":
            return LatentAttentionSpec(rot_dim=int(m["rot_dim"]), latent_size=int(m["kv_rank"]), q_rank=int(m["q_rank"]), norm_eps=self.norm_eps,
                                       output_gate="head", sink_name="sink", **common)
        mask = m.get("mask") or {}
        chunk = int(mask["size"]) if mask.get("size") is not None else None
        common.update(num_kv_heads=int(m["kv_heads"]), qk_norm=True, qk_norm_eps=self.norm_eps, chunk=chunk, sink=True,
                      shares_kv=m.get("kv_from") is not None)
        if kind == "attention":
            return ConvAttentionSpec(conv_taps=0, element_gate=True, **common)
        return ConvAttentionSpec(conv_taps=int(m["conv"]), temp_name="temp", sink_name="sink", **common)

    def _ffn_spec(self, mlp: Optional[dict]):
        if mlp is None:
            return None
        router = mlp["router"]
        groups = router.get("groups")
        return RoutedExpertsSpec(hidden_size=self.width, num_experts=int(router["experts"]), num_identity=int(router.get("identity") or 0),
                                 top=int(router["top"]), expert_size=int(mlp["expert"]["ff"]), act="silu", scale_input=False,
                                 score_form="softmax", correction_name="correction",
                                 groups=None if groups is None else (int(groups["count"]), int(groups["keep"])))

    def model_spec(self) -> ModelSpec:
        norm = RMSNormSpec(size=self.width, eps=self.norm_eps, weight_name="", one_plus=True)
        blocks, order = [], []
        for i, layer in enumerate(self.layers):
            ffn, source = self._ffn_spec(layer["mlp"]), layer["mixer"].get("kv_from")
            blocks.append(ParallelBlockSpec(mixer=self._mixer_spec(layer["type"], layer["mixer"]), feed_forward=ffn, mixer_norm=norm,
                                            ffn_norm=None if ffn is None else norm, residual_scale=self.residual_mult, shift_name="shift"))
            order.append(RunEntry(layer=i, cache=i if source is None else int(source), writes_cache=source is None))
        return ModelSpec(architecture="fupapel", hidden_size=self.width, vocab_size=self.vocab, max_positions=self.max_positions,
                         layers=tuple(blocks), order=tuple(order), final_norm=norm, embed_scale=1.0, logit_scale=1.0,
                         tie_embeddings=False, embed_name="embed", lm_head_name="head", final_norm_prefix="final.norm",
                         layer_prefix="l{}.", eos_token_ids=())
