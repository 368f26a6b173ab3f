"""Typed configuration of Lovapel, a small decoder whose layers norm both sides of every branch with layer norms without
biases and mix tokens with grouped-query attention over a sliding window: queries and keys normed over the whole
projection, rotated in halves, a sink in the softmax.  Feed-forwards are dense layers gated by the tanh form of GELU, or
mixtures of small SiLU-gated experts behind a softmax router that chooses inside its best groups, with identity experts
among them and a shared expert beside them.  A span of the layers may run several times in a row with the same weights.
Logits come from the embedding table and are scaled and softly capped.

config.json keys (every size and every constant that differs between models of the design comes from here):

  architecture      "Lovapel"
  vocab, width      vocabulary and width of the residual stream
  norm.eps          eps of every norm (the layers' and those of queries and keys)
  logit_scale       what the logits are multiplied by (absent: 1), logit_softcap the cap c of c tanh(z / c) (absent: none)
  layers[i]         {"type": "attention", "mixer": {...}, "mlp": {...} | null}
    attention       {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"} | absent, "rot": {"dims", "base"} | absent}
    mlp             {"kind": "dense", "ff"}  or
                    {"kind": "moe", "expert": {"ff"}, "shared": {"ff"} | absent,
                     "router": {"experts", "top", "identity" | absent, "groups": {"count", "keep"} | absent}}
  loop              {"start", "stop", "times"} | absent: layers start .. stop-1 run `times` times in a row, each pass with
                    a cache of its own

Tensor names: `embed`, `final.norm`, and per layer `l<i>.norm1`, `l<i>.norm1b`, `l<i>.norm2`, `l<i>.norm2b`,
`l<i>.mix.q|k|v|o|sink|q.norm|k.norm`, `l<i>.mlp.gate|up|down` or `l<i>.mlp.router|correction`,
`l<i>.mlp.e<j>.gate|up|down`, `l<i>.mlp.shared.gate|up|down`."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .dunelix import DEFAULT_MAX_POSITIONS, _need, _number, _pos_int
from .errors import ConfigError
from .registry import register_architecture
from .spec import LayerCall, LayerSpec, ModelSpec, PartSpec

MIXERS = ("attention",)


def _check_attention(m: dict, where: str) -> None:
    heads, kv = _pos_int(m, "heads", where), _pos_int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f'config.json: {where}: "heads" ({heads}) must be a multiple of "kv_heads" ({kv})')
    _pos_int(m, "dim", where)
    _pos_int(m, "vdim", where)
    _number(m, "scale", where)
    if m.get("mask") is not None:
        _pos_int(m["mask"], "size", where + ".mask")
    rot = m.get("rot")
    if rot is not None:
        dims = _pos_int(rot, "dims", where + ".rot")
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f'config.json: {where}.rot: "dims" ({dims}) must be even and at most "dim" ({m["dim"]})')
        if _number(rot, "base", where + ".rot") <= 0:
            raise ConfigError(f'config.json: {where}.rot: "base" must be positive')


def _check_mlp(mlp: dict, where: str) -> None:
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        _pos_int(mlp, "ff", where)
        return
    if kind != "moe":
        raise ConfigError(f'config.json: {where}: unknown kind {kind!r} (known: dense, moe)')
    _pos_int(_need(mlp, "expert", where), "ff", where + ".expert")
    if mlp.get("shared") is not None:
        _pos_int(mlp["shared"], "ff", where + ".shared")
    r, at = _need(mlp, "router", where), where + ".router"
    n, top = _pos_int(r, "experts", at), _pos_int(r, "top", at)
    identity = r.get("identity") or 0
    if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
        raise ConfigError(f'config.json: {at}: "identity" must be a count of experts, found {r["identity"]!r}')
    groups = r.get("groups")
    count = keep = 1
    if groups is not None:
        count, keep = _pos_int(groups, "count", at + ".groups"), _pos_int(groups, "keep", at + ".groups")
    if (n + identity) % count:
        raise ConfigError(f'config.json: {at}.groups: "count" ({count}) must divide the {n + identity} experts')
    if keep > count:
        raise ConfigError(f'config.json: {at}.groups: "keep" ({keep}) exceeds "count" ({count})')
    if top > keep * ((n + identity) // count):
        raise ConfigError(f'config.json: {at}: "top" ({top}) exceeds the experts that stand for choice')


@dataclass(frozen=True)
class LovapelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[Dict[str, Any], ...]
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None
    loop: Optional[Tuple[int, int, int]] = None   # (start, stop, times)
    eos_token_ids: Tuple[int, ...] = ()
    initializer_range: float = 0.06

    architecture = "Lovapel"

    @classmethod
    def from_dict(cls, d: dict) -> "LovapelConfig":
        vocab, width = _pos_int(d, "vocab", "top level"), _pos_int(d, "width", "top level")
        layers_in = _need(d, "layers", "top level")
        if not isinstance(layers_in, list) or not layers_in:
            raise ConfigError('config.json: "layers" must be a non-empty list')
        layers = []
        for i, l in enumerate(layers_in):
            where = f"layers[{i}]"
            kind, mixer = _need(l, "type", where), _need(l, "mixer", where)
            if kind not in MIXERS:
                raise ConfigError(f'config.json: {where}: unknown mixer type {kind!r} (known: {", ".join(MIXERS)})')
            _check_attention(mixer, where + ".mixer")
            mlp = l.get("mlp")
            if mlp is not None:
                _check_mlp(mlp, where + ".mlp")
            layers.append(copy.deepcopy({"type": kind, "mixer": mixer, "mlp": mlp}))
        loop = None
        if d.get("loop") is not None:
            lp = d["loop"]
            start, stop, times = _need(lp, "start", "loop"), _need(lp, "stop", "loop"), _pos_int(lp, "times", "loop")
            if any(isinstance(v, bool) or not isinstance(v, int) for v in (start, stop)) or not 0 <= start < stop <= len(layers):
                raise ConfigError(f'config.json: loop: layers {start!r} .. {stop!r} are not a span of the {len(layers)} layers')
            loop = (start, stop, times)
        cap = None if d.get("logit_softcap") is None else _number(d, "logit_softcap", "top level")
        if cap is not None and cap <= 0:
            raise ConfigError(f'config.json: top level: "logit_softcap" must be positive, found {d["logit_softcap"]!r}')
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab=vocab, width=width, norm_eps=_number(_need(d, "norm", "top level"), "eps", "norm"),
                   layers=tuple(layers), logit_softcap=cap, loop=loop, eos_token_ids=eos_ids,
                   logit_scale=_number(d, "logit_scale", "top level") if d.get("logit_scale") is not None else 1.0,
                   initializer_range=float(d.get("initializer_range", 0.06)))

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers)),
             "initializer_range": self.initializer_range}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    def run_order(self) -> List[LayerCall]:
        n = len(self.layers)
        if self.loop is None:
            return [LayerCall(i) for i in range(n)]
        start, stop, times = self.loop
        return [LayerCall(i) for i in [*range(start), *(times * list(range(start, stop))), *range(stop, n)]]

    def _mixer(self, m: dict) -> PartSpec:
        rot = m.get("rot") or {}
        return PartSpec("sink_attention", {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "key_dim": m["dim"],
            "value_dim": m["vdim"], "scale": float(m["scale"]), "eps": self.norm_eps, "bias": False, "qk_norm": "whole",
            "sink": True, "gate": False, "window": (m.get("mask") or {}).get("size"), "rot_dims": rot.get("dims", 0),
            "rot_base": float(rot.get("base", 10000.0)), "rot_layout": "halves"})

    def _ffn(self, mlp: dict) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": mlp["ff"],
                                       "names": ("gate", "up", "down"), "act": "gelu_tanh"})
        r, groups = mlp["router"], mlp["router"].get("groups") or {}
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "num_experts": r["experts"], "top": r["top"], "expert_size": mlp["expert"]["ff"],
            "router": "softmax", "correction": True, "glu": "silu", "renorm": True, "groups": groups.get("count", 1),
            "keep": groups.get("keep", 1), "identity": r.get("identity") or 0,
            "shared_size": (mlp.get("shared") or {}).get("ff"), "shared_gate": False})

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("layer_norm", {"size": self.width, "eps": self.norm_eps, "has_bias": False})
        layers: List[LayerSpec] = []
        for i, l in enumerate(self.layers):
            ffn = None if l["mlp"] is None else self._ffn(l["mlp"])
            more = (("norm1_out", "norm", norm, "norm1b"),) + ((("norm2_out", "norm", norm, "norm2b"),) if ffn else ())
            layers.append(LayerSpec(prefix=f"l{i}.", norm1=norm, mixer=self._mixer(l["mixer"]), norm2=norm if ffn else None,
                                    ffn=ffn, mixer_prefix="mix.", ffn_prefix="mlp.", norm1_name="norm1",
                                    norm2_name="norm2", block="sandwich_norm", more=more))
        on_logits = None
        if self.logit_scale != 1.0 or self.logit_softcap is not None:
            on_logits = PartSpec("soft_cap", {"scale": self.logit_scale, "cap": self.logit_softcap})
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width,
            max_positions=DEFAULT_MAX_POSITIONS, layers=layers, order=self.run_order(), final_norm=norm,
            embed_name="embed", final_norm_name="final.norm", tie_word_embeddings=True, eos_token_ids=self.eos_token_ids,
            initializer_range=self.initializer_range, on_logits=on_logits)


register_architecture(LovapelConfig.architecture, LovapelConfig)
