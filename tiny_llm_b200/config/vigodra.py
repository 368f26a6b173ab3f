"""Typed configuration of Vigodra, a small decoder whose layers norm the SUM of the scaled stream and a branch
(x <- n1(a x + mixer(x)); x <- n2(a x + ff(x)), layer norms with weight and bias) and hand on a learned weighted sum of
the embedding output and every layer's result so far.  A layer mixes tokens in one of two ways: grouped-query attention
behind short causal filters on q, k and v, with queries and keys normed over the whole projection, no rotation but a
learned bias per head and distance, a sliding window that keeps the sequence's first positions, a sink in the softmax and
biases on every projection; or latent attention (keys and values projected from one small cached vector per token, a key
part rotated in halves and shared by the heads, a sliding window, a gate per output value), whose layers may read the
latents that an earlier layer cached.  Feed-forwards are gated with both sides clamped.  The embedding is multiplied by
a constant.

config.json keys (every size and every constant that differs between models of the design comes from here):

  architecture      "Vigodra"
  vocab, width      vocabulary and width of the residual stream
  embedding.scale   what the embedding rows are multiplied by
  norm.eps          eps of every norm
  postln_alpha      what the stream is multiplied by where a branch joins it
  layers[i]         {"type": "attention" | "latent_attention", "mixer": {...}, "mlp": {...} | null}
    attention         {"heads", "kv_heads", "dim", "vdim", "scale", "conv", "bias_max",
                       "mask": {"size", "keep_first"?} | absent}   (the number of distance buckets is the table's)
    latent_attention  {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot": {"dims", "base"},
                       "mask": {"size"} | absent, "kv_from": j | absent}
                      (with kv_from the layer has no `dkv` and reads layer j's cache)
    mlp               {"kind": "dense", "ff", "limit"}

Tensor names: `embed`, `head`, `final.norm`, `final.norm.b`, and per layer `l<i>.norm1`, `l<i>.norm2` (each with `.b`),
`l<i>.mix.*`, `l<i>.mlp.gate|up|down`, `l<i>.dwa` (i + 2 numbers)."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Tuple

from .dunelix import DEFAULT_MAX_POSITIONS, _need, _number, _pos_int
from .errors import ConfigError
from .registry import register_architecture
from .spec import LayerCall, LayerSpec, ModelSpec, PartSpec

MIXERS = ("attention", "latent_attention")


def _check_mask(m: dict, where: str) -> None:
    mask = m.get("mask")
    if mask is None:
        return
    _pos_int(mask, "size", where + ".mask")
    keep = mask.get("keep_first", 0)
    if keep is not None and (isinstance(keep, bool) or not isinstance(keep, int) or keep < 0):
        raise ConfigError(f'config.json: {where}.mask: "keep_first" must be a count of positions, found {keep!r}')


def _check_attention(m: dict, where: str) -> None:
    heads, kv = _pos_int(m, "heads", where), _pos_int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f'config.json: {where}: "heads" ({heads}) must be a multiple of "kv_heads" ({kv})')
    for k in ("dim", "vdim", "conv"):
        _pos_int(m, k, where)
    _number(m, "scale", where)
    if _number(m, "bias_max", where) <= 1:
        raise ConfigError(f'config.json: {where}: "bias_max" must be a distance above 1, found {m["bias_max"]!r}')
    _check_mask(m, where)


def _check_latent(m: dict, where: str, index: int, layers: list) -> None:
    for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"):
        _pos_int(m, k, where)
    _number(m, "scale", where)
    rot = _need(m, "rot", where)
    dims = _pos_int(rot, "dims", where + ".rot")
    if dims % 2 or dims > m["rot_dim"]:
        raise ConfigError(f'config.json: {where}.rot: "dims" ({dims}) must be even and at most "rot_dim" ({m["rot_dim"]})')
    if _number(rot, "base", where + ".rot") <= 0:
        raise ConfigError(f'config.json: {where}.rot: "base" must be positive')
    _check_mask(m, where)
    if (m.get("mask") or {}).get("keep_first"):
        raise ConfigError(f'config.json: {where}.mask: a latent attention\'s window keeps no first positions')
    src = m.get("kv_from")
    if src is not None:
        if not isinstance(src, int) or isinstance(src, bool) or not 0 <= src < index:
            raise ConfigError(f'config.json: {where}: "kv_from" must name an earlier layer, found {src!r}')
        other = layers[src]
        if other.get("type") != "latent_attention" or other["mixer"].get("kv_from") is not None:
            raise ConfigError(f'config.json: {where}: "kv_from" names layer {src}, which keeps no latents of its own')
        for k in ("kv_rank", "rot_dim", "rot"):
            if other["mixer"].get(k) != m.get(k):
                raise ConfigError(f'config.json: {where}: "{k}" differs from layer {src}, whose cache this layer reads')


@dataclass(frozen=True)
class VigodraConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    alpha: float
    layers: Tuple[Dict[str, Any], ...]
    eos_token_ids: Tuple[int, ...] = ()
    initializer_range: float = 0.06

    architecture = "Vigodra"

    @classmethod
    def from_dict(cls, d: dict) -> "VigodraConfig":
        vocab, width = _pos_int(d, "vocab", "top level"), _pos_int(d, "width", "top level")
        layers_in = _need(d, "layers", "top level")
        if not isinstance(layers_in, list) or not layers_in:
            raise ConfigError('config.json: "layers" must be a non-empty list')
        layers = []
        for i, l in enumerate(layers_in):
            where = f"layers[{i}]"
            kind, mixer = _need(l, "type", where), _need(l, "mixer", where)
            if kind == "attention":
                _check_attention(mixer, where + ".mixer")
            elif kind == "latent_attention":
                _check_latent(mixer, where + ".mixer", i, layers_in)
            else:
                raise ConfigError(f'config.json: {where}: unknown mixer type {kind!r} (known: {", ".join(MIXERS)})')
            mlp = l.get("mlp")
            if mlp is not None:
                if _need(mlp, "kind", where + ".mlp") != "dense":
                    raise ConfigError(f'config.json: {where}.mlp: unknown kind {mlp["kind"]!r} (known: dense)')
                _pos_int(mlp, "ff", where + ".mlp")
                if _number(mlp, "limit", where + ".mlp") <= 0:
                    raise ConfigError(f'config.json: {where}.mlp: "limit" must be positive, found {mlp["limit"]!r}')
            layers.append(copy.deepcopy({"type": kind, "mixer": mixer, "mlp": mlp}))
        emb = d.get("embedding") or {}
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab=vocab, width=width,
                   embedding_scale=_number(emb, "scale", "embedding") if emb.get("scale") is not None else 1.0,
                   norm_eps=_number(_need(d, "norm", "top level"), "eps", "norm"),
                   alpha=_number(d, "postln_alpha", "top level"), layers=tuple(layers), eos_token_ids=eos_ids,
                   initializer_range=float(d.get("initializer_range", 0.06)))

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
             "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps}, "postln_alpha": self.alpha,
             "layers": copy.deepcopy(list(self.layers)), "initializer_range": self.initializer_range}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    def _mixer(self, l: dict) -> PartSpec:
        m, w, eps = l["mixer"], self.width, self.norm_eps
        mask = m.get("mask") or {}
        if l["type"] == "attention":
            return PartSpec("sink_attention", {
                "hidden_size": w, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "key_dim": m["dim"],
                "value_dim": m["vdim"], "scale": float(m["scale"]), "eps": eps, "bias": True, "qk_norm": "whole",
                "sink": True, "gate": False, "window": mask.get("size"), "keep_first": mask.get("keep_first") or 0,
                "conv": m["conv"], "bias_max": float(m["bias_max"]), "out_bias": True})
        rot = m["rot"]
        return PartSpec("latent_attention", {
            "hidden_size": w, "num_heads": m["heads"], "plain_dim": m["dim"], "rot_part": m["rot_dim"],
            "value_dim": m["vdim"], "rank": m["kv_rank"], "scale": float(m["scale"]), "eps": eps, "rot_dims": rot["dims"],
            "rot_base": float(rot["base"]), "rot_layout": "halves", "window": mask.get("size"), "sink": False,
            "gate": "value"})

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("layer_norm", {"size": self.width, "eps": self.norm_eps})
        layers: List[LayerSpec] = []
        order: List[LayerCall] = []
        for i, l in enumerate(self.layers):
            ffn = None
            if l["mlp"] is not None:
                ffn = PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": l["mlp"]["ff"],
                                          "names": ("gate", "up", "down"), "act": "clamped", "limit": float(l["mlp"]["limit"])})
            layers.append(LayerSpec(prefix=f"l{i}.", norm1=norm, mixer=self._mixer(l), norm2=norm if ffn else None,
                                    ffn=ffn, mixer_prefix="mix.", ffn_prefix="mlp.", norm1_name="norm1",
                                    norm2_name="norm2", block="post_norm", stream_scale=self.alpha))
            order.append(LayerCall(i, reads_cache_of=l["mixer"].get("kv_from") if l["type"] == "latent_attention" else None))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width,
            max_positions=DEFAULT_MAX_POSITIONS, layers=layers, order=order, final_norm=norm, embed_name="embed",
            final_norm_name="final.norm", lm_head_name="head", tie_word_embeddings=False,
            eos_token_ids=self.eos_token_ids, initializer_range=self.initializer_range,
            embedding_scale=self.embedding_scale, depth_average="dwa")


register_architecture(VigodraConfig.architecture, VigodraConfig)
