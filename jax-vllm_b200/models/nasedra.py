"""Nasedra: config.json -> typed configuration -> `ModelSpec`.

A decoder-only design whose layers are listed one by one in config.json (`layers`: each entry has `type`, the mixer's
sizes under `mixer`, and `mlp` or null).  What the design fixes is fixed here; every size and constant that config.json
carries is read from it, and the rank of the decay's projection, which only a tensor's shape gives, is left open until the
weights are bound.  With norm(x) an RMSNorm (eps = `norm.eps`):

    x = embed[token] * embedding.scale
    x <- x + mixer(norm1(x)) + ff(norm2(x))                both of the same x (a layer without `mlp` has no second term)
    logits = head norm_final(x)

mixers:

    "attention"   causal grouped-query softmax attention: rotation of the first `rot.dims` elements of a head in interleaved
                  pairs, frequencies and gain by YaRN (`rot.scaling`); scores capped by tanh (`softcap`); a window of
                  `mask.size` positions under which the first `mask.keep_first` tokens stay visible; a sigmoid gate per
                  output element.  With `kv_from` = j it reads layer j's cached keys and values and has no projections of
                  its own for them
    "gla"         gated linear attention: a matrix state per head with a decay per key channel (parts/recurrent.py)

feed-forwards: `dense` (gated silu) or `moe` (softmax router with a correction for the choice and identity experts, gated
silu experts, an optional shared expert).  Tensor names: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.*`, `l<i>.mlp.*`,
`final.norm`, `head`.
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass
from pathlib import Path

from ..config.model_spec import (GatedLinearAttentionSpec, GatedMLPSpec, GeneralAttentionSpec, LayerSpec, ModelSpec, NormSpec,
                                 RopeSpec, RoutedExpertsSpec)

ARCHITECTURE = "Nasedra"
MIXERS = ("attention", "gla")
FEED_FORWARDS = ("dense", "moe")
RENORM_EPS = 1e-20
SCALING = ("factor", "original", "fast", "slow")


def _need(d: dict, keys, where: str) -> None:
    if not isinstance(d, dict):
        raise KeyError(f"config.json: {where} is not an object")
    missing = [k for k in keys if k not in d]
    if missing:
        raise KeyError(f"config.json: {where} lacks {missing}")


def _positive(d: dict, keys, where: str) -> None:
    for k in keys:
        if int(d[k]) < 1:
            raise ValueError(f"{where}.{k} must be positive")


@dataclass(frozen=True)
class NasedraConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: tuple                 # the entries of config.json's `layers`, as read

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, c: dict) -> "NasedraConfig":
        _need(c, ("vocab", "width", "layers", "norm", "embedding"), "the top level")
        _need(c["norm"], ("eps",), "norm")
        _need(c["embedding"], ("scale",), "embedding")
        cfg = cls(vocab=int(c["vocab"]), width=int(c["width"]), norm_eps=float(c["norm"]["eps"]),
                  embedding_scale=float(c["embedding"]["scale"]), layers=tuple(copy.deepcopy(layer) for layer in c["layers"]))
        cfg.validate()
        return cfg

    @classmethod
    def from_path(cls, path) -> "NasedraConfig":
        p = Path(path)
        if p.is_dir():
            p = p / "config.json"
        return cls.from_dict(json.loads(p.read_text()))

    def validate(self) -> None:
        if self.vocab < 1 or self.width < 1 or not self.layers:
            raise ValueError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ValueError("norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            kind, mx = layer["type"], layer["mixer"]
            if kind not in MIXERS:
                raise ValueError(f"{where}: mixer type {kind!r} is not part of this design ({MIXERS})")
            if kind == "gla":
                _need(mx, ("heads", "dim", "vdim", "tau"), f"{where}.mixer")
                _positive(mx, ("heads", "dim", "vdim"), f"{where}.mixer")
                if not float(mx["tau"]) > 0:
                    raise ValueError(f"{where}: tau must be positive")
            else:
                self._validate_attention(i, mx, f"{where}.mixer")
            self._validate_mlp(layer.get("mlp"), f"{where}.mlp")

    def _validate_attention(self, i: int, mx: dict, where: str) -> None:
        _need(mx, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
        _positive(mx, ("heads", "kv_heads", "dim", "vdim"), where)
        if int(mx["heads"]) % int(mx["kv_heads"]):
            raise ValueError(f"{where}: heads must be a multiple of kv_heads")
        rot = mx.get("rot")
        if rot is not None:
            _need(rot, ("base", "dims"), f"{where}.rot")
            if int(rot["dims"]) % 2 or not 2 <= int(rot["dims"]) <= int(mx["dim"]):
                raise ValueError(f"{where}: rot.dims must be even, positive and at most dim")
            if rot.get("scaling") is not None:
                _need(rot["scaling"], SCALING, f"{where}.rot.scaling")
        if mx.get("softcap") is not None and not float(mx["softcap"]) > 0:
            raise ValueError(f"{where}: softcap must be positive")
        mask = mx.get("mask")
        if mask is not None:
            _need(mask, ("size",), f"{where}.mask")
            if int(mask["size"]) < 1 or int(mask.get("keep_first", 0)) < 0:
                raise ValueError(f"{where}: mask.size must be positive and mask.keep_first not negative")
        j = mx.get("kv_from")
        if j is not None:
            owner = self.layers[j] if isinstance(j, int) and 0 <= j < i else None
            if owner is None or owner["type"] != "attention" or owner["mixer"].get("kv_from") is not None:
                raise ValueError(f"{where}: kv_from={j} must name an earlier attention layer with keys and values of its own")
            if any(int(mx[k]) != int(owner["mixer"][k]) for k in ("kv_heads", "dim", "vdim")):
                raise ValueError(f"{where}: the key/value heads must be those of layer {j}")

    @staticmethod
    def _validate_mlp(ml, where: str) -> None:
        if ml is None:
            return
        _need(ml, ("kind",), where)
        if ml["kind"] not in FEED_FORWARDS:
            raise ValueError(f"{where}: feed-forward kind {ml['kind']!r} is not part of this design ({FEED_FORWARDS})")
        if ml["kind"] == "dense":
            _need(ml, ("ff",), where)
            _positive(ml, ("ff",), where)
            return
        _need(ml, ("expert", "router"), where)
        _need(ml["expert"], ("ff",), f"{where}.expert")
        _positive(ml["expert"], ("ff",), f"{where}.expert")
        ro = ml["router"]
        _need(ro, ("experts", "top", "scale"), f"{where}.router")
        _positive(ro, ("experts", "top"), f"{where}.router")
        identity = int(ro.get("identity", 0))
        if identity < 0 or int(ro["top"]) > int(ro["experts"]) + identity:
            raise ValueError(f"{where}: {ro['experts']} experts, {identity} identity experts, top {ro['top']} do not fit")
        if ml.get("shared") is not None:
            _need(ml["shared"], ("ff",), f"{where}.shared")
            _positive(ml["shared"], ("ff",), f"{where}.shared")

    def to_dict(self) -> dict:
        """config.json content for this configuration."""
        return {"architecture": ARCHITECTURE, "embedding": {"scale": self.embedding_scale},
                "layers": [copy.deepcopy(layer) for layer in self.layers], "norm": {"eps": self.norm_eps},
                "vocab": self.vocab, "width": self.width}

    # ----------------------------------------------------------------- the model
    def _mixer(self, kind: str, mx: dict):
        W = self.width
        if kind == "gla":
            return GatedLinearAttentionSpec(hidden_size=W, num_heads=int(mx["heads"]), key_dim=int(mx["dim"]),
                                            value_dim=int(mx["vdim"]), tau=float(mx["tau"]), q_scale=int(mx["dim"]) ** -0.5,
                                            norm_eps=self.norm_eps, prefix="mix")
        rot, mask = mx.get("rot"), mx.get("mask") or {}
        position = None
        if rot is not None:
            scaling = rot.get("scaling")
            position = RopeSpec(dim=int(rot["dims"]), theta=float(rot["base"]), exact_table=True, layout="interleaved",
                                yarn=None if scaling is None else tuple(float(scaling[k]) for k in SCALING))
        return GeneralAttentionSpec(
            hidden_size=W, num_heads=int(mx["heads"]), num_kv_heads=int(mx["kv_heads"]), key_dim=int(mx["dim"]),
            value_dim=int(mx["vdim"]), scale=float(mx["scale"]), position=position, gate="element", prefix="mix",
            score_cap=None if mx.get("softcap") is None else float(mx["softcap"]),
            window=int(mask["size"]) if mask else None, keep_first=int(mask.get("keep_first", 0)))

    def _feed_forward(self, ml):
        W = self.width
        if ml is None:
            return None
        if ml["kind"] == "dense":
            return GatedMLPSpec(hidden_size=W, intermediate_size=int(ml["ff"]), prefix="mlp", names=("gate", "up", "down"))
        ro, shared = ml["router"], ml.get("shared")
        return RoutedExpertsSpec(hidden_size=W, num_experts=int(ro["experts"]), top_k=int(ro["top"]),
                                 expert_size=int(ml["expert"]["ff"]), scoring="softmax", renormalize=True, activation="swiglu",
                                 renorm_eps=RENORM_EPS, weight_scale=float(ro["scale"]), correction="correction",
                                 identity=int(ro.get("identity", 0)), shared_size=0 if shared is None else int(shared["ff"]),
                                 prefix="mlp")

    def to_spec(self) -> ModelSpec:
        eps, W = self.norm_eps, self.width
        layers = []
        for i, layer in enumerate(self.layers):
            ff = self._feed_forward(layer.get("mlp"))
            layers.append(LayerSpec(prefix=f"l{i}", mixer=self._mixer(layer["type"], layer["mixer"]), feed_forward=ff,
                                    mixer_norm=NormSpec(W, eps, "norm1"),
                                    ffn_norm=None if ff is None else NormSpec(W, eps, "norm2"),
                                    cache_from=layer["mixer"].get("kv_from"), kind="parallel"))
        # a layer without a feed-forward reads no second norm: a folder that holds one all the same is taken as it is
        unused = tuple(f"l{i}.norm2" for i, layer in enumerate(layers) if layer.feed_forward is None)
        spec = ModelSpec(architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=W, layers=tuple(layers),
                         final_norm=NormSpec(W, eps, "final.norm"), embedding_name="embed", lm_head_name="head",
                         embedding_scale=self.embedding_scale, unused_tensors=unused)
        spec.validate()
        return spec
