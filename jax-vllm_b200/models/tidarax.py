"""Tidarax: config.json -> typed configuration -> `ModelSpec`.

A decoder-only design whose layers are listed one by one in config.json (`layers`: each entry has `type`, the mixer's
sizes under `mixer`, and `mlp` or null).  What the design fixes is fixed here; every size and constant that config.json
carries is read from it.  With norm(x) = x / sqrt(mean(x^2) + eps) * (1 + w):

    x = embed[token]
    x <- x + mixer(norm1(x));   x <- x + ff(norm2(x))            (a layer may have no feed-forward)
    logits = head norm_final(x)

The one mixer, `parallel`, is two mixers on the same input, left_scale * left + right_scale * right
(parts/mixer_pair.py):

    left    causal grouped-query attention (parts/general_attention.py): queries and keys rotated in halves over the
            first `rot.dims` elements (frequencies scaled by wavelength bands, `rot.scaling`) and divided by their root
            mean square head by head; the heads' scaled scores mixed by a matrix [heads, heads] before the softmax, whose
            denominator has one added
    right   a recurrence whose gates read only the current token (parts/min_gru.py)

feed-forwards: `dense` (down(act(up u)) with a polynomial of normed powers as the activation) or `moe` (gated silu
experts that a table names for each token id, all with the same weight).  Tensor names: `embed`, `l<i>.norm1|norm2`,
`l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass
from pathlib import Path

from ..config.model_spec import (DenseMLPSpec, GeneralAttentionSpec, LayerSpec, MinGRUSpec, MixerPairSpec, ModelSpec,
                                 NormSpec, RopeSpec, RoutedExpertsSpec)

ARCHITECTURE = "Tidarax"
MIXERS = ("parallel",)
FEED_FORWARDS = ("dense", "moe")


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
class TidaraxConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple                 # the entries of config.json's `layers`, as read

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, c: dict) -> "TidaraxConfig":
        _need(c, ("vocab", "width", "layers", "norm"), "the top level")
        _need(c["norm"], ("eps",), "norm")
        cfg = cls(vocab=int(c["vocab"]), width=int(c["width"]), norm_eps=float(c["norm"]["eps"]),
                  layers=tuple(copy.deepcopy(layer) for layer in c["layers"]))
        cfg.validate()
        return cfg

    @classmethod
    def from_path(cls, path) -> "TidaraxConfig":
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
            if layer["type"] not in MIXERS:
                raise ValueError(f"{where}: mixer type {layer['type']!r} is not part of this design ({MIXERS})")
            mx = layer["mixer"]
            _need(mx, ("left", "right", "left_scale", "right_scale"), f"{where}.mixer")
            left, right = mx["left"], mx["right"]
            _need(left, ("heads", "kv_heads", "dim", "vdim", "scale"), f"{where}.mixer.left")
            _positive(left, ("heads", "kv_heads", "dim", "vdim"), f"{where}.mixer.left")
            if int(left["heads"]) % int(left["kv_heads"]):
                raise ValueError(f"{where}: heads must be a multiple of kv_heads")
            rot = left.get("rot")
            if rot is not None:
                _need(rot, ("base", "dims"), f"{where}.mixer.left.rot")
                if int(rot["dims"]) % 2 or not 2 <= int(rot["dims"]) <= int(left["dim"]):
                    raise ValueError(f"{where}: rot.dims must be even, positive and at most dim")
                if rot.get("scaling") is not None:
                    _need(rot["scaling"], ("factor", "low", "high", "original"), f"{where}.mixer.left.rot.scaling")
            _need(right, ("width",), f"{where}.mixer.right")
            _positive(right, ("width",), f"{where}.mixer.right")
            ml = layer.get("mlp")
            if ml is None:
                continue
            _need(ml, ("kind",), f"{where}.mlp")
            if ml["kind"] not in FEED_FORWARDS:
                raise ValueError(f"{where}: feed-forward kind {ml['kind']!r} is not part of this design ({FEED_FORWARDS})")
            if ml["kind"] == "dense":
                _need(ml, ("ff",), f"{where}.mlp")
                _positive(ml, ("ff",), f"{where}.mlp")
            else:
                _need(ml, ("expert", "router"), f"{where}.mlp")
                _need(ml["expert"], ("ff",), f"{where}.mlp.expert")
                _need(ml["router"], ("experts", "top"), f"{where}.mlp.router")
                _positive(ml["expert"], ("ff",), f"{where}.mlp.expert")
                _positive(ml["router"], ("experts", "top"), f"{where}.mlp.router")
                if int(ml["router"]["top"]) > int(ml["router"]["experts"]):
                    raise ValueError(f"{where}: a token cannot use more experts than there are")

    def to_dict(self) -> dict:
        """config.json content for this configuration."""
        return {"architecture": ARCHITECTURE, "layers": [copy.deepcopy(layer) for layer in self.layers],
                "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}

    # ----------------------------------------------------------------- the model
    def _mixer(self, mx: dict) -> MixerPairSpec:
        eps, W = self.norm_eps, self.width
        left, right, rot = mx["left"], mx["right"], mx["left"].get("rot")
        position = None
        if rot is not None:
            sc = rot.get("scaling")
            position = RopeSpec(dim=int(rot["dims"]), theta=float(rot["base"]), exact_table=True,
                                bands=None if sc is None else tuple(float(sc[k]) for k in ("factor", "low", "high", "original")))
        attention = GeneralAttentionSpec(
            hidden_size=W, num_heads=int(left["heads"]), num_kv_heads=int(left["kv_heads"]), key_dim=int(left["dim"]),
            value_dim=int(left["vdim"]), scale=float(left["scale"]), position=position, head_norm_eps=eps,
            head_norm_weight=False, talk=True, sink_score=0.0, output_scale=float(mx["left_scale"]), prefix="left")
        gru = MinGRUSpec(hidden_size=W, width=int(right["width"]), output_scale=float(mx["right_scale"]), prefix="right")
        return MixerPairSpec(hidden_size=W, left=attention, right=gru, combine="sum", prefix="mix")

    def _feed_forward(self, ml):
        W = self.width
        if ml is None:
            return None
        if ml["kind"] == "dense":
            return DenseMLPSpec(hidden_size=W, intermediate_size=int(ml["ff"]), activation="poly_norm",
                                norm_eps=self.norm_eps, prefix="mlp")
        return RoutedExpertsSpec(hidden_size=W, num_experts=int(ml["router"]["experts"]), top_k=int(ml["router"]["top"]),
                                 expert_size=int(ml["expert"]["ff"]), scoring="table", activation="swiglu",
                                 vocab_size=self.vocab, prefix="mlp")

    def to_spec(self) -> ModelSpec:
        eps, W = self.norm_eps, self.width
        layers = []
        for i, layer in enumerate(self.layers):
            ff = self._feed_forward(layer.get("mlp"))
            layers.append(LayerSpec(prefix=f"l{i}", mixer=self._mixer(layer["mixer"]), feed_forward=ff,
                                    mixer_norm=NormSpec(W, eps, "norm1", offset=1.0),
                                    ffn_norm=None if ff is None else NormSpec(W, eps, "norm2", offset=1.0), kind="pre_norm"))
        # a layer without a feed-forward reads no second norm: a folder that holds one all the same is taken as it is
        unused = tuple(f"l{i}.norm2" for i, layer in enumerate(layers) if layer.feed_forward is None)
        spec = ModelSpec(architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=W, layers=tuple(layers),
                         final_norm=NormSpec(W, eps, "final.norm", offset=1.0), embedding_name="embed",
                         lm_head_name="head", unused_tensors=unused)
        spec.validate()
        return spec
