"""Typed configuration of the Kobolix family, read from its config.json.

Keys: "architecture" ("Kobolix"), "width", "vocab", "norm" {"eps"}, "residual_mult" (the factor on every sub-layer's output; absent:
1), "embedding" {"scale"} (absent: 1) and "layers", a list whose entries give "type" (which mixer the layer has), the mixer's sizes
under "mixer" and the feed-forward under "mlp" (null: none).

Mixers:
  "mlstm"     "heads", "dim", "vdim", "gate_cap".
  "parallel"  "left": "heads", "kv_heads", "dim", "vdim", "scale", "rot" {"dims", "base"} (absent or null: nothing rotates);
              "right": "heads", "kv_heads", "dim", "vdim", "conv".
Feed-forwards:
  {"kind": "dense", "ff"}
  {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "groups" {"count", "keep"} (absent or null: one group), "scale"
   (absent: 1)}, "shared": {"ff"} (absent or null: none)}

Every size is read from the file; a missing key is an error at once.
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field

from .errors import ConfigError
from .specs import EmbeddingSpec, FeedForwardSpec, LayerCall, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec

NAME = "Kobolix"
_MAX_POSITION = 1 << 30          # the design has no position table: int32 positions are the only bound
MEMORY_TINY = 1e-6               # what the design adds to the matrix memory's divisor
UNIT_TINY = 1e-6                 # what it adds to the squared length of the delta rule's queries and keys
GROUP_WORTH = 2                  # a group of experts is worth the sum of that many of its largest scores


def _get(d: dict, key: str, where: str):
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"config.json lacks required key {key!r} in {where}")
    return d[key]


def _positive(d: dict, keys: tuple, where: str) -> None:
    for k in keys:
        if int(_get(d, k, where)) <= 0:
            raise ConfigError(f"{where}.{k} must be positive")


def _grouped(d: dict, where: str) -> None:
    if int(d["heads"]) % int(d["kv_heads"]):
        raise ConfigError(f"{where}: heads {d['heads']} is not a multiple of kv_heads {d['kv_heads']}")


@dataclass
class KobolixConfig:
    width: int
    vocab: int
    eps: float
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    layers: list = field(default_factory=list)       # the file's "layers" entries, as read

    # ---- reading -------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, c: dict) -> "KobolixConfig":
        emb, mult = c.get("embedding"), c.get("residual_mult")
        cfg = cls(width=int(_get(c, "width", "the file")), vocab=int(_get(c, "vocab", "the file")),
                  eps=float(_get(_get(c, "norm", "the file"), "eps", "norm")),
                  residual_mult=1.0 if mult is None else float(mult),
                  embedding_scale=float(_get(emb, "scale", "embedding")) if emb is not None else 1.0,
                  layers=copy.deepcopy(list(_get(c, "layers", "the file"))))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "KobolixConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path, encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        return {"architecture": NAME, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
                "residual_mult": self.residual_mult, "embedding": {"scale": self.embedding_scale},
                "layers": copy.deepcopy(self.layers)}

    # ---- checks --------------------------------------------------------------------------
    def validate(self) -> None:
        if self.width <= 0 or self.vocab <= 0:
            raise ConfigError("width and vocab must be positive")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.eps}")
        if not self.layers:
            raise ConfigError("layers is empty")
        for i, layer in enumerate(self.layers):
            self._validate_mixer(layer, f"layers[{i}]")
            if layer.get("mlp") is not None:
                self._validate_mlp(layer["mlp"], f"layers[{i}].mlp")

    @staticmethod
    def _validate_mixer(layer: dict, where: str) -> None:
        kind, m = _get(layer, "type", where), _get(layer, "mixer", where)
        where += ".mixer"
        if kind == "mlstm":
            _positive(m, ("heads", "dim", "vdim"), where)
            if not float(_get(m, "gate_cap", where)) > 0:
                raise ConfigError(f"{where}.gate_cap must be positive")
        elif kind == "parallel":
            left, right = _get(m, "left", where), _get(m, "right", where)
            _positive(left, ("heads", "kv_heads", "dim", "vdim"), where + ".left")
            _positive(right, ("heads", "kv_heads", "dim", "vdim", "conv"), where + ".right")
            _grouped(left, where + ".left")
            _grouped(right, where + ".right")
            if float(_get(left, "scale", where + ".left")) == 0:
                raise ConfigError(f"{where}.left.scale must not be zero")
            rot = left.get("rot")
            if rot is not None:
                dims = int(_get(rot, "dims", where + ".left.rot"))
                if float(_get(rot, "base", where + ".left.rot")) <= 0:
                    raise ConfigError(f"{where}.left.rot.base must be positive")
                if dims % 2 or dims < 0 or dims > int(left["dim"]):
                    raise ConfigError(f"{where}.left.rot.dims {dims} must be even and at most dim {left['dim']}")
        else:
            raise ConfigError(f"{where}: type {kind!r} is not known (mlstm, parallel)")

    @staticmethod
    def _validate_mlp(mlp: dict, where: str) -> None:
        kind = _get(mlp, "kind", where)
        if kind == "dense":
            _positive(mlp, ("ff",), where)
            return
        if kind != "moe":
            raise ConfigError(f"{where}: mlp.kind {kind!r} is not known (dense, moe)")
        _positive(_get(mlp, "expert", where), ("ff",), where + ".expert")
        if mlp.get("shared") is not None:
            _positive(mlp["shared"], ("ff",), where + ".shared")
        r = _get(mlp, "router", where)
        experts, top = int(_get(r, "experts", where + ".router")), int(_get(r, "top", where + ".router"))
        if experts <= 0 or not 1 <= top <= experts:
            raise ConfigError(f"{where}: router takes {top} of {experts} experts")
        g = r.get("groups")
        if g is not None:
            count, keep = int(_get(g, "count", where + ".router.groups")), int(_get(g, "keep", where + ".router.groups"))
            if count < 1 or experts % count or not 1 <= keep <= count:
                raise ConfigError(f"{where}: {experts} experts in {count} groups of which {keep} are kept")
            if top > experts // count * keep:
                raise ConfigError(f"{where}: router takes {top} of the {experts // count * keep} experts of {keep} groups")

    # ---- derived -------------------------------------------------------------------------
    def _mixer_spec(self, layer: dict) -> MixerSpec:
        m = layer["mixer"]
        if layer["type"] == "mlstm":
            return MixerSpec(kind="matrix_memory", width=self.width, heads=int(m["heads"]), head_dim=int(m["dim"]), value_dim=int(m["vdim"]),
                             options=(("eps", self.eps), ("gate_cap", float(m["gate_cap"])), ("tiny", MEMORY_TINY)))
        lm, rm, rot = m["left"], m["right"], m["left"].get("rot")
        pos = None
        if rot is not None and int(rot["dims"]):
            pos = PositionSpec(kind="rope", head_dim=int(lm["dim"]), rotary_dim=int(rot["dims"]), theta=float(rot["base"]),
                               scaling=(("float64", True), ("type", "none")), max_position=_MAX_POSITION, pairing="interleaved")
        left = MixerSpec(kind="gated_attention", width=self.width, heads=int(lm["heads"]), kv_heads=int(lm["kv_heads"]),
                         head_dim=int(lm["dim"]), value_dim=int(lm["vdim"]), softmax_scale=float(lm["scale"]), position=pos,
                         options=(("eps", self.eps),))
        right = MixerSpec(kind="gated_delta", width=self.width, heads=int(rm["heads"]), kv_heads=int(rm["kv_heads"]),
                          head_dim=int(rm["dim"]), value_dim=int(rm["vdim"]),
                          options=(("conv_taps", int(rm["conv"])), ("eps", self.eps), ("unit_tiny", UNIT_TINY)))
        return MixerSpec(kind="parallel", width=self.width, position=pos,
                         options=(("eps", self.eps), ("left", left), ("right", right), ("scale", 0.5)))

    def _feed_forward_spec(self, mlp: dict) -> FeedForwardSpec:
        if mlp["kind"] == "dense":
            return FeedForwardSpec(kind="swiglu", width=self.width, inner=int(mlp["ff"]))
        r = mlp["router"]
        g, scale = r.get("groups"), r.get("scale")
        options = {"correction": False, "expert": "silu", "router": "sigmoid",
                   "groups": (int(g["count"]), int(g["keep"])) if g else None, "group_worth": GROUP_WORTH,
                   "weight_scale": 1.0 if scale is None else float(scale),
                   "shared": int(mlp["shared"]["ff"]) if mlp.get("shared") is not None else 0}
        return FeedForwardSpec(kind="routed_glu", width=self.width, inner=int(mlp["expert"]["ff"]), experts=int(r["experts"]),
                               experts_per_token=int(r["top"]), options=tuple(sorted(options.items())))

    def model_spec(self) -> ModelSpec:
        """The layers as data.  A layer of matrix memory owns one cache entry (a record per request), a parallel layer two: pages for
        its attention and a record for its delta rule."""
        norm = NormSpec(kind="rmsnorm_one_plus", width=self.width, eps=self.eps, options=(("branch_factor", self.residual_mult),))
        layers, order, entries = [], [], 0
        for i, layer in enumerate(self.layers):
            parallel = layer["type"] == "parallel"
            order.append(LayerCall(layer=i, cache=entries, state=entries + 1 if parallel else None))
            entries += 2 if parallel else 1
            mixer, mlp = self._mixer_spec(layer), layer.get("mlp")
            if mlp is None:
                layers.append(LayerSpec.of("prenorm_mixer", mixer_norm=norm, mixer=mixer))
            else:
                layers.append(LayerSpec.of("prenorm", mixer_norm=norm, mixer=mixer, feed_forward_norm=norm,
                                           feed_forward=self._feed_forward_spec(mlp)))
        return ModelSpec(width=self.width, vocab=self.vocab, layers=tuple(layers), order=tuple(order), final_norm=norm,
                         tie_embeddings=True, max_position=_MAX_POSITION,
                         embedding=EmbeddingSpec(kind="table", vocab=self.vocab, width=self.width, scale=self.embedding_scale))
