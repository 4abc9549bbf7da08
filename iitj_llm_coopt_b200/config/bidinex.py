"""Typed configuration of the Bidinex family, read from its config.json.

Keys: "architecture" ("Bidinex"), "width", "vocab", "norm" {"eps"} (of the latent rows' norm), "residual_mult" (the factor on every
sub-layer's output), "embedding" {"scale"} (absent: 1), "logit_softcap" (absent, null or 0: none), "loop" {"start", "stop", "times"}
(layers start .. stop - 1 run `times` times in a row; absent or null: every layer once) and "layers", a list whose entries give "type"
(which mixer the layer has), the mixer's sizes under "mixer" and the feed-forward under "mlp" (null: none).

Mixer:
  "latent_attention"  "heads", "dim" (unrotated query/key numbers of a head), "rot_dim" (rotated ones), "vdim", "kv_rank" (width of
                      the latent row that is cached), "scale", "rot" {"dims", "base"}.
Feed-forward:
  {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "groups" {"count", "keep"} (absent or null: one group)}}

Every size is read from the file; a missing key is an error at once.
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field

from .errors import ConfigError
from .specs import (EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerCall, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec,
                    StreamJoinSpec)

NAME = "Bidinex"
_MAX_POSITION = 1 << 30          # the design has no position table: int32 positions are the only bound
WEIGHT_SUM_TINY = 1e-20          # what the design adds to the sum of a token's chosen scores before it divides by it


def _get(d: dict, key: str, where: str):
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"config.json lacks required key {key!r} in {where}")
    return d[key]


@dataclass
class BidinexConfig:
    width: int
    vocab: int
    eps: float
    residual_mult: float
    embedding_scale: float = 1.0
    logit_softcap: float = 0.0                       # 0: none
    loop: tuple | None = None                        # (start, stop, times)
    layers: list = field(default_factory=list)       # the file's "layers" entries, as read

    # ---- reading -------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, c: dict) -> "BidinexConfig":
        emb, loop = c.get("embedding"), c.get("loop")
        cfg = cls(width=int(_get(c, "width", "the file")), vocab=int(_get(c, "vocab", "the file")),
                  eps=float(_get(_get(c, "norm", "the file"), "eps", "norm")),
                  residual_mult=float(_get(c, "residual_mult", "the file")),
                  embedding_scale=float(_get(emb, "scale", "embedding")) if emb is not None else 1.0,
                  logit_softcap=float(c.get("logit_softcap") or 0.0),
                  loop=tuple(int(_get(loop, k, "loop")) for k in ("start", "stop", "times")) if loop is not None else None,
                  layers=copy.deepcopy(list(_get(c, "layers", "the file"))))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "BidinexConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path, encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        out = {"architecture": NAME, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
               "residual_mult": self.residual_mult, "embedding": {"scale": self.embedding_scale},
               "layers": copy.deepcopy(self.layers)}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    # ---- checks --------------------------------------------------------------------------
    def validate(self) -> None:
        if self.width <= 0 or self.vocab <= 0:
            raise ConfigError("width and vocab must be positive")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.eps}")
        if self.logit_softcap < 0:
            raise ConfigError("logit_softcap must not be negative")
        if not self.layers:
            raise ConfigError("layers is empty")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ConfigError(f"loop: layers {start} .. {stop - 1} of {len(self.layers)}, {times} times")
        for i, layer in enumerate(self.layers):
            self._validate_layer(layer, f"layers[{i}]")

    @staticmethod
    def _validate_layer(layer: dict, where: str) -> None:
        kind, m = _get(layer, "type", where), _get(layer, "mixer", where)
        if kind != "latent_attention":
            raise ConfigError(f"{where}: type {kind!r} is not known (latent_attention)")
        for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"):
            _get(m, k, where + ".mixer")
        if any(int(m[k]) <= 0 for k in ("heads", "dim", "vdim", "kv_rank")) or int(m["rot_dim"]) < 0:
            raise ConfigError(f"{where}: sizes must be positive")
        rot = _get(m, "rot", where + ".mixer")
        dims = int(_get(rot, "dims", where + ".mixer.rot"))
        if float(_get(rot, "base", where + ".mixer.rot")) <= 0:
            raise ConfigError(f"{where}: rot.base must be positive")
        if dims % 2 or dims < 0 or dims > int(m["rot_dim"]):
            raise ConfigError(f"{where}: rot.dims {dims} must be even and at most rot_dim {m['rot_dim']}")
        mlp = layer.get("mlp")
        if mlp is None:
            return
        ff_kind = _get(mlp, "kind", where + ".mlp")
        if ff_kind != "moe":
            raise ConfigError(f"{where}: mlp.kind {ff_kind!r} is not known (moe)")
        if int(_get(_get(mlp, "expert", where + ".mlp"), "ff", where + ".mlp.expert")) <= 0:
            raise ConfigError(f"{where}: mlp.expert.ff must be positive")
        r = _get(mlp, "router", where + ".mlp")
        experts, top = int(_get(r, "experts", where + ".mlp.router")), int(_get(r, "top", where + ".mlp.router"))
        if experts <= 0 or not 1 <= top <= experts:
            raise ConfigError(f"{where}: router takes {top} of {experts} experts")
        g = r.get("groups")
        if g is not None:
            count, keep = int(_get(g, "count", where + ".mlp.router.groups")), int(_get(g, "keep", where + ".mlp.router.groups"))
            if count < 1 or experts % count or not 1 <= keep <= count:
                raise ConfigError(f"{where}: {experts} experts in {count} groups of which {keep} are kept")
            if top > experts // count * keep:
                raise ConfigError(f"{where}: router takes {top} of the {experts // count * keep} experts of {keep} groups")

    # ---- derived -------------------------------------------------------------------------
    def _layer_spec(self, layer: dict, norm: NormSpec) -> LayerSpec:
        m, rot, mlp = layer["mixer"], layer["mixer"]["rot"], layer.get("mlp")
        pos = PositionSpec(kind="rope", head_dim=int(m["rot_dim"]), rotary_dim=int(rot["dims"]), theta=float(rot["base"]),
                           scaling=(("float64", True), ("type", "none")), max_position=_MAX_POSITION, pairing="half")
        mixer = MixerSpec(kind="latent_attention", width=self.width, heads=int(m["heads"]), kv_heads=1, head_dim=int(m["dim"]),
                          value_dim=int(m["vdim"]), softmax_scale=float(m["scale"]), position=pos if pos.rotary_dim else None,
                          options=(("eps", self.eps), ("gate", "head"), ("kv_rank", int(m["kv_rank"])), ("rot_dim", int(m["rot_dim"]))))
        if mlp is None:
            return LayerSpec.of("prenorm_mixer", mixer_norm=norm, mixer=mixer)
        r = mlp["router"]
        g = r.get("groups")
        ff = FeedForwardSpec(kind="routed_glu", width=self.width, inner=int(mlp["expert"]["ff"]), activation="silu",
                             experts=int(r["experts"]), experts_per_token=int(r["top"]),
                             options=(("correction", False), ("expert", "silu"), ("groups", (int(g["count"]), int(g["keep"])) if g else None),
                                      ("renormalize", WEIGHT_SUM_TINY), ("router", "softmax")))
        return LayerSpec.of("prenorm", mixer_norm=norm, mixer=mixer, feed_forward_norm=norm, feed_forward=ff)

    def model_spec(self) -> ModelSpec:
        """The layers as data.  Cache entry i (pages of latent rows) belongs to the i-th layer run: each pass through the repeated
        layers keeps rows of its own, and its first run enters through the stream join."""
        norm = NormSpec(kind="dynamic_tanh", width=self.width, eps=self.eps, options=(("branch_factor", self.residual_mult),))
        n = len(self.layers)
        start, stop, times = self.loop if self.loop is not None else (0, 0, 0)
        runs = [(i, False) for i in range(start)]
        runs += [(i, i == start) for _ in range(times) for i in range(start, stop)]
        runs += [(i, False) for i in range(stop, n)]
        join = StreamJoinSpec(kind="concat", width=self.width, options=norm.options) if self.loop is not None else None
        return ModelSpec(width=self.width, vocab=self.vocab, layers=tuple(self._layer_spec(l, norm) for l in self.layers),
                         order=tuple(LayerCall(layer=i, cache=c, join=enters) for c, (i, enters) in enumerate(runs)),
                         final_norm=norm, tie_embeddings=True, max_position=_MAX_POSITION, join=join,
                         embedding=EmbeddingSpec(kind="table_dynamic_tanh", vocab=self.vocab, width=self.width, scale=self.embedding_scale),
                         head=HeadSpec(kind="linear", vocab=self.vocab, width=self.width,
                                       options=(("softcap", self.logit_softcap),) if self.logit_softcap else ()))
