"""Bidinex: layers of latent attention (one normed low-rank row and one rotated key part per token serve every head as key and as
value, a sigmoid gate of one number a head on the heads' outputs) and of routed silu-gated experts (only experts of the best groups,
softmax scores divided by the sum of the chosen ones), norms tanh(alpha x) * gain + shift in front of every sub-layer, behind the
embedding and before the head, one factor on every sub-layer's output, capped logits.  A run of layers may be walked several times in
a row with the same weights and rows of its own in the cache; every pass enters through a product of the stream and the embedding's
output.

Checkpoint tensor names: embed (also the output projection), embed.norm, final.norm, loop.in, and for layer i: l<i>.norm1, l<i>.norm2,
l<i>.mix.{q,dkv,dkv.norm,uk,uv,g,o}, l<i>.mlp.router and l<i>.mlp.e<j>.{gate,up,down} for every expert j.  Beside the gain of every
norm but dkv.norm stand <norm>.b and <norm>.alpha.
"""
from __future__ import annotations

import re

from ..config.bidinex import NAME, BidinexConfig
from ..config.registry import register_architecture
from .base import Architecture

_LAYER = re.compile(r"^layers\.(\d+)\.(.+)$")

_MIXER = {            # (parameter, piece) -> what follows "l<i>.mix."
    ("q_dkv", "q"): "q", ("q_dkv", "dkv"): "dkv", ("dkv_norm", None): "dkv.norm", ("uk", None): "uk", ("uv", None): "uv",
    ("gate", None): "g", ("o", None): "o",
}
_NORM = {"weight": "", "bias": ".b", "alpha": ".alpha"}
_IN_LAYER = {"feed_forward.router": "mlp.router"}
_IN_LAYER.update({f"{part}.{p}": name + suffix for part, name in (("mixer_norm", "norm1"), ("feed_forward_norm", "norm2"))
                  for p, suffix in _NORM.items()})
_TOP = {"embedding.weight": "embed", "embedding.norm": "embed.norm", "embedding.bias": "embed.norm.b",
        "embedding.alpha": "embed.norm.alpha", "stream_join.weight": "loop.in"}
_TOP.update({f"final_norm.{p}": "final.norm" + suffix for p, suffix in _NORM.items()})
_EXPERT_PIECE = re.compile(r"^e(\d+)\.(gate|up|down)$")


class Bidinex(Architecture):
    name = NAME
    config_class = BidinexConfig

    def checkpoint_name(self, path: str, piece: str | None) -> str:
        if path in _TOP and piece is None:
            return _TOP[path]
        m = _LAYER.match(path)
        if m:
            rest = m.group(2)
            if rest in _IN_LAYER and piece is None:
                return f"l{m.group(1)}." + _IN_LAYER[rest]
            if rest in ("feed_forward.expert_gate_up", "feed_forward.expert_down") and piece and _EXPERT_PIECE.match(piece):
                return f"l{m.group(1)}.mlp.{piece}"
            if rest.startswith("mixer.") and (rest[6:], piece) in _MIXER:
                return f"l{m.group(1)}.mix." + _MIXER[(rest[6:], piece)]
        raise KeyError(f"{NAME} has no checkpoint tensor for parameter {path!r} piece {piece!r}")


register_architecture(Bidinex())
