"""Kobolix: layers of matrix memory (a matrix state per head with exponential input gates and a running maximum beside it) and layers
in which causal grouped attention (neighbours rotate) and a gated delta rule behind short convolutions read the same input and their
normed outputs are averaged; dense silu-gated feed-forwards or routed ones (sigmoid scores, only experts of the best groups, a shared
expert beside them); norms in front of the sub-layers with gains stored around zero, one factor on every sub-layer's output.

Checkpoint tensor names: embed (also the output projection), final.norm, and for layer i: l<i>.norm1, l<i>.norm2, l<i>.mix.<name>,
l<i>.mlp.<name>.  Mixer tensors of the matrix memory: q, k, v, g, o, norm, i, i.b, f, f.b; of a parallel layer left.{q,k,v,o,out} and
right.{q,k,v,q.conv,k.conv,v.conv,g,b,a,A_log,dt_bias,norm,o,out}.  Feed-forward tensors: gate, up, down; routed: router,
e<j>.{gate,up,down} for every expert j and shared.{gate,up,down}.
"""
from __future__ import annotations

import re

from ..config.kobolix import NAME, KobolixConfig
from ..config.registry import register_architecture
from .base import Architecture

_LAYER = re.compile(r"^layers\.(\d+)\.(.+)$")

_MIXER = {            # (parameter, piece) -> what follows "l<i>.mix."
    ("qkvg", "q"): "q", ("qkvg", "k"): "k", ("qkvg", "v"): "v", ("qkvg", "g"): "g", ("gates", "i"): "i", ("gates", "f"): "f",
    ("gate_bias", "i"): "i.b", ("gate_bias", "f"): "f.b", ("norm", None): "norm", ("o", None): "o",
    ("left_qkv", "q"): "left.q", ("left_qkv", "k"): "left.k", ("left_qkv", "v"): "left.v", ("left_o", None): "left.o",
    ("right_qkvg", "q"): "right.q", ("right_qkvg", "k"): "right.k", ("right_qkvg", "v"): "right.v", ("right_qkvg", "g"): "right.g",
    ("right_conv", "q"): "right.q.conv", ("right_conv", "k"): "right.k.conv", ("right_conv", "v"): "right.v.conv",
    ("right_gates", "b"): "right.b", ("right_gates", "a"): "right.a", ("right_A_log", None): "right.A_log",
    ("right_dt_bias", None): "right.dt_bias", ("right_norm", None): "right.norm", ("right_o", None): "right.o",
    ("left_gain", None): "left.out", ("right_gain", None): "right.out",
}
_IN_LAYER = {
    ("mixer_norm.weight", None): "norm1", ("feed_forward_norm.weight", None): "norm2",
    ("feed_forward.gate_up", "gate"): "mlp.gate", ("feed_forward.gate_up", "up"): "mlp.up", ("feed_forward.down", None): "mlp.down",
    ("feed_forward.router", None): "mlp.router", ("feed_forward.shared_gate_up", "gate"): "mlp.shared.gate",
    ("feed_forward.shared_gate_up", "up"): "mlp.shared.up", ("feed_forward.shared_down", None): "mlp.shared.down",
}
_TOP = {"embedding.weight": "embed", "final_norm.weight": "final.norm"}
_EXPERT_PIECE = re.compile(r"^e(\d+)\.(gate|up|down)$")


class Kobolix(Architecture):
    name = NAME
    config_class = KobolixConfig

    def checkpoint_name(self, path: str, piece: str | None) -> str:
        if path in _TOP and piece is None:
            return _TOP[path]
        m = _LAYER.match(path)
        if m:
            rest = m.group(2)
            if (rest, piece) in _IN_LAYER:
                return f"l{m.group(1)}." + _IN_LAYER[(rest, piece)]
            if rest in ("feed_forward.expert_gate_up", "feed_forward.expert_down") and piece and _EXPERT_PIECE.match(piece):
                return f"l{m.group(1)}.mlp.{piece}"
            if rest.startswith("mixer.") and (rest[6:], piece) in _MIXER:
                return f"l{m.group(1)}.mix." + _MIXER[(rest[6:], piece)]
        raise KeyError(f"{NAME} has no checkpoint tensor for parameter {path!r} piece {piece!r}")


register_architecture(Kobolix())
