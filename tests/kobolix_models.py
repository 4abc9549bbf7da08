"""Tiny Kobolix configurations for the tests and a writer of random model folders for them.

The writer names the checkpoint's tensors itself (from the configuration alone), so the engine's mapping from its parameters to
tensor names is tested against it.  The configurations differ in everything a model of this family can vary: widths and vocabularies
that are no multiples of 8, layers of different sizes, head counts from one to six, key and value sizes that all differ, delta rules
with as many query heads as value heads or fewer, convolutions of one tap to nine, rotations of some, all or none of a head's numbers,
gate caps, experts (one chosen, several, all), groups (none, some kept, all kept, groups of one), with or without a shared expert and a
scale, layers without a feed-forward, factors and embedding scales of one or not.  The attention scales are large on purpose, the
memories' forget gates and the delta rules' decays close to one: a key too many or a state that is lost moves the logits far beyond any
tolerance.
"""
import json
import os

import torch
from safetensors.torch import save_file


def mlstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def parallel(left, right):
    """left = (heads, kv_heads, dim, vdim, scale, rot dims or None, base), right = (heads, kv_heads, dim, vdim, taps)"""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left))
    if left[5] is not None:
        l["rot"] = {"dims": left[5], "base": left[6]}
    return {"type": "parallel", "mixer": {"left": l, "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, scale=None, shared=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale is not None:
        r["scale"] = scale
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, eps, layers, mult=None, scale=None):
    c = {"architecture": "Kobolix", "width": width, "vocab": vocab, "norm": {"eps": eps},
         "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}
    if mult is not None:
        c["residual_mult"] = mult
    if scale is not None:
        c["embedding"] = {"scale": scale}
    return c


# every kind of layer; a layer without a feed-forward; two of three groups; a shared expert
KOB_A = config(64, 150, 1e-5, [
    (mlstm(3, 12, 20, 5.0), dense(40)),
    (parallel((4, 2, 16, 24, 0.8, 8, 1000.0), (4, 2, 12, 10, 3)), moe(6, 2, 20, groups=(3, 2), scale=1.3, shared=28)),
    (mlstm(2, 8, 6, 12.0), None),
    (parallel((2, 2, 8, 12, 1.0, 4, 50.0), (2, 2, 6, 16, 2)), dense(24)),
], mult=0.6, scale=2.0)
# odd sizes, heads of one, no rotation, a convolution of one tap, one expert of several, nothing optional given
KOB_B = config(40, 77, 2e-5, [
    (parallel((1, 1, 9, 7, 0.9, None, 0.0), (3, 1, 7, 5, 1)), moe(5, 1, 12)),
    (mlstm(1, 7, 5, 3.0), dense(18)),
    (mlstm(6, 5, 9, 8.0), moe(4, 4, 10, groups=(4, 4), scale=0.5)),
])
# sizes that the chunked kernels take; a whole head rotates; groups of one expert; a shared expert alone beside one choice
KOB_C = config(100, 131, 1e-6, [
    (mlstm(2, 32, 48, 15.0), dense(52)),
    (parallel((6, 3, 32, 16, 0.5, 32, 20.0), (4, 1, 64, 40, 4)), moe(6, 3, 24, groups=(6, 4), scale=2.0, shared=16)),
    (mlstm(3, 48, 24, 10.0), moe(3, 1, 33, shared=40)),
], mult=0.5, scale=1.0)
# wide heads, a long convolution, a parallel layer first and last
KOB_D = config(96, 90, 1e-5, [
    (parallel((3, 1, 24, 40, 0.7, 16, 500.0), (2, 2, 128, 72, 9)), dense(30)),
    (mlstm(1, 80, 136, 6.0), moe(8, 3, 16, groups=(2, 1), scale=1.1)),
    (parallel((2, 1, 16, 16, 0.8, 6, 1e6), (4, 2, 32, 24, 4)), None),
], mult=0.8, scale=3.0)

CONFIGS = {"A": (KOB_A, 61, 16), "B": (KOB_B, 62, 8), "C": (KOB_C, 63, 16), "D": (KOB_D, 64, 4)}      # config, seed, page size


def make_tensors(cfg, seed):
    """{checkpoint name: bfloat16 tensor}."""
    g = torch.Generator().manual_seed(seed)

    def normal(*shape, s=0.1):
        return torch.randn(*shape, generator=g) * s

    w, t = cfg["width"], {}
    t["embed"], t["final.norm"] = normal(cfg["vocab"], w, s=1.0), normal(w, s=0.2)
    for i, lay in enumerate(cfg["layers"]):
        m, p = lay["mixer"], f"l{i}.mix."
        t[f"l{i}.norm1"] = normal(w, s=0.2)
        if lay["type"] == "mlstm":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            t[p + "q"], t[p + "k"], t[p + "v"], t[p + "g"] = normal(H * D, w, s=0.2), normal(H * D, w, s=0.2), normal(H * V, w), normal(H * V, w)
            t[p + "i"], t[p + "f"] = normal(H, w, s=0.2), normal(H, w, s=0.1)
            t[p + "i.b"], t[p + "f.b"] = normal(H, s=1.0), 3.0 + normal(H, s=1.0)
            t[p + "norm"], t[p + "o"] = 1.0 + normal(H * V, s=0.2), normal(w, H * V, s=0.2)
        else:
            l, r = m["left"], m["right"]
            t[p + "left.q"], t[p + "left.k"] = normal(l["heads"] * l["dim"], w, s=0.2), normal(l["kv_heads"] * l["dim"], w, s=0.2)
            t[p + "left.v"], t[p + "left.o"] = normal(l["kv_heads"] * l["vdim"], w), normal(w, l["heads"] * l["vdim"], s=0.2)
            H, G, D, V, n = (r[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
            for name, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                t[p + "right." + name], t[p + f"right.{name}.conv"] = normal(rows, w, s=0.2), normal(rows, n, s=0.6)
            t[p + "right.b"], t[p + "right.a"], t[p + "right.g"] = normal(H, w, s=0.2), normal(H, w, s=0.1), normal(H * V, w)
            t[p + "right.A_log"], t[p + "right.dt_bias"] = normal(H, s=0.7) - 2.5, normal(H, s=0.5)
            t[p + "right.norm"], t[p + "right.o"] = 1.0 + normal(V, s=0.2), normal(w, H * V, s=0.2)
            t[p + "left.out"], t[p + "right.out"] = 1.0 + normal(w, s=0.2), 1.0 + normal(w, s=0.2)
        mlp, q = lay["mlp"], f"l{i}.mlp."
        if mlp is None:
            continue
        t[f"l{i}.norm2"] = normal(w, s=0.2)

        def glu(name, ff):
            t[name + "gate"], t[name + "up"], t[name + "down"] = normal(ff, w, s=0.15), normal(ff, w, s=0.15), normal(w, ff, s=0.15)
        if mlp["kind"] == "dense":
            glu(q, mlp["ff"])
            continue
        t[q + "router"] = normal(mlp["router"]["experts"], w, s=0.4)
        for e in range(mlp["router"]["experts"]):
            glu(f"{q}e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            glu(q + "shared.", mlp["shared"]["ff"])
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def plant_needle(cfg, t, needle):
    """Changes the tensors so that every mixer hangs on the token `needle` wherever it stands: channel 0 of the stream says "needle",
    channel 1 is the same for every token, neither is ever written by a sub-layer.  Attention scores the needle far above all others
    (an unrotated number of every head reads channel 1 in the query and channel 0 in the key); the matrix memories' input gates stand
    high for it and low for the others, and nothing is forgotten; the delta rules write it whole, the others hardly, and nothing decays."""
    t = {k: v.float().clone() for k, v in t.items()}
    t["embed"][:, 0], t["embed"][:, 1] = 0.0, 4.0
    t["embed"][needle, 0] = 8.0
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", lay["mixer"]
        for n in (f"l{i}.norm1", f"l{i}.norm2"):
            if n in t:
                t[n][:2] = 0.0
        if lay["type"] == "mlstm":
            t[p + "i"][:], t[p + "f"][:] = 0.0, 0.0
            t[p + "i"][:, 0], t[p + "i.b"][:], t[p + "f.b"][:] = 4.0, -3.0, 12.0
            for n in "qk":                 # every query reads every key with a part that is always the same: no state is read near zero
                x = t[p + n].view(m["heads"], m["dim"], -1)
                x[:, 0], x[:, 0, 1] = 0.0, 2.0
            t[p + "o"][:2] = 0.0
        else:
            l = m["left"]
            at = int(l["rot"]["dims"]) if l.get("rot") else 0
            assert at < l["dim"], "the needle needs a number that does not rotate"
            q, k = t[p + "left.q"].view(l["heads"], l["dim"], -1), t[p + "left.k"].view(l["kv_heads"], l["dim"], -1)
            q[:, at], k[:, at] = 0.0, 0.0
            q[:, at, 1], k[:, at, 0] = 4.0, 4.0
            t[p + "right.b"][:], t[p + "right.a"][:] = 0.0, 0.0
            t[p + "right.b"][:, 0], t[p + "right.b"][:, 1] = 6.0, -1.5
            t[p + "right.A_log"][:] = -12.0
            r = m["right"]
            for n in "qk":
                x, taps = t[p + "right." + n].view(r["kv_heads"], r["dim"], -1), t[p + f"right.{n}.conv"].view(r["kv_heads"], r["dim"], -1)
                x[:, 0], x[:, 0, 1], taps[:, 0] = 0.0, 2.0, 0.5
            t[p + "left.out"][:2], t[p + "right.out"][:2] = 0.0, 0.0
        for n in t:
            if n.startswith(f"l{i}.mlp.") and n.endswith("down"):
                t[n][:2] = 0.0
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def write_model(cfg, out_dir, seed, tensors=None):
    os.makedirs(out_dir, exist_ok=True)
    save_file(tensors or make_tensors(cfg, seed), os.path.join(out_dir, "model.safetensors"))
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    return out_dir
