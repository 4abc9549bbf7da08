"""Tiny Bidinex configurations for the tests and a writer of random model folders for them.

The writer names the checkpoint's tensors itself (from the configuration alone), so the engine's mapping from its parameters to
tensor names is tested against it.  The configurations differ in everything a model of this family can vary: widths and vocabularies
that are no multiples of 8, layers of different sizes, head counts from one to nine, unrotated, rotated and value sizes that all
differ, latent rows narrower and wider than a head, experts (one, several chosen, all chosen), groups (none, one kept, all kept, as
many groups as experts), layers without a feed-forward, repeated runs at the start, in the middle, at the end or over the whole model,
walked once or several times, or no repetition, capped logits or none.  The attention scales are large on purpose: with a peaked
softmax one key too many or too few moves the logits far beyond any tolerance.
"""
import json
import os

import torch
from safetensors.torch import save_file


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
            "rot": {"dims": rot_dim, "base": base}}


def moe(experts, top, ff, groups=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(mixer, mlp):
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def config(width, vocab, eps, layers, mult, scale, loop=None, softcap=None):
    c = {"architecture": "Bidinex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
         "embedding": {"scale": scale}, "layers": layers}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if softcap is not None:
        c["logit_softcap"] = softcap
    return c


# the middle of the model repeated twice; one group of three kept; a repeated layer without a feed-forward; low cap
BID_A = config(64, 150, 1e-5, [
    layer(latent(3, 12, 8, 20, 24, 0.5, base=1000.0), moe(6, 2, 20, groups=(3, 1))),
    layer(latent(2, 8, 16, 8, 40, 0.4), None),
    layer(latent(5, 6, 4, 10, 16, 0.6, base=50.0), moe(4, 3, 12, groups=(4, 3))),
    layer(latent(1, 20, 12, 16, 12, 0.45), moe(5, 5, 16)),
], mult=0.7, scale=1.5, loop=(1, 3, 2), softcap=6.0)
# the end repeated three times; every group kept; one expert; odd sizes
BID_B = config(40, 77, 2e-5, [
    layer(latent(9, 6, 6, 7, 10, 0.7, base=300.0), moe(1, 1, 24)),
    layer(latent(4, 10, 2, 12, 9, 0.8), moe(8, 3, 10, groups=(2, 2))),
], mult=1.0, scale=1.0, loop=(1, 2, 3), softcap=25.0)
# one pass through the whole model (the stream join alone); no cap; groups of one expert
BID_C = config(100, 131, 1e-6, [
    layer(latent(2, 16, 8, 24, 32, 0.35, base=20.0), moe(6, 2, 33, groups=(6, 4))),
    layer(latent(6, 8, 2, 4, 8, 0.8), None),
], mult=0.45, scale=0.3, loop=(0, 2, 1))
# nothing repeated, no groups
BID_D = config(48, 90, 1e-5, [
    layer(latent(4, 8, 4, 12, 12, 0.5), moe(3, 1, 16)),
    layer(latent(2, 16, 8, 8, 48, 0.4, base=500.0), moe(2, 2, 8)),
], mult=0.25, scale=2.0, softcap=12.0)

CONFIGS = {"A": (BID_A, 51, 16), "B": (BID_B, 52, 8), "C": (BID_C, 53, 16), "D": (BID_D, 54, 4)}      # config, seed, page size


def make_tensors(cfg, seed, std=0.08):
    """{checkpoint name: bfloat16 tensor}."""
    g = torch.Generator().manual_seed(seed)

    def normal(*shape, s=std):
        return torch.randn(*shape, generator=g) * s

    w, t = cfg["width"], {}

    def norm(name, alpha):
        t[name], t[name + ".b"], t[name + ".alpha"] = 1.0 + normal(w, s=0.2), normal(w, s=0.15), torch.tensor(alpha)

    t["embed"] = normal(cfg["vocab"], w, s=1.0)
    norm("embed.norm", 0.9)
    norm("final.norm", 0.6)
    if cfg.get("loop"):
        t["loop.in"] = normal(w, 2 * w, s=w ** -0.5)
    for i, lay in enumerate(cfg["layers"]):
        m, p = lay["mixer"], f"l{i}.mix."
        H, D, R, V, C = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        norm(f"l{i}.norm1", 0.7 + 0.2 * i)
        t[p + "q"] = normal(H * (D + R), w, s=0.3)
        t[p + "dkv"], t[p + "dkv.norm"] = normal(C + R, w, s=0.3), 1.0 + normal(C, s=0.1)
        t[p + "uk"], t[p + "uv"] = normal(H * D, C, s=0.3), normal(H * V, C, s=0.2)
        t[p + "g"], t[p + "o"] = normal(H, w, s=0.3), normal(w, H * V, s=0.2)
        if lay["mlp"] is None:
            continue
        norm(f"l{i}.norm2", 1.1 - 0.2 * i)
        r, ff, q = lay["mlp"]["router"], lay["mlp"]["expert"]["ff"], f"l{i}.mlp."
        t[q + "router"] = normal(r["experts"], w, s=0.5)
        for e in range(r["experts"]):
            t[f"{q}e{e}.gate"], t[f"{q}e{e}.up"], t[f"{q}e{e}.down"] = normal(ff, w, s=0.2), normal(ff, w, s=0.2), normal(w, ff, s=0.2)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def plant_needle(cfg, t, needle, strength=4.0):
    """Changes the tensors so that every query of every layer scores the token `needle` far above all others, wherever it stands:
    channel 0 of the stream says "needle", channel 1 is the same for every token, neither is ever written by a sub-layer; the latent
    row of the needle is its first number alone, and every head's first unrotated query number reads channel 1."""
    t = {k: v.float().clone() for k, v in t.items()}
    w = cfg["width"]
    t["embed"][:, 0], t["embed"][:, 1] = 0.0, 4.0
    t["embed"][needle, 0] = 6.0
    for name in [n[:-6] for n in t if n.endswith(".alpha")]:
        t[name][:2], t[name + ".b"][:2], t[name + ".alpha"] = 1.0, 0.0, torch.tensor(1.0)
    if "loop.in" in t:
        t["loop.in"][:2] = 0.0
        t["loop.in"][0, 0] = t["loop.in"][1, 1] = 1.0
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", lay["mixer"]
        C, D, R = m["kv_rank"], m["dim"], m["rot_dim"]
        t[p + "dkv"][0] = 0.0
        t[p + "dkv"][0, 0] = 60.0
        t[p + "dkv.norm"][0] = 1.0
        q, uk = t[p + "q"].view(-1, D + R, w), t[p + "uk"].view(-1, D, C)
        q[:, 0], uk[:, 0], uk[:, :, 0] = 0.0, 0.0, 0.0
        q[:, 0, 1], uk[:, 0, 0] = strength, strength
        t[p + "o"][:2] = 0.0
        for n in t:
            if n.startswith(f"l{i}.mlp.e") and n.endswith(".down"):
                t[n][:2] = 0.0
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def write_model(cfg, out_dir, seed, std=0.08, tensors=None):
    os.makedirs(out_dir, exist_ok=True)
    save_file(tensors or make_tensors(cfg, seed, std), os.path.join(out_dir, "model.safetensors"))
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    return out_dir
