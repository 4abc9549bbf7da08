"""A plain, slow restatement of the Bidinex family in float64 torch: one function per mechanism, whole sequences at once, no
cache, nothing carried between calls.  It shares no code with the engine: it reads config.json and the checkpoint's tensors by
their names.  The tests compare the engine with it.

Notation: x [T, w] is the residual stream of one sequence (positions 0 .. T-1), x0 what the embedding made, N the squashing norm,
m the factor on every branch.  A layer is

    x += m * mixer(N1(x));   x += m * ff(N2(x))          (the second if the layer has a feed-forward)

and the layers start .. stop - 1 run `times` times in a row, each pass entered by x = W_in [x; x0].
"""
import json
import math
import os

import torch
from safetensors import safe_open


def read_model_dir(path):
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    w = {}
    with safe_open(os.path.join(path, "model.safetensors"), "pt") as f:
        for k in f.keys():
            w[k] = f.get_tensor(k).double()
    return cfg, w


def squash_norm(x, w, name):
    """tanh(alpha x) * gain + shift, number by number; alpha is one number."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rms_norm(x, gain, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def silu(z):
    return z * torch.sigmoid(z)


def embedding(tokens, w, cfg):
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    return squash_norm(x, w, "embed.norm")


def enter_pass(x, x0, w):
    """The stream that a pass through the repeated layers starts from."""
    return torch.cat([x, x0], dim=-1) @ w["loop.in"].T


def run_order(cfg):
    """[(layer, whether a pass starts right before it)]."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + \
        [(i, False) for i in range(b, n)]


# ---- mixer --------------------------------------------------------------------------------------------------------
def rotate_halves(v, dims, base):
    """v [T, n, D]: the leading `dims` numbers of each row rotate, i with i + dims/2, by position * base^(-2i/dims)."""
    T, half = v.shape[0], dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = torch.arange(T, dtype=torch.float64).view(T, 1, 1) * f.view(1, 1, half)
    u, t = v[..., :half], v[..., half:dims]
    return torch.cat([u * torch.cos(a) - t * torch.sin(a), t * torch.cos(a) + u * torch.sin(a), v[..., dims:]], dim=-1)


def causal_softmax(s):
    T = s.shape[-1]
    hidden = torch.arange(T).view(1, T) > torch.arange(T).view(T, 1)
    return torch.softmax(s.masked_fill(hidden, float("-inf")), dim=-1)


def latent_attention(h, w, p, m, eps):
    """Keys and values of all heads from one normed low-rank row, one rotated key part that the heads share, and a sigmoid
    gate of one number a head on the heads' outputs."""
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    latent = rms_norm(down[:, :C], w[p + "dkv.norm"], eps)
    rot = (int(m["rot"]["dims"]), float(m["rot"]["base"]))
    q_rot, k_rot = rotate_halves(q[..., D:], *rot), rotate_halves(down[:, C:].reshape(T, 1, R), *rot)[:, 0]
    k = (latent @ w[p + "uk"].T).view(T, H, D)
    v = (latent @ w[p + "uv"].T).view(T, H, V)
    s = (torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihr,jr->hij", q_rot, k_rot)) * m["scale"]
    o = torch.einsum("hij,jhv->ihv", causal_softmax(s), v)
    o = o * torch.sigmoid(h @ w[p + "g"].T).view(T, H, 1)
    return o.reshape(T, H * V) @ w[p + "o"].T


# ---- feed-forward -------------------------------------------------------------------------------------------------
def route(h, w, p, r):
    """(chosen experts, their weights) [T, top]: softmax scores, only experts of the best groups (a group is worth its largest
    score), the chosen scores divided by their sum."""
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    T, E = s.shape
    g = r.get("groups") or {"count": 1, "keep": 1}
    worth = s.view(T, g["count"], E // g["count"]).amax(dim=-1)
    kept = torch.zeros(T, g["count"], dtype=torch.bool)
    kept.scatter_(1, torch.topk(worth, g["keep"], dim=-1).indices, True)
    open_ = kept.repeat_interleave(E // g["count"], dim=1)
    chosen = torch.topk(s.masked_fill(~open_, -1.0), r["top"], dim=-1).indices
    weights = torch.gather(s, 1, chosen)
    return chosen, weights / (weights.sum(dim=-1, keepdim=True) + 1e-20)


def experts(h, w, p, r):
    chosen, weights = route(h, w, p, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t].tolist(), weights[t]):
            q = f"{p}e{e}."
            out[t] += c * (w[q + "down"] @ (silu(w[q + "gate"] @ h[t]) * (w[q + "up"] @ h[t])))
    return out


# ---- the model ----------------------------------------------------------------------------------------------------
def layer(x, w, i, lay, cfg):
    m = cfg["residual_mult"]
    x = x + m * latent_attention(squash_norm(x, w, f"l{i}.norm1"), w, f"l{i}.mix.", lay["mixer"], cfg["norm"]["eps"])
    if lay["mlp"] is not None:
        x = x + m * experts(squash_norm(x, w, f"l{i}.norm2"), w, f"l{i}.mlp.", lay["mlp"]["router"])
    return x


def head(x, w, cfg):
    z = squash_norm(x, w, "final.norm") @ w["embed"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z


def forward(cfg, w, tokens, layer_outputs=None):
    """Logits [T, vocab]; `layer_outputs`: a list that receives the stream after every layer run."""
    x = x0 = embedding(tokens, w, cfg)
    for i, starts in run_order(cfg):
        if starts:
            x = enter_pass(x, x0, w)
        x = layer(x, w, i, cfg["layers"][i], cfg)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return head(x, w, cfg)


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
