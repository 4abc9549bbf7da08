"""A plain, slow restatement of the Kobolix family in float64 torch: one function per mechanism, whole sequences at once, no
cache, nothing carried between calls.  It shares no code with the engine: it reads config.json and the checkpoint's tensors by
their names.  The tests compare the engine with it.

Notation: x [T, w] is the residual stream of one sequence (positions 0 .. T-1), N a root-mean-square norm with gain 1 + stored, c the
factor on every branch.  A layer is

    x += c * mixer(N1(x));   x += c * ff(N2(x))          (the second if the layer has a feed-forward)
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


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def stream_norm(x, w, name, eps):
    """The gain is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w[name])


def silu(z):
    return z * torch.sigmoid(z)


def embedding(tokens, w, cfg):
    return w["embed"][torch.tensor(tokens, dtype=torch.long)] * (cfg.get("embedding") or {"scale": 1.0})["scale"]


# ---- mixer: matrix memory with exponential gates ------------------------------------------------------------------
def memory_gates(h, w, p, cap):
    """(log input gate, log forget gate) [T, heads]."""
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    return i, f


def memory_walk(q, k, v, i, f):
    """q, k [T, D], v [T, V], i, f [T] of one head -> [T, V].  The state is kept divided by e^top, `top` the running maximum of
    what is in it, which starts at 0."""
    T, D, V = q.shape[0], q.shape[1], v.shape[1]
    S, n, top = torch.zeros(D, V, dtype=torch.float64), torch.zeros(D, dtype=torch.float64), 0.0
    out = torch.zeros(T, V, dtype=torch.float64)
    for t in range(T):
        new = max(float(f[t]) + top, float(i[t]))
        keep, add = math.exp(float(f[t]) + top - new), math.exp(float(i[t]) - new)
        top = new
        S = keep * S + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        out[t] = (q[t] @ S) / (max(abs(float(n @ q[t])), math.exp(-top)) + 1e-6)
    return out


def matrix_memory(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    i, f = memory_gates(h, w, p, float(m["gate_cap"]))
    o = torch.stack([memory_walk(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n]) for n in range(H)], dim=1)
    o = unit_rms(o, eps).reshape(T, H * V) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---- mixer: attention beside a gated delta rule -------------------------------------------------------------------
def rotate_neighbours(x, dims, base):
    """x [T, n, D]: of the leading `dims` numbers of each row 2i rotates with 2i + 1, by position * base^(-2i/dims)."""
    if not dims:
        return x
    T = x.shape[0]
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.arange(T, dtype=torch.float64).view(T, 1, 1) * f.view(1, 1, -1)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return out


def causal_softmax(s):
    T = s.shape[-1]
    hidden = torch.arange(T).view(1, T) > torch.arange(T).view(T, 1)
    return torch.softmax(s.masked_fill(hidden, float("-inf")), dim=-1)


def grouped_attention(h, w, p, m):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = (int(m["rot"]["dims"]), float(m["rot"]["base"])) if m.get("rot") else (0, 1.0)
    q = rotate_neighbours((h @ w[p + "q"].T).view(T, H, D), *rot)
    k = rotate_neighbours((h @ w[p + "k"].T).view(T, G, D), *rot).repeat_interleave(H // G, dim=1)
    v = (h @ w[p + "v"].T).view(T, G, V).repeat_interleave(H // G, dim=1)
    pr = causal_softmax(torch.einsum("ihd,jhd->hij", q, k) * m["scale"])
    return torch.einsum("hij,jhv->ihv", pr, v).reshape(T, H * V) @ w[p + "o"].T


def short_convolution(z, taps):
    """z [T, C], taps [C, n], the last tap the current token's."""
    T, n = z.shape[0], taps.shape[1]
    before = torch.cat([torch.zeros(n - 1, z.shape[1], dtype=z.dtype), z])
    return sum(before[j:j + T] * taps[:, j] for j in range(n))


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_walk(q, k, v, g, beta):
    """q, k [T, D], v [T, V], g, beta [T] of one head -> [T, V]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=torch.float64)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - k[t] @ S))
        out[t] = q[t] @ S
    return out


def delta_rule(h, w, p, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q = unit_vectors(q.view(T, G, D)).repeat_interleave(H // G, dim=1) * D ** -0.5
    k = unit_vectors(k.view(T, G, D)).repeat_interleave(H // G, dim=1)
    v = v.view(T, H, V)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * torch.nn.functional.softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = torch.stack([delta_walk(q[:, n], k[:, n], v[:, n], g[:, n], beta[:, n]) for n in range(H)], dim=1)
    o = unit_rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    a = unit_rms(grouped_attention(h, w, p + "left.", m["left"]), eps) * w[p + "left.out"]
    b = unit_rms(delta_rule(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (a + b)


MIXERS = {"mlstm": matrix_memory, "parallel": side_by_side}


# ---- feed-forward -------------------------------------------------------------------------------------------------
def gated(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, r):
    """(chosen experts, their weights) [T, top]: sigmoid scores, only experts of the best groups (a group is worth the sum of its
    two largest scores), the chosen scores times a constant."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    T, E = s.shape
    g = r.get("groups") or {"count": 1, "keep": 1}
    size = E // g["count"]
    worth = torch.topk(s.view(T, g["count"], size), min(2, size), dim=-1).values.sum(dim=-1)
    kept = torch.zeros(T, g["count"], dtype=torch.bool)
    kept.scatter_(1, torch.topk(worth, g["keep"], dim=-1).indices, True)
    open_ = kept.repeat_interleave(size, dim=1)
    chosen = torch.topk(s.masked_fill(~open_, -1.0), r["top"], dim=-1).indices
    return chosen, torch.gather(s, 1, chosen) * r.get("scale", 1.0)


def experts(h, w, p, mlp):
    chosen, weights = route(h, w, p, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t].tolist(), weights[t]):
            out[t] += c * gated(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out + gated(h, w, p + "shared.") if mlp.get("shared") else out


# ---- the model ----------------------------------------------------------------------------------------------------
def layer(x, w, i, lay, cfg):
    c, eps, p = cfg.get("residual_mult", 1.0), cfg["norm"]["eps"], f"l{i}."
    x = x + c * MIXERS[lay["type"]](stream_norm(x, w, p + "norm1", eps), w, p + "mix.", lay["mixer"], eps)
    if lay["mlp"] is not None:
        h = stream_norm(x, w, p + "norm2", eps)
        x = x + c * (gated(h, w, p + "mlp.") if lay["mlp"]["kind"] == "dense" else experts(h, w, p + "mlp.", lay["mlp"]))
    return x


def forward(cfg, w, tokens, layer_outputs=None):
    """Logits [T, vocab]; `layer_outputs`: a list that receives the stream after every layer."""
    x = embedding(tokens, w, cfg)
    for i, lay in enumerate(cfg["layers"]):
        x = layer(x, w, i, lay, cfg)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return stream_norm(x, w, "final.norm", cfg["norm"]["eps"]) @ w["embed"].T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
