"""A plain, slow Ronolorn in float64 on the CPU: one function per mechanism, whole sequences only
(no cache, no state carried between calls, no batches).  It shares no code with the package;
the GPU tests hold the engine to it.

Notation: h [T, width] is the normalised input of a sub-layer, X [s, T, width] the streams, W[name]
the checkpoint tensor of that name (linear weights [out, in], applied as h @ W.T)."""
from __future__ import annotations

import json
import math
import os

import torch
from safetensors.torch import load_file


def load_folder(folder):
    with open(os.path.join(folder, "config.json")) as fh:
        cfg = json.load(fh)
    weights = {k: v.double() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}
    return cfg, weights


# ----------------------------------------------------------------------------- small pieces
def centred_norm(x, w, eps):
    """Mean taken off, divided by the standard deviation (eps under the root), times w."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def unit_length(x, eps=1e-6):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def past_convolution(u, w):
    """u [T, C], w [C, taps]: every channel's newest input times the last tap, the one before times
    the tap before, and so on; nothing comes before the first row."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def pair_frequencies(rot):
    """(one frequency per neighbouring pair, factor on cos and sin)."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def place(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(place(s["fast"])), 0)
    high = min(math.ceil(place(s["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def rotate_first(x, rot):
    """x [T, heads, dim]: neighbouring pairs among the first rot.dims elements turn by position times
    frequency, the rest pass."""
    if not rot or not rot["dims"]:
        return x
    f, magnitude = pair_frequencies(rot)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * f[None, :]
    c, s = (a.cos() * magnitude)[:, None, :], (a.sin() * magnitude)[:, None, :]
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2), x[..., rot["dims"]:]], dim=-1)


def window_mask(T, size):
    """Query i sees key j with 0 <= i - j < size."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & ((back < size) if size else True)


def softmax_over(scores, visible, one_more):
    """exp(s) / (sum of exp(s), plus one with ``one_more``) over the visible keys."""
    s = scores.masked_fill(~visible, -math.inf)
    m = s.max(-1, keepdim=True).values
    if one_more:
        m = m.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if one_more else 0.0))


def attend(q, k, v, scale, visible, one_more):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H vdim]."""
    share = q.shape[1] // k.shape[1]
    out = []
    for a in range(q.shape[1]):
        p = softmax_over((q[:, a] @ k[:, a // share].T) * scale, visible, one_more)
        out.append(p @ v[:, a // share])
    return torch.cat(out, dim=-1)


# ----------------------------------------------------------------------------- mixers
def delta_gates(h, W, p):
    """(decay, write strength), [T, heads] each."""
    raw = h @ W[p + "a"].T + W[p + "dt_bias"]
    decay = torch.exp(-torch.exp(W[p + "A_log"]) * torch.nn.functional.softplus(raw, threshold=1e9))
    return decay, torch.sigmoid(h @ W[p + "b"].T)


def delta_memory(q, k, v, decay, strength, state=None):
    """One head.  q, k [T, dim], v [T, vdim], decay, strength [T]: the memory fades, what it holds under
    the key is replaced (by the share ``strength``) by the value, and the query reads it.
    Returns ([T, vdim], the state after the last token)."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype) if state is None else state
    out = []
    for t in range(q.shape[0]):
        S = decay[t] * S
        S = S + torch.outer(k[t], strength[t] * (v[t] - S.T @ k[t]))
        out.append(S.T @ q[t])
    return torch.stack(out), S


def delta(h, W, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    part = {n: silu(past_convolution(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v")}
    q = unit_length(part["q"].view(T, G, m["dim"])) * m["dim"] ** -0.5
    k = unit_length(part["k"].view(T, G, m["dim"]))
    v = part["v"].view(T, H, m["vdim"])
    decay, strength = delta_gates(h, W, p)
    heads = [unit_rms(delta_memory(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], decay[:, a], strength[:, a])[0], eps)
             * W[p + "norm"] for a in range(H)]
    return (torch.cat(heads, dim=-1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def attention(h, W, p, m):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]

    def project(name, heads, size):
        return (h @ W[p + name].T + W[p + name + ".b"]).view(T, heads, size)

    q, k, v = project("q", H, m["dim"]), project("k", G, m["dim"]), project("v", G, m["vdim"])
    seen = window_mask(T, m["mask"]["size"])
    o = attend(rotate_first(q, m["rot"]), rotate_first(k, m["rot"]), v, m["scale"], seen, False)
    return o @ W[p + "o"].T + W[p + "o.b"]


def attention_2(h, W, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k = h @ W[p + "q"].T + W[p + "q.b"], h @ W[p + "k"].T + W[p + "k.b"]
    v = k.view(T, G, m["dim"])
    q, k = unit_rms(q, eps) * W[p + "q.norm"], unit_rms(k, eps) * W[p + "k.norm"]
    q, k = rotate_first(q.view(T, H, m["dim"]), m["rot"]), rotate_first(k.view(T, G, m["dim"]), m["rot"])
    return attend(q, k, v, m["scale"], window_mask(T, m["mask"]["size"]), True) @ W[p + "o"].T


def feed_forward(h, W, p):
    return torch.relu(h @ W[p + "up"].T).pow(2) @ W[p + "down"].T


# ----------------------------------------------------------------------------- the streams and the whole model
def streams_in(X, weights):
    return torch.einsum("s,stc->tc", weights, X)


def streams_out(X, y, mix, out):
    """mix [from, to]."""
    return torch.einsum("fo,ftc->otc", mix, X) + out[:, None, None] * y[None]


def mixer(h, W, p, layer, eps):
    if layer["type"] == "delta":
        return delta(h, W, p, layer["mixer"], eps)
    if layer["type"] == "attention":
        return attention(h, W, p, layer["mixer"])
    return attention_2(h, W, p, layer["mixer"], eps)


def forward(cfg, W, tokens, keep_layers=False):
    """Logits [T, vocab] (and the sum of the streams after every layer, [layers, T, width])."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    X = x[None].repeat(cfg["streams"], 1, 1)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = mixer(centred_norm(streams_in(X, W[p + "hc1.in"]), W[p + "norm1"], eps), W, p + "mix.", layer, eps)
        X = streams_out(X, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if layer.get("mlp") is not None:
            y = feed_forward(centred_norm(streams_in(X, W[p + "hc2.in"]), W[p + "norm2"], eps), W, p + "mlp.")
            X = streams_out(X, y, W[p + "hc2.mix"], W[p + "hc2.out"])
        after.append(X.sum(0))
    logits = centred_norm(X.sum(0), W["final.norm"], eps) @ W["embed"].T
    return (logits, torch.stack(after)) if keep_layers else logits


def logits(cfg, W, tokens):
    with torch.no_grad():
        return forward(cfg, W, tokens)


def greedy(cfg, W, prompt, count):
    """``count`` greedy tokens, and by how much each led the second best."""
    ids, out, gaps = list(prompt), [], []
    for _ in range(count):
        top = logits(cfg, W, ids)[-1].topk(2)
        out.append(int(top.indices[0]))
        gaps.append(float(top.values[0] - top.values[1]))
        ids.append(out[-1])
    return out, gaps
