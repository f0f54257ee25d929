"""A plain, slow Gunulorn in float64 on the CPU: one function per mechanism, whole sequences only
(no cache, no state carried between calls, no batches).  It shares no code with the package;
the GPU tests hold the engine to it.

Notation: x [T, width] is the stream, h the normalised input of a sub-layer, W[name] the
checkpoint tensor of that name (linear weights [out, in], applied as h @ W.T)."""
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
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return unit_rms(x, eps) * w


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


def turn_pairs(x, angles):
    """x [T, heads, 2 n], angles [T, n]: elements 2i and 2i + 1 of a row turn by angles[:, i]."""
    c, s = angles.cos()[:, None, :], angles.sin()[:, None, :]
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)


def pair_angles(positions, base, dims):
    """[T, dims / 2]: p * base^(-2i / dims)."""
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    return positions.double()[:, None] * f[None, :]


def rotate_first(x, positions, rot):
    """The first rot.dims elements of every head turn, the rest pass."""
    dims = rot["dims"]
    if not dims:
        return x
    turned = turn_pairs(x[..., :dims], pair_angles(positions, rot["base"], dims))
    return torch.cat([turned, x[..., dims:]], dim=-1)


def rotate_values(v, positions, rot, back=False):
    """A whole value head turned by its token's position, or an output turned back by its own."""
    a = pair_angles(positions, rot["base"], v.shape[-1])
    return turn_pairs(v, -a if back else a)


def softmax_with_sink(scores, visible, sink):
    """exp(s) / (exp(sink) + sum of exp(s)) over the visible keys; scores [T, T] (query, key)."""
    s = scores.masked_fill(~visible, -math.inf)
    m = torch.maximum(s.max(-1, keepdim=True).values, torch.as_tensor(sink, dtype=s.dtype))
    e = torch.exp(s - m)
    return e / (torch.exp(sink - m) + e.sum(-1, keepdim=True))


def causal_mask(T):
    return torch.ones(T, T, dtype=torch.bool).tril()


def window_mask(T, size, keep_first):
    """Query i, key j <= i: the last ``size`` keys (i itself among them), and the first ``keep_first``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


# ----------------------------------------------------------------------------- mixers
def convolved(h, W, name):
    u = h @ W[name].T
    return past_convolution(u, W[name + ".conv"]) if name + ".conv" in W else u


def attention_keys_values(h, W, p, m):
    T = h.shape[0]
    k = convolved(h, W, p + "k").view(T, m["kv_heads"], m["dim"])
    return k, convolved(h, W, p + "v").view(T, m["kv_heads"], m["vdim"])


def attention(h, W, p, m, kv):
    """Convolved q against the given keys and values, one factor and one sink per head."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    k, v = kv
    q = convolved(h, W, p + "q").view(T, H, m["dim"])
    seen = causal_mask(T)
    out = []
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"] * W[p + "temp"][a]
        out.append(softmax_with_sink(s, seen, W[p + "sink"][a]) @ v[:, g])
    return torch.cat(out, dim=-1) @ W[p + "o"].T


def window_attention(h, W, p, m):
    """Rotated q, k and values, a window beside the first tokens, one more in the softmax's sum."""
    T = h.shape[0]
    H, G, n, nv, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    pos = torch.arange(T)
    q = rotate_first((h @ W[p + "q"].T).view(T, H, n), pos, rot)
    k = rotate_first((h @ W[p + "k"].T).view(T, G, n), pos, rot)
    v = rotate_values((h @ W[p + "v"].T).view(T, G, nv), pos, rot)
    seen = window_mask(T, m["mask"]["size"], m["mask"]["keep_first"])
    out = []
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"]
        out.append(softmax_with_sink(s, seen, 0.0) @ v[:, g])
    return rotate_values(torch.stack(out, dim=1), pos, rot, back=True).reshape(T, H * nv) @ W[p + "o"].T


# ----------------------------------------------------------------------------- feed-forward
def poly_norm(z, coefficients, eps):
    a, b, c, e = coefficients
    return a * unit_rms(z, eps) + b * unit_rms(z.pow(2), eps) + c * unit_rms(z.pow(3), eps) + e


def dense_ff(h, W, p, eps):
    z = h @ W[p + "up"].T + W[p + "up.b"]
    return poly_norm(z, W[p + "act"], eps) @ W[p + "down"].T + W[p + "down.b"]


def silu(z):
    return z * torch.sigmoid(z)


def route(h, W, p, r):
    """(expert numbers [T, top], their weights): the choice by score + correction, the weights by score."""
    s = torch.softmax(h @ W[p + "router"].T, dim=-1)
    idx = torch.topk(s + W[p + "correction"], r["top"], dim=-1).indices
    w = s.gather(1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20)


def experts(h, W, p, mlp):
    """The experts with tensors, then the ones whose output is their input."""
    idx, w = route(h, W, p, mlp["router"])
    n = mlp["router"]["experts"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(idx[t].tolist(), w[t]):
            if e >= n:
                out[t] += g * h[t]
                continue
            q = f"{p}e{e}."
            out[t] += g * (W[q + "down"] @ (silu(W[q + "gate"] @ h[t]) * (W[q + "up"] @ h[t])))
    return out


def feed_forward(h, W, p, mlp, eps):
    return dense_ff(h, W, p, eps) if mlp["kind"] == "dense" else experts(h, W, p, mlp)


# ----------------------------------------------------------------------------- the model
def layer(x, cfg, W, i, kept):
    """``kept``: the keys and values of the layers before, by layer; this layer's join it."""
    eps, spec, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    m = spec["mixer"]
    h = norm(x, W[p + "norm1"], eps)
    if spec["type"] == "attention":
        if m.get("kv_from") is None:
            kept[i] = attention_keys_values(h, W, p + "mix.", m)
        y = attention(h, W, p + "mix.", m, kept[m["kv_from"] if m.get("kv_from") is not None else i])
    elif spec["type"] == "attention_2":
        y = window_attention(h, W, p + "mix.", m)
    else:
        raise ValueError(spec["type"])
    if spec.get("mlp") is not None:
        y = y + feed_forward(norm(x, W[p + "norm2"], eps), W, p + "mlp.", spec["mlp"], eps)
    return x + y


def head(x, cfg, W):
    y = norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(y / cap) if cap else y


def forward(cfg, W, tokens, return_layers=False):
    """Logits [T, vocab] of one whole sequence (and, on request, the stream after every layer)."""
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kept, streams = {}, []
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, W, i, kept)
        streams.append(x)
    y = head(x, cfg, W)
    return (y, torch.stack(streams)) if return_layers else y


def logits(cfg, W, tokens):
    return forward(cfg, W, tokens)


def greedy(cfg, W, prompt, n):
    """n greedy tokens after ``prompt``; with each, the gap between the best and the second logit."""
    ids, out, gaps = list(prompt), [], []
    for _ in range(n):
        row = forward(cfg, W, ids)[-1]
        best = torch.topk(row, 2)
        out.append(int(best.indices[0]))
        gaps.append(float(best.values[0] - best.values[1]))
        ids.append(out[-1])
    return out, gaps
