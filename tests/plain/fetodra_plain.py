"""Plain, slow statement of the Fetodra design: one function per mechanism, whole sequences, no cache.
It shares no code with the package; the tests compare the engine with it.

Notation: h is a sublayer's input [T, width]; weights are [out, in]; positions count from 0 in a sequence;
N(y) = y / sqrt(mean(y^2) + eps) over the last axis.
A layer:   x <- N(alpha x + mixer(x)) (1 + norm1);   x <- N(alpha x + ff(x)) (1 + norm2)   (the second only with a feed-forward)
The model: x0 = embed[token]; layers in order; logits = head (N(x) (1 + final.norm)).
"""
from __future__ import annotations

import json
import os
import struct

import torch
import torch.nn.functional as F


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_{t - taps + 1 + j}, zeros before the first row."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))


# ------------------------------------------------------------------ attention
def rotate_pairs(x, dims, base):
    """x [T, heads, D]: coordinates 2i and 2i + 1 (i < dims / 2) turned by the angle p * base^(-2i / dims)."""
    T = x.shape[0]
    i = torch.arange(dims // 2, dtype=torch.float64)
    ang = torch.arange(T, dtype=torch.float64)[:, None] * (base ** (-2.0 * i / dims))[None, :]
    cos, sin = ang.cos().to(x.dtype)[:, None, :], ang.sin().to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def visible(T, size, keep_first):
    """[T, T]: position i (row) sees j when j <= i and (i - j < size or j < keep_first)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def capped(s, cap):
    return cap * torch.tanh(s / cap)


def project(h, w, name):
    """Product, bias, short convolution of one of q, k, v."""
    return causal_conv(h @ w[name].T + w[name + ".b"], w[name + ".conv"])


def keys_values(h, w, pre, m, eps):
    """(k [T, G, dim] normed over the whole projection and rotated, v [T, G, vdim] convolved only)."""
    T, G = h.shape[0], m["kv_heads"]
    k = rms(project(h, w, pre + "k"), eps) * w[pre + "k.norm"]
    k = rotate_pairs(k.view(T, G, m["dim"]), m["rot"]["dims"], m["rot"]["base"])
    return k, project(h, w, pre + "v").view(T, G, m["vdim"])


def queries(h, w, pre, m, eps):
    q = rms(project(h, w, pre + "q"), eps) * w[pre + "q.norm"]
    return rotate_pairs(q.view(h.shape[0], m["heads"], m["dim"]), m["rot"]["dims"], m["rot"]["base"])


def attend(q, k, v, m):
    """q [T, H, D] over k [T, G, D], v [T, G, V]: scaled, capped, masked, softmax."""
    T, H, rep = q.shape[0], m["heads"], m["heads"] // m["kv_heads"]
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = capped(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], m["softcap"])
    s = s.masked_fill(~visible(T, m["mask"]["size"], m["mask"]["keep_first"]), float("-inf"))
    return torch.einsum("hij,jhv->ihv", torch.softmax(s, dim=-1), v)


def attention(h, w, pre, m, eps, shared=None):
    """(output, (k, v)).  shared: the keys and values of the layer this one borrows them from."""
    T = h.shape[0]
    k, v = shared if shared is not None else keys_values(h, w, pre, m, eps)
    o = attend(queries(h, w, pre, m, eps), k, v, m).reshape(T, -1)
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T, (k, v)


# ------------------------------------------------------------------ Mamba-2
def state_space(x, B, C, dt, a_log, D):
    """x [T, H, V], B and C [T, H, N] (each head's group already picked), dt [T, H]:
    S <- exp(-exp(a_log) dt) S + dt B x^T;  y = S^T C + D x."""
    T, H, V = x.shape
    S = torch.zeros(H, B.shape[-1], V, dtype=x.dtype)
    out = torch.zeros_like(x)
    for t in range(T):
        decay = torch.exp(-torch.exp(a_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = torch.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t]
    return out


def gated_part_norm(y, z, weight, parts, eps):
    """y * silu(z), normed in equal parts, times the weight."""
    T = y.shape[0]
    return rms((y * F.silu(z)).view(T, parts, -1), eps).reshape(T, -1) * weight


def mamba2(h, w, pre, m, eps):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    p = h @ w[pre + "in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = F.silu(causal_conv(xbc, w[pre + "conv"]) + w[pre + "conv.b"])
    x = xbc[:, :inner].view(T, H, V)
    B = xbc[:, inner:inner + G * N].view(T, G, N).repeat_interleave(H // G, dim=1)
    C = xbc[:, inner + G * N:].view(T, G, N).repeat_interleave(H // G, dim=1)
    y = state_space(x, B, C, F.softplus(dt + w[pre + "dt_bias"]), w[pre + "A_log"], w[pre + "D"])
    return gated_part_norm(y.reshape(T, inner), z, w[pre + "norm"], m["norm_groups"], eps) @ w[pre + "o"].T


# ------------------------------------------------------------------ feed-forward and model
def clamped_ff(h, w, pre, limit):
    g = (h @ w[pre + "gate"].T).clamp(max=limit)
    u = (h @ w[pre + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def forward_layers(cfg, w, ids):
    """The stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.tensor(list(ids), dtype=torch.long)]
    kv, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            src = m.get("kv_from")
            y, kv[i] = attention(x, w, p + "mix.", m, eps, None if src is None else kv[src])
        else:
            y = mamba2(x, w, p + "mix.", m, eps)
        x = one_plus_norm(alpha * x + y, w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = one_plus_norm(alpha * x + clamped_ff(x, w, p + "mlp.", layer["mlp"]["limit"]), w[p + "norm2"], eps)
        after.append(x)
    return after


def forward_logits(cfg, w, ids):
    x = forward_layers(cfg, w, ids)[-1]
    return one_plus_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T


# ------------------------------------------------------------------ reading a model folder
_DT = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}


def load_model_dir(d, dtype=torch.float64):
    with open(os.path.join(d, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(d, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    w = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=_DT[e["dtype"]]) if b > a else torch.zeros(0)
        w[name] = t.reshape(e["shape"]).to(dtype)
    return cfg, w
