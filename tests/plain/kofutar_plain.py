"""Plain, slow statement of the Kofutar design: one function per mechanism, whole sequences, no cache.
It shares no code with the package; the tests compare the engine with it.

Notation: h is a mixer's input [T, width]; weights are [out, in]; positions count from 0 in a sequence;
L(y) = (y - mean) / sqrt(var + eps) * w (layer norm without a bias), N(y) = y / sqrt(mean(y^2) + eps) * w, both over the last axis.
A layer:   x <- x + L1b(mixer(L1(x)));   x <- x + L2b(ff(L2(x)))   (the second only with a feed-forward)
The model: x0 = embed[token]; layers in order, a span of them several times in a row, x <- W_in [x; x0] before every such pass;
           logits = head L_f(x).
"""
from __future__ import annotations

import json
import os
import struct

import torch
import torch.nn.functional as F


def layer_norm(x, w, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt(centred.pow(2).mean(-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


# ------------------------------------------------------------------ rotation
def rotate_half(x, dims, base, factor=1.0):
    """x [T, heads, D]: coordinates i and i + dims / 2 (i < dims / 2) turned by the angle p * base^(-2i / dims) / factor."""
    T, half = x.shape[0], dims // 2
    freq = base ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims) / factor
    ang = torch.arange(T, dtype=torch.float64)[:, None] * freq[None, :]
    cos, sin = ang.cos().to(x.dtype)[:, None, :], ang.sin().to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def rotated(x, rot):
    return rotate_half(x, rot["dims"], rot["base"], (rot.get("scaling") or {}).get("factor", 1.0))


# ------------------------------------------------------------------ softmax attention
def attend(q, k, v, scale, sink=None):
    """q [T, H, D], k [T, H, D], v [T, H, V] (each head's own keys already picked): causal softmax; sink [H]: one more term
    exp(sink_h) in the denominator."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(-1, T, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)[..., :T]
    return torch.einsum("hij,jhv->ihv", p, v)


def attention(h, w, pre, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm((h @ w[pre + "q"].T).view(T, H, m["dim"]), w[pre + "q.norm"], eps)
    k = rms_norm((h @ w[pre + "k"].T).view(T, G, m["dim"]), w[pre + "k.norm"], eps)
    v = (h @ w[pre + "v"].T).view(T, G, m["vdim"])
    q, k = rotated(q, m["rot"]), rotated(k, m["rot"])
    o = attend(q, k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1), m["scale"])
    return o.reshape(T, -1) @ w[pre + "o"].T


def latent_attention(h, w, pre, m, eps):
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    q = (cq @ w[pre + "uq"].T).view(T, H, D + R)
    ckr = h @ w[pre + "dkv"].T
    c = rms_norm(ckr[:, :C], w[pre + "dkv.norm"], eps)
    kr = rotated(ckr[:, None, C:], m["rot"]).expand(T, H, R)
    q = torch.cat([q[..., :D], rotated(q[..., D:], m["rot"])], dim=-1)
    k = torch.cat([(c @ w[pre + "uk"].T).view(T, H, D), kr], dim=-1)
    v = (c @ w[pre + "uv"].T).view(T, H, V)
    o = attend(q, k, v, m["scale"], w[pre + "sink"]).reshape(T, -1)
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ------------------------------------------------------------------ gated delta rule
def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_{t - taps + 1 + j}, zeros before the first row."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))


def unit(x, eps=1e-6):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + eps)


def delta_scan(q, k, v, beta, g):
    """q, k [T, H, D], v [T, H, V], beta, g [T, H]: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * F.softplus(a + dt_bias))


def delta(h, w, pre, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda n: F.silu(causal_conv(h @ w[pre + n].T, w[pre + n + ".conv"]))      # noqa: E731
    q = unit(conv("q").view(T, G, D)) * D ** -0.5
    k = unit(conv("k").view(T, G, D))
    v = conv("v").view(T, H, V)
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    g = decay(h @ w[pre + "a"].T, w[pre + "A_log"], w[pre + "dt_bias"])
    o = delta_scan(q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1), v, beta, g)
    o = rms_norm(o, w[pre + "norm"], eps).reshape(T, -1) * F.silu(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


# ------------------------------------------------------------------ feed-forward and model
def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh((2.0 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))


def dense_ff(h, w, pre):
    return (gelu_tanh(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "delta": delta}


def layer_runs(cfg):
    """[(layer, whether it opens a pass of the repeated span)] in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    span = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + span * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


def forward_layers(cfg, w, ids):
    """The stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.tensor(list(ids), dtype=torch.long)]
    x, after = x0, []
    for i, opens in layer_runs(cfg):
        if opens:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T
        layer, p = cfg["layers"][i], f"l{i}."
        y = MIXERS[layer["type"]](layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        x = x + layer_norm(y, w[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            x = x + layer_norm(dense_ff(layer_norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
        after.append(x)
    return after


def forward_logits(cfg, w, ids):
    return layer_norm(forward_layers(cfg, w, ids)[-1], w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T


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
