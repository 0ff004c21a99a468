"""Grouped softmax attention over the paged cache whose projections pass a short causal convolution:

  q, k, v   u = W h + b, then y_t = sum_j w[:, j] u_(t - taps + 1 + j) on every channel (zeros before a sequence's start); the last
            taps - 1 projected rows of a request are state beside its pages
  norm      q, and k, divided by the root mean square over the WHOLE projection (all heads together), times a learned weight per channel
  rotation  the position part's interleaved frequencies on the first coordinates of every q and k head; v is neither normed nor rotated
  scores    s = scale * q . k, then softcap * tanh(s / softcap) (softcap None: s as it is); position i sees j <= i with
            i - j < window or j < keep_first (window None: all)
  output    o * sigmoid(W_g h) element by element, then W_o

  borrows_keys  the layer has no keys and values of its own: it reads the pages of an earlier step (ExecStep.cache_from) with its own
            queries, window and cap; its own state holds the convolution's inputs of q alone

One product makes q, k, v and the gate; one kernel adds the biases, convolves, norms, rotates and writes k and v into the step's pages
before attention runs; the gate is applied where attention writes its rows.  Norms, angles, scores and softmax are float32."""
from __future__ import annotations

import torch

from .attention import paged_attention_step_arrays
from .base import KVCacheNeed, Part, StateNeed, WeightSpec, pad_rows, register_mixer


@register_mixer("filtered_attention")
class FilteredAttention(Part):
    step_arrays_key = "paged_attention"
    keeps_states_when_borrowing = True

    def __init__(self, spec):
        super().__init__(spec)
        g = spec.get
        self.hidden, self.H, self.KV = int(g("hidden_size")), int(g("num_heads")), int(g("num_kv_heads"))
        self.D, self.V, self.scale, self.taps = int(g("key_dim")), int(g("value_dim")), float(g("scale")), int(g("conv_taps"))
        self.eps = float(g("norm_eps"))
        self.softcap = float(g("softcap")) if g("softcap") is not None else None
        self.window = int(g("window")) if g("window") is not None else None
        self.keep_first = int(g("keep_first", 0)) if self.window is not None else 0
        self.borrows = bool(g("borrows_keys", False))
        if self.H % self.KV:
            raise ValueError(f"{self.H} query heads are not a multiple of {self.KV} kv heads")
        if self.taps < 1:
            raise ValueError("filtered_attention needs at least one tap")
        # channels that pass the convolution: q, and k and v when they are the layer's own
        self.own_kv = 0 if self.borrows else self.KV
        self.C = self.H * self.D + self.own_kv * (self.D + self.V)
        self.proj = self.bias = self.conv = self.q_norm = self.k_norm = self.o = None

    def weight_specs(self):
        hid, rows = self.hidden, {"q": self.H * self.D, "k": self.KV * self.D, "v": self.KV * self.V}
        specs = []
        for n in ("q",) if self.borrows else ("q", "k", "v"):
            specs += [WeightSpec(n, (rows[n], hid)), WeightSpec(n + ".b", (rows[n],), kind="vector", init="zeros"),
                      WeightSpec(n + ".conv", (rows[n], self.taps), kind="vector")]
            if n != "v":
                specs.append(WeightSpec(n + ".norm", (rows[n],), kind="vector", init="norm"))
        return specs + [WeightSpec("g", (self.H * self.V, hid)), WeightSpec("o", (hid, self.H * self.V))]

    def cache_need(self):
        pages = KVCacheNeed(self.KV, self.D, self.window, value_dim=None if self.V == self.D else self.V, keep_first=self.keep_first)
        if self.taps == 1:
            return pages
        return pages, StateNeed(((self.taps - 1) * self.C,), "float32")

    def load(self, tensors, dtype, device):
        names = ("q",) if self.borrows else ("q", "k", "v")
        self.proj = pad_rows(torch.cat([tensors.pop(n) for n in names + ("g",)], dim=0), 8)         # one product: q | k | v | gate (| unused)
        self.bias = torch.cat([tensors.pop(n + ".b").float() for n in names]).contiguous()
        self.conv = torch.cat([tensors.pop(n + ".conv") for n in names], dim=0).to(dtype).contiguous()
        self.q_norm = tensors.pop("q.norm").float().contiguous()
        self.k_norm = None if self.borrows else tensors.pop("k.norm").float().contiguous()
        self.o = tensors.pop("o")

    step_arrays = staticmethod(paged_attention_step_arrays)

    @property
    def first_weight(self):
        return self.proj

    def step_flops(self, rows, pairs):
        return 2 * self.H * (self.D + self.V) * pairs

    def forward(self, h, ctx, cache, position, owns_cache=True):
        if owns_cache == self.borrows:
            raise ValueError("a layer reads an earlier step's pages exactly when it has no keys and values of its own")
        ops, H, KV, D, V = ctx.ops, self.H, self.KV, self.D, self.V
        meta = ctx.batch.group_view(cache.group, self.step_arrays_key)
        p = ops.linear(h, self.proj)
        own = not self.borrows
        q = ops.conv_qkv_cache(p, H, self.own_kv, D, V, self.bias, self.conv, self.taps, self.q_norm, self.k_norm, self.eps,
                               position.rotary_inv_freq(), cache.state, ctx.batch, meta, cache.k if own else None, cache.v if own else None)
        o = ops.masked_attention(q, cache.k, cache.v, meta, H, KV, D, V, self.scale, None, self.window, False, softcap=self.softcap,
                                 keep_first=self.keep_first, gate=p[:, self.C:self.C + H * V])
        return ops.linear(o, self.o)
