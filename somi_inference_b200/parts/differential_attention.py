"""Attention in two maps: every head has two softmaxes over the same values, and the second's output,
times a learned number, is taken off the first's.

Per token, with h the mixer's input:
    q = Wq h + bq, k = Wk h + bk, v = Wv h + bv; a head has two queries, a key/value head two keys, of
          `key_dim` elements each, side by side                       (`qkv_bias`)
    q, k: each divided by its root mean square (eps inside the root) and multiplied by a weight of
          that width which all heads and both maps share              (`head_norm`)
    q, k: entry i < dims / 2 is paired with entry i + dims / 2; the pair of the token at position p
          turns by p * base^(-2i / dims); entries from `dims` on pass (`rotary`)
    a_n, n = 1, 2: softmax of q_n.k_n * scale over the keys the mask leaves, times v: all earlier
          ones, or those at most `size` - 1 back together with the `keep_first` first ones
          (`mask` = {"kind": "window", "size", "keep_first"})
    factor = exp(lq1.lk1) - exp(lq2.lk2) + start, one number per layer from four vectors of key_dim
    d = a_1 - factor a_2;  head = d / sqrt(mean(d^2) + eps) * (1 - start), the mean over value_dim
    head i times sigmoid(Wg h)_i, one logit per head                  (`head_gate`)
    out = Wo heads
Query head i reads key/value head i // (heads / kv_heads).

One product makes q, k, v and the gate's logits; one kernel normalises, rotates and writes keys and
values to their pages, both keys of a head in one cache row; the attention kernel runs both maps
over the same key and value tiles and takes the difference from its float32 accumulators.  Norms,
scores, softmax, difference and gate are float32; angles are formed in float64.
"""

from __future__ import annotations

import torch

from .base import BuildContext, CacheNeeds, PagedKVNeeds, TensorDecl, names_of
from .linear import Linear
from .position import rotary_frequencies
from .registry import MIXERS


@MIXERS.register("differential_attention")
class DifferentialAttentionMixer:
    graph_safe = True
    FACTOR_PARTS = ("lq1", "lk1", "lq2", "lk2")

    @staticmethod
    def _sizes(params):
        return (int(params["num_heads"]), int(params["num_kv_heads"]), int(params["key_dim"]),
                int(params["value_dim"]))

    @staticmethod
    def declare(params) -> list[TensorDecl]:
        n = names_of(params)
        hidden = int(params["hidden_size"])
        heads, kv_heads, d, dv = DifferentialAttentionMixer._sizes(params)
        decl = []
        for part, rows in (("q", heads * 2 * d), ("k", kv_heads * 2 * d), ("v", kv_heads * dv)):
            decl.append(TensorDecl(n[part + "_weight"], (rows, hidden)))
            if params.get("qkv_bias"):
                decl.append(TensorDecl(n[part + "_bias"], (rows,), init="zeros", matrix=False))
        if params.get("head_norm"):
            decl += [TensorDecl(n["q_norm"], (d,), init="ones", matrix=False),
                     TensorDecl(n["k_norm"], (d,), init="ones", matrix=False)]
        decl += [TensorDecl(n[part], (d,), matrix=False) for part in DifferentialAttentionMixer.FACTOR_PARTS]
        if params.get("head_gate"):
            decl.append(TensorDecl(n["gate_weight"], (heads, hidden)))
        decl.append(TensorDecl(n["o_weight"], (hidden, heads * dv)))
        return decl

    def __init__(self, params, tensors, ctx: BuildContext) -> None:
        n = names_of(params)
        self.ctx = ctx
        self.heads, self.kv_heads, self.key_dim, self.value_dim = self._sizes(params)
        if self.kv_heads <= 0 or self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads cannot be grouped over {self.kv_heads} "
                             "key/value heads")
        if not (1 <= self.key_dim <= 256 and 1 <= self.value_dim <= 256):
            raise ValueError("key and value widths of 1 to 256 are supported")
        self.scale = float(params["scale"])
        self.eps = float(params["eps"])
        start = float(params["start"])
        self.gain = 1.0 - start
        lq1, lk1, lq2, lk2 = (tensors[n[part]].double() for part in self.FACTOR_PARTS)
        self.factor = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + start)
        mask = params.get("mask") or {}
        kind, size = mask.get("kind"), mask.get("size")
        if kind not in (None, "window") or (kind is not None and not (size and size > 0)):
            raise ValueError(f"unknown mask {mask!r} (kinds: 'window' with a size)")
        self.window = int(size) if kind == "window" else None
        self.keep_first = int(mask.get("keep_first", 0)) if kind == "window" else 0
        if self.keep_first < 0:
            raise ValueError("the number of kept first tokens cannot be negative")
        rotary = params.get("rotary") or {}
        self.rotary_dim = int(rotary.get("dims", 0))
        if self.rotary_dim % 2 or self.rotary_dim > self.key_dim:
            raise ValueError("rotary dims must be even and at most the key width")
        inv, self.magnitude = rotary_frequencies(rotary)
        self.inv_freq = inv.to(ctx.device)
        parts = ("q", "k", "v")
        bias = None
        if params.get("qkv_bias"):
            bias = torch.cat([tensors[n[p + "_bias"]].float() for p in parts], 0)
        weights = [tensors[n[p + "_weight"]] for p in parts]
        # the gate's logits are further columns of the same product (rows of zeros behind them keep its
        # rows a multiple of 16 bytes, which the tensor-core attention kernels need)
        self.gate_at = sum(w.shape[0] for w in weights)
        self.head_gate = bool(params.get("head_gate"))
        extra = self.heads if self.head_gate else 0
        extra += -(self.gate_at + extra) % 8
        if self.head_gate:
            weights.append(tensors[n["gate_weight"]])
        pad = self.gate_at + extra - sum(w.shape[0] for w in weights)
        weights.append(weights[0].new_zeros((pad, weights[0].shape[1])))
        if bias is not None and extra:
            bias = torch.cat([bias, torch.zeros(extra, dtype=bias.dtype, device=bias.device)])
        self.proj = Linear(torch.cat(weights, 0).contiguous(), bias, ctx.ops)
        self.q_norm = tensors[n["q_norm"]] if params.get("head_norm") else None
        self.k_norm = tensors[n["k_norm"]] if params.get("head_norm") else None
        self.out = Linear(tensors[n["o_weight"]], None, ctx.ops)

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(paged=PagedKVNeeds(
            self.kv_heads, 2 * self.key_dim, self.window,
            None if self.value_dim == 2 * self.key_dim else self.value_dim, self.keep_first))

    def forward(self, x: torch.Tensor, batch, cache, owns_cache: bool) -> torch.Tensor:
        ops, paged = self.ctx.ops, cache.paged
        qkv = self.proj(x)
        group = batch.groups[paged.group]
        ops.headnorm_rotary_store(qkv, batch.positions, self.inv_freq, 2 * self.heads, 2 * self.kv_heads,
                                  self.key_dim, self.value_dim, self.rotary_dim, self.q_norm, self.k_norm,
                                  self.eps, group.slot_map if owns_cache else None, paged.keys,
                                  paged.values, magnitude=self.magnitude, maps=2)
        out = torch.empty((x.shape[0], self.heads * self.value_dim), dtype=x.dtype, device=x.device)
        gate = qkv[:, self.gate_at:self.gate_at + self.heads] if self.head_gate else None
        ops.two_map_attention(qkv, paged.keys, paged.values, batch, group, self.heads, self.kv_heads,
                              self.key_dim, self.value_dim, self.scale, self.window, self.keep_first,
                              self.factor, self.eps, self.gain, gate, out, storage=paged.storage)
        partial = self.out.partial_sums(out)
        return partial if partial is not None else self.out(out)
