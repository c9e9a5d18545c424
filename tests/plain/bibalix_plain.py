"""A plain, slow restatement of the Bibalix decoder, one function per mechanism.

Written from the design's equations with whole-sequence tensors and Python loops.  It shares nothing
with the engine (no cache, no pages, no kernels, no portions, no folding of one product into
another) and is the oracle of the engine's tests.  `cfg` is the dictionary of a model's config.json,
`w` maps tensor names to tensors; all arithmetic runs in `dtype` (float64 by default).

Notation: S tokens of one sequence at positions 0..S-1, D the model width, x the residual stream.
"""

from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------ norms
def root_mean_square(x, eps):
    return torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    """x over its root mean square (eps inside the root), times `weight`."""
    return x / root_mean_square(x, eps) * weight


def layer_norm(x, weight, bias, eps):
    """Mean off, over the root of the mean squared deviation + eps, times `weight`, plus `bias`."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * weight + bias


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# -------------------------------------------------------------------- positions
def turn_frequencies(rot):
    """-> (a frequency per pair, factor on sines and cosines).  Pair m turns by base^(-2m / dims) per
    position; with `scaling` the slow pairs turn `factor` times slower, with a ramp in between."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * m / dims) for m in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return plain, 1.0

    def place(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(place(sc["fast"])), 0)
    hi = min(math.ceil(place(sc["slow"])), dims - 1)
    out = []
    for m, f in enumerate(plain):
        r = min(max((m - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x, rot, first=0):
    """x [S, heads, d]: entry m < dims/2 is paired with entry m + dims/2; entries from `dims` on
    pass.  `first`: the position of row 0."""
    dims = rot["dims"]
    if dims == 0:
        return x
    freq, mag = turn_frequencies(rot)
    pos = torch.arange(first, first + x.shape[0], dtype=x.dtype)
    a = (pos[:, None] * torch.tensor(freq, dtype=x.dtype)[None, :])[:, None, :]
    c, s = torch.cos(a) * mag, torch.sin(a) * mag
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


# -------------------------------------------------------------------- attention
def visible(S, mask):
    """[S, S] booleans: i sees j <= i, with a mask only those with i - j < size or j < keep_first."""
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    seen = j <= i
    if mask is not None:
        seen &= (i - j < mask["size"]) | (j < mask.get("keep_first", 0))
    return seen


def softmax_attention(q, k, v, scale, seen):
    """One head: q [S, d], k [S, d], v [S, dv], seen [S, S]."""
    s = torch.where(seen, (q @ k.T) * scale, torch.tensor(float("-inf"), dtype=q.dtype))
    e = torch.exp(s - s.max(dim=1, keepdim=True).values)
    return (e / e.sum(dim=1, keepdim=True)) @ v


def second_map_factor(w, p, diff):
    """The number by which the second map is multiplied before it is taken off."""
    return (torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum())
            - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff)


def difference_of_maps(a1, a2, factor, diff, eps):
    """a1 - factor a2, over its root mean square, times 1 - diff."""
    o = a1 - factor * a2
    return o / root_mean_square(o, eps) * (1.0 - diff)


def two_map_attention(h, w, p, m, eps):
    """The 'attention' mixer: per head two queries and two keys (normed each, rotated) over the same
    values, a window beside the kept first tokens, the second map's output taken off the first's, a
    norm without a weight, a gate per head."""
    S = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(S, H * 2, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(S, G * 2, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(S, G, dv)
    q = rotate_halves(rms_norm(q, w[p + "q.norm"], eps), m["rot"])
    k = rotate_halves(rms_norm(k, w[p + "k.norm"], eps), m["rot"])
    seen = visible(S, m.get("mask"))
    factor = second_map_factor(w, p, m["diff"])
    gate = sigmoid(h @ w[p + "g"].T)
    out = torch.zeros((S, H, dv), dtype=h.dtype)
    for i in range(H):
        g = i // (H // G)
        a = [softmax_attention(q[:, 2 * i + n], k[:, 2 * g + n], v[:, g], m["scale"], seen) for n in (0, 1)]
        out[:, i] = difference_of_maps(a[0], a[1], factor, m["diff"], eps) * gate[:, i:i + 1]
    return out.reshape(S, H * dv) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    """The 'latent_attention' mixer: queries straight from the input, keys and values of every head
    from one normed latent per position, one rotated key part shared by the heads, a window, a gate
    per head."""
    S = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(S, H, d + dr)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :r], w[p + "dkv.norm"], eps)
    shared = rotate_halves(down[:, None, r:], m["rot"])[:, 0]                  # [S, dr]
    turned = rotate_halves(q[..., d:], m["rot"])
    k = (c @ w[p + "uk"].T).reshape(S, H, d)
    v = (c @ w[p + "uv"].T).reshape(S, H, dv)
    seen = visible(S, m.get("mask"))
    gate = sigmoid(h @ w[p + "g"].T)
    out = torch.zeros((S, H, dv), dtype=h.dtype)
    for i in range(H):
        qi = torch.cat([q[:, i, :d], turned[:, i]], dim=-1)
        ki = torch.cat([k[:, i], shared], dim=-1)
        out[:, i] = softmax_attention(qi, ki, v[:, i], m["scale"], seen) * gate[:, i:i + 1]
    return out.reshape(S, H * dv) @ w[p + "o"].T


def mixer(kind, h, w, p, m, eps):
    return {"attention": two_map_attention, "latent_attention": latent_attention}[kind](h, w, p, m, eps)


# ----------------------------------------------------------------- feed-forward
def gelu_dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p, limit):
    """W_down (g sigmoid(1.702 g) (u + 1)), g = min(W_gate h, limit), u = W_up h within +-limit."""
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose_experts(logits, router):
    """-> (indices [S, top], weights [S, top]): the largest softmax scores over all experts; the
    weights are these scores times the router's scale, not brought to a sum of one."""
    e = torch.exp(logits - logits.max(dim=-1, keepdim=True).values)
    scores = e / e.sum(dim=-1, keepdim=True)
    idx = torch.sort(scores, dim=-1, descending=True, stable=True).indices[:, :router["top"]]
    return idx, torch.gather(scores, 1, idx) * router.get("scale", 1.0)


def choice_margin(logits, router):
    """[S]: the gap, in logits, between the last chosen expert and the best one left out."""
    ordered = torch.sort(logits, dim=-1, descending=True).values
    top = router["top"]
    if top >= logits.shape[1]:
        return torch.full((logits.shape[0],), float("inf"), dtype=logits.dtype)
    return ordered[:, top - 1] - ordered[:, top]


def expert_mixture(h, w, p, mlp, margins=None):
    """The chosen experts' weighted sum, and a shared expert that every token passes times the
    sigmoid of one number per token."""
    router = mlp["router"]
    logits = h @ w[p + "router"].T
    idx, wt = choose_experts(logits, router)
    if margins is not None:
        margins.append(choice_margin(logits, router))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(router["top"]):
            out[t] += wt[t, j] * expert(h[t], w, f"{p}e{int(idx[t, j])}.", mlp["expert"]["limit"])
    shared = mlp.get("shared")
    if shared is not None:
        out = out + sigmoid(h @ w[p + "shared.sg"].reshape(1, -1).T) * expert(h, w, p + "shared.", shared["limit"])
    return out


def feed_forward(h, w, p, mlp, margins=None):
    return gelu_dense(h, w, p) if mlp["kind"] == "dense" else expert_mixture(h, w, p, mlp, margins)


# ------------------------------------------------------------------------ model
def forward(cfg, w, tokens, dtype=torch.float64, streams=None, margins=None):
    """Logits [S, vocab] of one sequence.  `streams`: a list that receives the residual stream
    behind every layer; `margins`: one that receives a tensor [S] per mixture of experts that ran
    (see `choice_margin`)."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        x = x + mixer(layer["type"], h, w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            h = layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps)
            x = x + feed_forward(h, w, p + "mlp.", layer["mlp"], margins)
        if streams is not None:
            streams.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T


def greedy(cfg, weights, prompt, n_new, dtype=torch.float64):
    """Greedy continuation by recomputing the whole sequence for every new token."""
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(forward(cfg, weights, seq, dtype)[-1].argmax()))
    return seq[len(prompt):]
