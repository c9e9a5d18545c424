"""A plain, slow restatement of the Dosuvik decoder, one function per mechanism.

Written from the design's equations with whole-sequence tensors and Python loops over time.  It
shares nothing with the engine (no cache, no pages, no kernels, no portions) and is the oracle of
the engine's tests.  `cfg` is the dictionary of a model's config.json, `w` maps tensor names to
tensors; all arithmetic runs in `dtype` (float64 by default).

Notation: S tokens of one sequence at positions 0..S-1, D the model width, x the residual stream.
"""

from __future__ import annotations

import torch


# ------------------------------------------------------------------------ norms
def root_mean_square(x, eps):
    return torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    """x over its root mean square (eps inside the root), times `weight`."""
    return x / root_mean_square(x, eps) * weight


def shifted_norm(x, weight, eps):
    """The layers' norm: the stored weight is what the factor exceeds one by."""
    return x / root_mean_square(x, eps) * (1.0 + weight)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# -------------------------------------------------------------------- positions
def angles(S, dims, base, dtype, first=0):
    """[S, dims / 2]: pair m of the token at position p turns by p * base^(-2 m / dims)."""
    pos = torch.arange(first, first + S, dtype=dtype)
    freq = torch.tensor([base ** (-2.0 * m / dims) for m in range(dims // 2)], dtype=dtype)
    return pos[:, None] * freq[None, :]


def rotate_halves(x, dims, base, first=0, sign=1.0):
    """x [S, heads, d]: entry m < dims/2 is paired with entry m + dims/2; entries from `dims` on
    pass.  `first`: the position of row 0; `sign` -1 turns the other way."""
    if dims == 0:
        return x
    half = dims // 2
    a = sign * angles(x.shape[0], dims, base, x.dtype, first)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a),
                      x[..., dims:]], dim=-1)


def rotate_neighbours(x, dims, base, first=0):
    """x [S, heads, d]: entry 2m is paired with entry 2m + 1, below `dims`."""
    if dims == 0:
        return x
    a = angles(x.shape[0], dims, base, x.dtype, first)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y = x.clone()
    y[..., 0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    y[..., 1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return y


# -------------------------------------------------------------------- attention
def masked_attention(q, k, v, scale, window=None, sink=None):
    """q [S, H, d], k [S, G, d], v [S, G, dv]; query head h reads key/value head h // (H / G).
    Position i sees j <= i, with `window` only those with i - j < window.  Softmax over the
    visible keys; with `sink` [H] the denominator holds exp(sink_h) as well."""
    S, H, _ = q.shape
    G, dv = k.shape[1], v.shape[2]
    out = torch.zeros((S, H, dv), dtype=q.dtype)
    ago = torch.arange(S)[:, None] - torch.arange(S)[None, :]
    seen = ago >= 0 if window is None else (ago >= 0) & (ago < window)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = torch.where(seen, s, torch.full_like(s, float("-inf")))
        m = s.max(dim=1, keepdim=True).values
        if sink is not None:
            m = torch.clamp(m, min=float(sink[h]))
        e = torch.exp(s - m)
        den = e.sum(dim=1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - m)
        out[:, h] = (e / den) @ v[:, g]
    return out


def window_attention(h, w, p, m, eps):
    """The 'attention' mixer: one RMS norm over all query rows and one over all key rows, rotation
    of the halves, values turned by their own position over their whole width and the heads'
    outputs turned back by the query's, a sliding window, a sink per head."""
    S = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(S, H, d)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(S, G, d)
    v = (h @ w[p + "v"].T).reshape(S, G, dv)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q, k = rotate_halves(q, dims, base), rotate_halves(k, dims, base)
    v = rotate_halves(v, dv, base)
    mask = m.get("mask")
    o = masked_attention(q, k, v, m["scale"], None if mask is None else mask["size"], w[p + "sink"])
    return rotate_halves(o, dv, base, sign=-1.0).reshape(S, H * dv) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    """Queries straight from the input, keys and values of every head from one normed latent per
    position, one rotated key part shared by the heads; causal softmax; a sigmoid gate per output
    element."""
    S = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = (h @ w[p + "q"].T).reshape(S, H, d + dr)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :r], w[p + "dkv.norm"], eps)
    turned = rotate_neighbours(down[:, None, r:], dr, base)                  # [S, 1, dr]
    k = torch.cat([(c @ w[p + "uk"].T).reshape(S, H, d), turned.expand(S, H, dr)], dim=-1)
    q = torch.cat([q[..., :d], rotate_neighbours(q[..., d:], dr, base)], dim=-1)
    v = (c @ w[p + "uv"].T).reshape(S, H, dv)
    o = masked_attention(q, k, v, m["scale"]).reshape(S, H * dv)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------- recurrence
def decayed_sum(q, k, v, decay):
    """q, k [S, H, d], v [S, H, dv], decay [H]: per head a matrix M [d, dv] from zero,
    M_t = decay * M_(t-1) + k_t v_t^T, o_t = M_t^T q_t."""
    S, H, d = q.shape
    M = torch.zeros((H, d, v.shape[2]), dtype=q.dtype)
    out = torch.zeros((S, H, v.shape[2]), dtype=q.dtype)
    for t in range(S):
        M = decay[:, None, None] * M + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (M * q[t][:, :, None]).sum(dim=1)
    return out


def retention(h, w, p, m, eps):
    """Rotated queries and keys (keys over the root of their width), the decayed sum with a
    constant per head, every head over its root mean square, a SiLU gate."""
    S = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    q = rotate_halves((h @ w[p + "q"].T).reshape(S, H, d), rot["dims"], rot["base"])
    k = rotate_halves((h @ w[p + "k"].T).reshape(S, H, d), rot["dims"], rot["base"]) * d ** -0.5
    v = (h @ w[p + "v"].T).reshape(S, H, dv)
    o = decayed_sum(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    o = (o / root_mean_square(o, eps)).reshape(S, H * dv)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixer(kind, h, w, p, m, eps):
    return {"attention": window_attention, "latent_attention": latent_attention,
            "retention": retention}[kind](h, w, p, m, eps)


# ----------------------------------------------------------------- feed-forward
def clamped_dense(h, w, p, mlp):
    """W_down (g sigmoid(1.702 g) (u + 1)), g = min(W_gate h, limit), u = W_up h within +-limit."""
    limit = mlp["limit"]
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choice_scores(scores, correction, groups):
    """[S, E]: what the choice of experts compares: sigmoid scores plus the correction, minus
    infinity outside the `keep` groups whose two best members have the largest sum."""
    choice = scores + correction
    if not groups:
        return choice
    S, E = choice.shape
    count, keep = groups["count"], groups["keep"]
    size = E // count
    out = torch.full_like(choice, float("-inf"))
    for t in range(S):
        sums = []
        for g in range(count):
            members = sorted(choice[t, g * size:(g + 1) * size].tolist(), reverse=True)
            sums.append(sum(members[:2]))
        for g in sorted(range(count), key=lambda g: (-sums[g], g))[:keep]:
            out[t, g * size:(g + 1) * size] = choice[t, g * size:(g + 1) * size]
    return out


def choose_experts(logits, correction, router):
    """-> (indices [S, top], weights [S, top]); weights are the plain scores of the chosen."""
    scores = sigmoid(logits)
    choice = choice_scores(scores, correction, router.get("groups"))
    idx = torch.sort(choice, dim=-1, descending=True, stable=True).indices[:, :router["top"]]
    return idx, torch.gather(scores, 1, idx)


def choice_margin(logits, correction, router):
    """[S]: how far a choice score would have to move before another expert is chosen: the gap
    between the last chosen and the best one left out, and between the last kept group and the
    first one dropped (halved: two members make the sum); infinite where nothing is left out."""
    scores = sigmoid(logits)
    groups, top = router.get("groups"), router["top"]
    choice = choice_scores(scores, correction, groups)
    S, E = choice.shape
    inf = torch.full((S,), float("inf"), dtype=logits.dtype)
    ordered = torch.sort(choice, dim=-1, descending=True).values
    gap = inf if top >= E else ordered[:, top - 1] - ordered[:, top]
    if groups and groups["keep"] < groups["count"]:
        size = E // groups["count"]
        raw = (scores + correction).reshape(S, groups["count"], size)
        sums = torch.sort(raw, dim=-1, descending=True).values[..., :2].sum(-1)
        sums = torch.sort(sums, dim=-1, descending=True).values
        gap = torch.minimum(gap, 0.5 * (sums[:, groups["keep"] - 1] - sums[:, groups["keep"]]))
    return gap


def expert_mixture(h, w, p, mlp, margins=None):
    """y_t = sum over the chosen experts of score * W_down (silu(W_gate h_t) * (W_up h_t))."""
    router = mlp["router"]
    logits = h @ w[p + "router"].T
    idx, wt = choose_experts(logits, w[p + "correction"], router)
    if margins is not None:
        margins.append(choice_margin(logits, w[p + "correction"], router))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(router["top"]):
            e = f"{p}e{int(idx[t, j])}."
            out[t] += wt[t, j] * (w[e + "down"] @ (silu(w[e + "gate"] @ h[t]) * (w[e + "up"] @ h[t])))
    return out


def feed_forward(h, w, p, mlp, margins=None):
    return clamped_dense(h, w, p, mlp) if mlp["kind"] == "dense" else expert_mixture(h, w, p, mlp, margins)


# ------------------------------------------------------------------------ model
def depth_average(results, coefficients):
    """The sum over j of coefficients[j] * results[j]."""
    return sum(c * x for c, x in zip(coefficients, results, strict=True))


def forward(cfg, w, tokens, dtype=torch.float64, streams=None, margins=None):
    """Logits [S, vocab] of one sequence.  `streams`: a list that receives the residual stream
    behind every layer (after the average over depth); `margins`: one that receives a tensor [S]
    per mixture of experts that ran (see `choice_margin`)."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    results = [x]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + shifted_norm(mixer(layer["type"], x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + shifted_norm(feed_forward(x, w, p + "mlp.", layer["mlp"], margins), w[p + "norm2"], eps)
        results.append(x)
        x = depth_average(results, w[p + "dwa"])
        if streams is not None:
            streams.append(x.clone())
    return shifted_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, weights, prompt, n_new, dtype=torch.float64):
    """Greedy continuation by recomputing the whole sequence for every new token."""
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(forward(cfg, weights, seq, dtype)[-1].argmax()))
    return seq[len(prompt):]
