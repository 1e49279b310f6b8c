"""Plain restatement of the Goponex decoder (test infrastructure; nothing under vllm_neuron_b200/ imports it).

Goponex is a decoder whose layers norm AFTER the sum, x <- LN(a x + mixer(x)), x <- LN(a x + ff(x)), with a layer norm that has
a weight and no bias; the sublayers read x itself.  Two mixers:
  * 'parallel' -- half the sum of two mixers over the same input, each RMS-normed over the width:
      left:  grouped-query attention whose values are the keys as projected (before norm and rotation), RMS norm per head on q
             and k, neighbour-pair rotary positions with YaRN-blended frequencies, a sliding window beside which the first few
             tokens of the sequence stay visible;
      right: a selective state-space scan with a step size per channel and a full [channel, state] decay matrix;
  * 'mlstm'    -- matrix memory with exponential input gates, stabilised by a running maximum, and a normaliser.
Feed-forward: squared-relu with biases.  One function per mechanism, whole sequences, no cache: a token's output depends on
earlier tokens only, so every way of cutting a sequence into engine steps must reproduce `forward` on the full list.
`dtype` float64 gives the reference values.  `cfg` is the configuration in its file form (a dict).
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def yarn_frequencies(rot):
    """(frequencies of the dims / 2 pairs, factor on cos and sin), float64.  Pairs that turn more than `fast` times within
    `original` positions keep their frequency, those below `slow` turns are slowed by `factor`, a linear ramp over the pair
    index lies between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(pair_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, rot):
    """x [T, heads, D]: columns 2i and 2i + 1 (2i < dims) turn by position * frequency i; the rest pass unchanged."""
    f, mag = yarn_frequencies(rot)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * f
    c, s = (torch.cos(a) * mag).to(x.dtype), (torch.sin(a) * mag).to(x.dtype)
    out = x.clone()
    for i in range(int(rot["dims"]) // 2):
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c[:, None, i] - v * s[:, None, i]
        out[..., 2 * i + 1] = v * c[:, None, i] + u * s[:, None, i]
    return out


def window_mask(T, size, keep):
    """[T, T] bool: row i sees column j.  size None or 0: every earlier token."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size:
        seen = seen & ((i - j < size) | (j < keep))
    return seen


def window_keep_attention(q, k, v, scale, size, keep):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]: softmax over the visible keys."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    seen = window_mask(T, size, keep)
    out = q.new_zeros(T, H, v.shape[2])
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        out[:, h] = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, h // rep]
    return out


def attention_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, G, D = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (h @ W[p + "q"].T).view(T, H, D)
    k = (h @ W[p + "k"].T).view(T, G, D)
    v = k
    q, k = rms_norm(q, W[p + "q.norm"], eps), rms_norm(k, W[p + "k.norm"], eps)
    if m.get("rot"):
        q, k = rotate_pairs(q, m["rot"]), rotate_pairs(k, m["rot"])
    mask = m.get("mask") or {}
    o = window_keep_attention(q, k, v, float(m["scale"]), mask.get("size"), int(mask.get("keep_first") or 0))
    return o.reshape(T, -1) @ W[p + "o"].T


def short_conv(x, w, b):
    """x [T, C], w [C, taps] (last column: the current token): causal convolution per channel plus bias, then silu."""
    taps = w.shape[1]
    xp = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    y = sum(xp[j:j + x.shape[0]] * w[:, j] for j in range(taps)) + b
    return y * torch.sigmoid(y)


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, inner]; A [inner, N]; B, C [T, N]; D [inner]:  S <- exp(dt A) S + dt x B^T,  y = S C + D x."""
    S = x.new_zeros(A.shape)
    y = torch.empty_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba_mixer(h, W, p, m):
    inner, rank, N = int(m["inner"]), int(m["dt_rank"]), int(m["state"])
    xz = h @ W[p + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = short_conv(x, W[p + "conv"], W[p + "conv.b"])
    xp = x @ W[p + "x"].T
    dt, B, C = xp[:, :rank], xp[:, rank:rank + N], xp[:, rank + N:]
    dt = torch.nn.functional.softplus(dt @ W[p + "dt"].T + W[p + "dt.b"], threshold=1e9 if h.dtype == torch.float64 else 20)
    y = selective_scan(x, dt, -torch.exp(W[p + "A_log"]), B, C, W[p + "D"])
    return (y * z * torch.sigmoid(z)) @ W[p + "o"].T


def parallel_mixer(h, W, p, m, eps):
    l = rms_norm(attention_mixer(h, W, p + "left.", m["left"], eps), W[p + "left.out"], eps)
    r = rms_norm(mamba_mixer(h, W, p + "right.", m["right"]), W[p + "right.out"], eps)
    return 0.5 * (l + r)


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, D] (already scaled), v [T, H, P], log gates i, f [T, H] -> o [T, H, P].  The running maximum starts at 0."""
    T, H, D = q.shape
    S, n, m = q.new_zeros(H, D, v.shape[2]), q.new_zeros(H, D), q.new_zeros(H)
    o = torch.empty_like(v)
    for t in range(T):
        m1 = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - m1), torch.exp(i[t] - m1)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        m = m1
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = torch.einsum("hdp,hd->hp", S, q[t]) / den[:, None]
    return o


def log_gates(h, W, p, cap):
    i = cap * torch.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = cap * torch.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap)
    return i, -torch.log1p(torch.exp(-f))


def mlstm_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, D, P = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ W[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, D)
    v = (h @ W[p + "v"].T).view(T, H, P)
    i, f = log_gates(h, W, p, float(m["gate_cap"]))
    o = matrix_memory(q, k, v, i, f)
    o = (o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, H * P) * W[p + "norm"]
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def squared_relu_ff(h, W, p):
    u = torch.relu(h @ W[p + "up"].T + W[p + "up.b"])
    return (u * u) @ W[p + "down"].T + W[p + "down.b"]


def forward(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """tokens: list of ids -> logits [T, vocab].  streams: a list that receives x after every layer."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    for n, L in enumerate(cfg["layers"]):
        p = f"l{n}."
        y = parallel_mixer(x, W, p + "mix.", L["mixer"], eps) if L["type"] == "parallel" else mlstm_mixer(x, W, p + "mix.", L["mixer"], eps)
        x = layer_norm(alpha * x + y, W[p + "norm1"], eps)
        if L.get("mlp"):
            x = layer_norm(alpha * x + squared_relu_ff(x, W, p + "mlp."), W[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.clone())
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T
