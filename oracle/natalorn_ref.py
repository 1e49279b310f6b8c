"""Plain restatement of the Natalorn decoder (test infrastructure; nothing under vllm_neuron_b200/ imports it).

Natalorn keeps several copies of the residual stream and mixes them around every sublayer: with copies x_s, a read vector r, a mix
matrix M (M_st: how much of copy s goes into the next copy t) and a write vector o,
  u = sum_s r_s x_s;   y = sublayer(N(u));   next x_t = sum_s M_st x_s + o_t y
with N a plain RMS norm.  Mixers:
  * 'attention'        -- grouped-query softmax attention without positions, a sliding window;
  * 'attention_2'      -- the same with projection biases, tanh-capped scores and keys confined to the query's chunk;
  * 'latent_attention' -- queries through a normed latent, keys and values as up-projections of one normed latent per token plus
                          one rotated key part shared by the heads, a sliding window, a sink logit per head in the softmax
                          denominator, an elementwise sigmoid gate on the concatenated heads.
Feed-forward: SiLU experts; softmax scores over all experts, the choice made on score + correction among the experts of the best
groups, the scores themselves (times a constant, not renormalised) as weights on the outputs; a shared expert is added.
A run of layers may be repeated with the same weights.  One function per mechanism, whole sequences, no cache: a token's output
depends on earlier tokens only, so every way of cutting a sequence into engine steps must reproduce `forward` on the full list.
`dtype` float64 gives the reference values.  `cfg` is the configuration in its file form (a dict).
"""
from __future__ import annotations

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def rotate_pairs(x, base, dims):
    """x [T, ..., D], row t at position t: columns (2i, 2i + 1), 2i < dims, turn by t * base^(-2i / dims); the rest pass."""
    out = x.clone()
    t = torch.arange(x.shape[0], dtype=torch.float64).view(-1, *([1] * (x.dim() - 2)))
    for i in range(dims // 2):
        a = t * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_mask(T, size):
    """[T, T] bool: row i sees columns i - size + 1 .. i; size None: every column up to i."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size) if size else d >= 0


def chunk_mask(T, size):
    """Row i sees the columns of its own run of `size` positions (the first run starts at 0), up to i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i // size == j // size) if size else seen


def cap_scores(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def softmax_weights(s, seen, sink=None):
    """Softmax over the visible columns; sink (a number) adds exp(sink) to the denominator."""
    s = s.masked_fill(~seen, float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    return e / (den if sink is None else den + torch.exp(sink - top))


def grouped_attention(q, k, v, scale, seen, cap=None):
    """q [T, H, D], k [T, G, D], v [T, G, P] -> [T, H * P]; query head h reads key / value head h // (H / G)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    heads = []
    for h in range(H):
        s = cap_scores((q[:, h] @ k[:, h // rep].T) * scale, cap)
        heads.append(softmax_weights(s, seen) @ v[:, h // rep])
    return torch.cat(heads, dim=-1)


def attention_mixer(h, W, p, m, chunked):
    """'attention' (sliding window, no biases) or, with `chunked`, 'attention_2' (biases, capped scores, chunks)."""
    T, H, G, D, P = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ W[p + n].T + (W[p + n + ".b"] if chunked else 0) for n in "qkv")
    size = (m.get("mask") or {}).get("size")
    seen = chunk_mask(T, size) if chunked else window_mask(T, size)
    o = grouped_attention(q.view(T, H, D), k.view(T, G, D), v.view(T, G, P), m["scale"], seen, m.get("softcap") if chunked else None)
    return o @ W[p + "o"].T


def latent_mixer(h, W, p, m, eps):
    T, H, D, R, P, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).view(T, H, D + R)
    kv = h @ W[p + "dkv"].T
    c = rms_norm(kv[:, :C], W[p + "dkv.norm"], eps)
    k_rot, q_rot = rotate_pairs(kv[:, C:], base, dims), rotate_pairs(q[..., D:], base, dims)
    k, v = (c @ W[p + "uk"].T).view(T, H, D), (c @ W[p + "uv"].T).view(T, H, P)
    seen = window_mask(T, (m.get("mask") or {}).get("size"))
    heads = []
    for i in range(H):
        s = (q[:, i, :D] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        heads.append(softmax_weights(s, seen, W[p + "sink"][i]) @ v[:, i])
    return (torch.cat(heads, dim=-1) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def choose_experts(z, correction, top, count, keep):
    """Router logits [T, E] -> (chosen experts, their softmax scores), each [T, top].  The choice is made on score + correction;
    the experts form `count` equal runs of neighbours, ranked by their largest choice score, and only the best `keep` runs may
    be drawn from."""
    s = torch.softmax(z, dim=-1)
    choice = s + correction
    T, E = z.shape
    size = E // count
    best = choice.view(T, count, size).max(-1).values
    kept = torch.zeros(T, count, dtype=torch.bool)
    for t in range(T):
        kept[t, best[t].topk(keep).indices] = True
    choice = choice.masked_fill(~kept.repeat_interleave(size, dim=1), float("-inf"))
    idx = choice.topk(top, dim=-1).indices
    return idx, s.gather(1, idx)


def expert(h, W, p):
    return (silu(h @ W[p + ".gate"].T) * (h @ W[p + ".up"].T)) @ W[p + ".down"].T


def moe_ff(h, W, p, f):
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    idx, s = choose_experts(h @ W[p + "router"].T, W[p + "correction"], r["top"], g["count"], g["keep"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        y = expert(h, W, f"{p}e{e}")
        out = out + y * (s * (idx == e)).sum(-1, keepdim=True) * r.get("scale", 1.0)
    return out + expert(h, W, p + "shared") if f.get("shared") else out


def read_streams(X, r):
    """X [streams, T, width] -> the sublayer's input before its norm."""
    return sum(r[s] * X[s] for s in range(X.shape[0]))


def write_streams(X, y, M, o):
    n = X.shape[0]
    return torch.stack([sum(M[s, t] * X[s] for s in range(n)) + o[t] * y for t in range(n)])


def layer_runs(cfg):
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


def forward(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """tokens: list of ids -> logits [T, vocab].  streams: a list that receives the sum of the copies after every layer run."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    X = torch.stack([x] * int(cfg["streams"]))
    for i in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        h = rms_norm(read_streams(X, W[p + "hc1.in"]), W[p + "norm1"], eps)
        if L["type"] == "latent_attention":
            y = latent_mixer(h, W, p + "mix.", L["mixer"], eps)
        else:
            y = attention_mixer(h, W, p + "mix.", L["mixer"], L["type"] == "attention_2")
        X = write_streams(X, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if L.get("mlp"):
            h = rms_norm(read_streams(X, W[p + "hc2.in"]), W[p + "norm2"], eps)
            X = write_streams(X, moe_ff(h, W, p + "mlp.", L["mlp"]), W[p + "hc2.mix"], W[p + "hc2.out"])
        if streams is not None:
            streams.append(X.sum(0))
    return rms_norm(X.sum(0), W["final.norm"], eps) @ W["head"].T
