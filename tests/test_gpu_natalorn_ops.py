"""GPU: every mechanism of the hyper-connected decoder (Natalorn) alone, against the plain restatement in oracle/natalorn_ref.py
(fp64).  Sizes are awkward on purpose (odd widths, head sizes and expert counts that are no multiple of a warp, a vector or a page;
pages handed out in reverse), and where random numbers would hide a fault (a window's edge, a chunk's border, a sink, a far key, a
group that must stay out) the inputs are made so that it shows."""
import pytest
import torch

pytestmark = pytest.mark.gpu

DEV = "cuda"


def _ops():
    from vllm_neuron_b200 import ops

    return ops


def _meta(entries, blocks, bs=8):
    from vllm_neuron_b200.hybrid import StepMeta

    return StepMeta.build(entries, blocks, bs, DEV)


def _err(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return (got - want).abs().max().item() / max(want.abs().max().item(), 1e-30)


def _close(got, want, tol):
    e = _err(got, want)
    assert e < tol, e


def _bf16_values(*shape, g, scale=1.0):
    """Random numbers that bf16 holds exactly: fp32 and bf16 pools then cache the same values."""
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).float()


# ------------------------------------------------------------------------------------------------ hyper-connections
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 9])
@pytest.mark.parametrize("width", [7, 60, 264, 2048, 5000])
def test_hyper_residual_mixes_all_copies_and_norms_the_next_input(S, width):
    """A branch that is a column range of wider rows, weighted expert rows, both, unweighted rows; a mix matrix that is far from
    symmetric; the stream stored or left alone."""
    from oracle.natalorn_ref import read_streams, rms_norm, write_streams

    ops = _ops()
    g = torch.Generator().manual_seed(100 * S + width)
    T, eps, top = 7, 1e-3, 3
    x = torch.randn(T, S, width, generator=g) * torch.logspace(-2, 1, T)[:, None, None]
    wide = torch.randn(T, width + 5, generator=g)
    rows, rw = torch.randn(T * top, width, generator=g), torch.rand(T, top, generator=g)
    mix, write, read = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    w = 1 + 0.3 * torch.randn(width, generator=g)
    dev = [t.to(DEV) for t in (mix, write, read, w)]
    wd = wide.to(DEV)
    ex = (rows.double().view(T, top, width) * rw.double()[:, :, None]).sum(1)
    cases = [(dict(y1=wd[:, 4:4 + width]), wide.double()[:, 4:4 + width]), (dict(y2=rows.to(DEV), nsum=top, y2_weight=rw.to(DEV)), ex),
             (dict(y1=wd[:, :width], y2=rows.to(DEV), nsum=top, y2_weight=rw.to(DEV)), ex + wide.double()[:, :width]),
             (dict(y1=wide[:, :width].contiguous().to(DEV), y2=rows.to(DEV), nsum=top),
              wide.double()[:, :width] + rows.double().view(T, top, width).sum(1))]
    X = x.double().transpose(0, 1)
    for terms, y in cases:
        new = write_streams(X, y, mix.double(), write.double())
        want = rms_norm(read_streams(new, read.double()), w.double(), eps)
        for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 6e-3)):
            xi = x.to(DEV)
            h = ops.hyper_residual(xi, *dev, eps, **terms, out_dtype=dt)
            assert h.dtype == dt
            _close(xi.transpose(0, 1), new, 2e-6)
            for t in range(T):
                _close(h[t], want[t], tol)
    xi = x.to(DEV)
    h2 = ops.hyper_residual(xi, *dev, eps, **cases[-1][0], out_dtype=torch.float32, store=False)
    assert torch.equal(xi.cpu(), x)
    _close(h2, want, 2e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S,width", [(1, 33), (2, 64), (3, 200), (6, 18)])
def test_hyper_embedding(dtype, S, width):
    from oracle.natalorn_ref import rms_norm

    ops = _ops()
    g = torch.Generator().manual_seed(S)
    table = torch.randn(19, width, generator=g).to(dtype)
    toks = torch.tensor([3, 18, 0, 7, 7], dtype=torch.int32)
    read, w = torch.randn(S, generator=g) - 2.0, torch.rand(width, generator=g)
    x, h = ops.hyper_embed(toks.to(DEV), table.to(DEV), S, read.to(DEV), w.to(DEV), 1e-4)
    e = table[toks.long()].double()
    assert x.shape == (5, S, width) and all(torch.equal(x[:, s].cpu().double(), e) for s in range(S))
    _close(h, rms_norm(e * read.double().sum(), w.double(), 1e-4), 3e-6 if dtype == torch.float32 else 6e-3)


# ------------------------------------------------------------------------------------------------ router
@pytest.mark.parametrize("E,top,count,keep", [(1, 1, 1, 1), (5, 2, 1, 1), (8, 4, 2, 1), (12, 3, 4, 2), (64, 8, 8, 3), (30, 7, 15, 6), (96, 33, 3, 3),
                                              (160, 20, 160, 40), (1000, 12, 50, 5)])
def test_grouped_router(E, top, count, keep):
    """Choice on score + correction inside the kept groups (most choice scores negative: an excluded group at zero would win), weights
    from the uncorrected scores; wide rows."""
    from oracle.natalorn_ref import choose_experts

    ops = _ops()
    g = torch.Generator().manual_seed(E + top)
    T = 41
    z = 2 * torch.randn(T, E + 3, generator=g)
    for corr in (0.3 * torch.randn(E, generator=g), -1.5 - torch.rand(E, generator=g), torch.zeros(E)):
        idx, wt = ops.moe_topk_grouped(z.to(DEV)[:, 2:2 + E], corr.to(DEV), top, groups=count, keep=keep, scale=1.7)
        wi, ws = choose_experts(z.double()[:, 2:2 + E], corr.double(), top, count, keep)
        assert (idx.cpu().sort(-1).values == wi.sort(-1).values).all()
        dense = torch.zeros(T, E, dtype=torch.float64).scatter_(1, wi, ws * 1.7)
        _close(torch.zeros(T, E, dtype=torch.float64).scatter_(1, idx.cpu().long(), wt.cpu().double()), dense, 3e-6)
    idx0, _ = ops.moe_topk_grouped(z.to(DEV)[:, 2:2 + E], None, top, groups=count, keep=keep)
    assert (idx0.cpu().sort(-1).values == wi.sort(-1).values).all()  # no correction = a zero one


@pytest.mark.parametrize("dtype,T", [(torch.float32, 9), (torch.bfloat16, 9), (torch.bfloat16, 300)])
def test_router_experts_and_shared_expert_together(dtype, T):
    from oracle.natalorn_ref import moe_ff

    from vllm_neuron_b200.hybrid import HybridCausalLM, HybridConfig, random_weights

    g = torch.Generator().manual_seed(T)
    for W, ff, sff, groups, keep in ((64, 32, 48, 3, 2), (42, 10, 7, 2, 1), (64, 40, 0, 1, 1)):
        mlp = {"kind": "moe", "router": {"experts": 6, "top": 2, "scale": 1.3, "groups": {"count": groups, "keep": keep}}, "expert": {"ff": ff},
               "shared": {"ff": sff} if sff else None}
        d = {"architecture": "Natalorn", "vocab": 20, "width": W, "norm": {"eps": 1e-6}, "streams": 2, "layers": [
            {"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.3, "mask": {"size": 4}}, "mlp": mlp}]}
        cfg = HybridConfig.from_dict(d)
        weights = random_weights(cfg, seed=3)
        m = HybridCausalLM(cfg, weights, num_blocks=3, max_num_seqs=1, max_model_len=64, dtype=dtype)
        h = torch.randn(T, W, generator=g).to(dtype)
        shared, pairs, wt = m._grouped_moe(m.layers[0], h.to(DEV))
        assert (shared is None) == (sff == 0)
        got = (pairs.view(T, 2, W) * wt[:, :, None]).sum(1) + (shared if shared is not None else 0)
        want = moe_ff(h.double(), {k: v.double() for k, v in weights.items()}, "l0.mlp.", mlp)
        _close(got, want, 2e-5 if dtype == torch.float32 else 3e-2)


# ------------------------------------------------------------------------------------------------ projection biases
@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,P,lead", [(5, 1, 9, 7, 3), (4, 2, 24, 12, 4), (6, 3, 10, 10, 0), (8, 2, 128, 64, 8)])
@pytest.mark.parametrize("norm", [False, "whole", "head"])
def test_projection_biases_join_before_norm_rotation_and_cache(kv_dtype, H, G, D, P, lead, norm):
    """Biases as large as the projections; also in front of a norm over the projection or per head and a rotation, which other
    designs combine them with."""
    from oracle.natalorn_ref import rms_norm, rotate_pairs

    from vllm_neuron_b200.hybrid import RotSpec

    ops = _ops()
    g = torch.Generator().manual_seed(H * D + P)
    bs, pos0, n, eps = 8, 29, 13, 1e-3
    cq, ck, cv = H * D, G * D, G * P
    rows = torch.randn(n, lead + cq + ck + cv + (1 if lead % 4 else 0), generator=g)
    bias = torch.randn(cq + ck + cv, generator=g)
    rot_n = 0 if not norm else D // 4 * 4
    cos, sin = (t.to(DEV) for t in RotSpec(rot_n, 300.0).tables(64)) if rot_n else (None, None)
    qn, kn = (1 + 0.3 * torch.randn(D if norm == "head" else c, generator=g) for c in (cq, ck))
    pages = [6, 5, 4, 3, 2, 1, 7]
    meta = _meta([(0, pos0, n)], {0: pages}, bs)
    k_pool = torch.zeros(8, G, bs, D, dtype=kv_dtype, device=DEV)
    v_pool = torch.zeros(8, G, bs, P, dtype=kv_dtype, device=DEV)
    kw = dict(q_norm=qn.to(DEV), k_norm=kn.to(DEV), eps=eps, head_norm=norm == "head", rot_n=rot_n, rot_half=False, cos=cos, sin=sin) if norm else {}
    q = ops.qk_norm_rope_kv_write(rows.to(DEV), lead, lead + cq, lead + cq + ck, H, k_pool, v_pool, meta, bias=bias.to(DEV), **kw)
    r = rows.double()[:, lead:lead + cq + ck + cv] + bias.double()

    def side(u, heads, w):
        if norm == "whole":
            u = rms_norm(u, w.double(), eps)
        u = u.reshape(n, heads, D)
        if norm == "head":
            u = rms_norm(u, w.double(), eps)
        return rotate_pairs(torch.cat([u.new_zeros(pos0, heads, D), u]), 300.0, rot_n)[pos0:] if rot_n else u

    _close(q, side(r[:, :cq], H, qn).reshape(n, -1), 3e-6)
    wk, wv = side(r[:, cq:cq + ck], G, kn), r[:, cq + ck:].reshape(n, G, P)
    tol = 3e-6 if kv_dtype == torch.float32 else 5e-3
    for i in range(n):
        p = pos0 + i
        _close(k_pool[pages[p // bs], :, p % bs], wk[i], tol)
        _close(v_pool[pages[p // bs], :, p % bs], wv[i], tol)


# ------------------------------------------------------------------------------------------------ window / chunk attention
def _cuts(T):
    """Whole (a tensor-core prompt kernel in bf16), token by token (the decode kernels), and ragged portions down to two tokens."""
    ragged, k = [], 0
    sizes = [2, 3, 17, 2, 40, 1, 1, 29, 64, 5]
    while sum(ragged) < T:
        ragged.append(min(sizes[k % len(sizes)], T - sum(ragged)))
        k += 1
    return {"whole": [T], "single": [1] * T, "ragged": ragged}


def _attend(q, k, v, scale, *, kv_dtype, portions, window=0, chunk=0, softcap=0.0, bs=8):
    """One sequence through the pools: q [T, H, D], k [T, G, D], v [T, G, P], cut into `portions`; pages in reverse order, in row 1 of
    the block table.  Returns outputs [T, H * P]."""
    ops = _ops()
    T, H, D = q.shape
    G, P = k.shape[1], v.shape[2]
    nb = -(-T // bs) + 1
    pages = list(range(nb - 1, 0, -1))
    k_pool = torch.zeros(nb, G, bs, D, dtype=kv_dtype, device=DEV)
    v_pool = torch.zeros(nb, G, bs, P, dtype=kv_dtype, device=DEV)
    table = torch.zeros(3, nb, dtype=torch.int32, device=DEV)
    table[1, :len(pages)] = torch.tensor(pages, dtype=torch.int32)
    rows = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=1).to(DEV)
    out, at = [], 0
    for n in portions:
        meta = _meta([(1, at, n)], {1: pages}, bs)
        part = rows[at:at + n]
        ops.kv_write_vmix(part, H * D, (H + G) * D, k_pool, v_pool, meta.slot_mapping)
        out.append(ops.swa_sink_attn(part, H, k_pool, v_pool, table, meta, None, scale, window or (1 << 30), chunk=chunk, softcap=softcap,
                                     split_p=True).float())
        at += n
    assert at == T
    return torch.cat(out)


def _loud(k, places):
    for j in places:
        k[j] *= 4
    return k.to(torch.bfloat16).float()


SHAPES = {"off_grid": (4, 2, 20, 36), "mma": (4, 2, 32, 48), "three_heads_on_one": (3, 1, 16, 16)}


@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [1, 2, 7, 16, 33, 64, None])
def test_sliding_window_at_every_edge(kv_dtype, shape, window):
    """Loud keys at page, tile and window borders: a window that is one position off moves late outputs by their whole size."""
    from oracle.natalorn_ref import grouped_attention, window_mask

    H, G, D, P = SHAPES[shape]
    g = torch.Generator().manual_seed((window or 0) + D)
    T, scale = 150, 0.4
    q, v = _bf16_values(T, H, D, g=g), _bf16_values(T, G, P, g=g)
    k = _loud(_bf16_values(T, G, D, g=g), (0, 31, 32, 64, 65, 100))
    dbl = [t.double() for t in (q, k, v)]
    want = grouped_attention(*dbl, scale, window_mask(T, window))
    if window:
        for off in {window + 1, max(window - 1, 1)} - {window}:
            assert _err(grouped_attention(*dbl, scale, window_mask(T, off)), want) > 0.2
    for name, portions in _cuts(T).items():
        got = _attend(q, k, v, scale, kv_dtype=kv_dtype, portions=portions, window=window)
        assert _err(got, want) < (2e-5 if kv_dtype == torch.float32 else 6e-3), name


@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("chunk,cap", [(1, 5.0), (7, 2.0), (32, 0.0), (50, 30.0), (64, 8.0), (None, 4.0)])
def test_capped_scores_inside_chunks(kv_dtype, shape, chunk, cap):
    """Loud keys on both sides of chunk borders (also where a border falls inside a page or a portion); scores far above the cap."""
    from oracle.natalorn_ref import chunk_mask, grouped_attention

    H, G, D, P = SHAPES[shape]
    g = torch.Generator().manual_seed((chunk or 0) + D)
    T, scale = 150, 0.5
    q, v = _bf16_values(T, H, D, g=g), _bf16_values(T, G, P, g=g)
    k = _loud(_bf16_values(T, G, D, g=g), (0, 6, 7, 31, 32, 49, 50, 63, 64, 99, 100, 128))
    dbl = [t.double() for t in (q, k, v)]
    want = grouped_attention(*dbl, scale, chunk_mask(T, chunk), cap)
    if chunk:
        assert _err(grouped_attention(*dbl, scale, chunk_mask(T, chunk + 1), cap), want) > 0.03
    if chunk != 1 and cap:
        assert _err(grouped_attention(*dbl, scale, chunk_mask(T, chunk), None), want) > 0.03
    for name, portions in _cuts(T).items():
        got = _attend(q, k, v, scale, kv_dtype=kv_dtype, portions=portions, chunk=chunk or 0, softcap=cap)
        assert _err(got, want) < (2e-5 if kv_dtype == torch.float32 else 6e-3), name


@pytest.mark.parametrize("H,G", [(4, 2), (3, 1), (2, 2)])
@pytest.mark.parametrize("kind,size", [("window", 40), ("window", 129), ("window", None), ("chunk", 128), ("chunk", 100), ("chunk", None)])
def test_wide_keys_narrow_values_on_the_tcgen05_prompt_kernel(H, G, kind, size):
    """Keys of 128 and values of 64 columns, pages of 32: whole prompts and portions cut off the tile grid."""
    from oracle.natalorn_ref import chunk_mask, grouped_attention, window_mask

    from vllm_neuron_b200 import _cabi

    assert _cabi.load().b200_swa_sink_attn_prefill_tc_supported(128, 64, 32, 1, 0, 0)
    g = torch.Generator().manual_seed((size or 0) + H)
    T, D, P, scale, cap = 391, 128, 64, 0.09, 6.0
    q, v = _bf16_values(T, H, D, g=g), _bf16_values(T, G, P, g=g)
    k = _loud(_bf16_values(T, G, D, g=g), (0, 99, 100, 127, 128, 255, 256, 300))
    if kind == "window":
        want, kw = grouped_attention(*(t.double() for t in (q, k, v)), scale, window_mask(T, size)), dict(window=size)
    else:
        want, kw = grouped_attention(*(t.double() for t in (q, k, v)), scale, chunk_mask(T, size), cap), dict(chunk=size or 0, softcap=cap)
    for portions in ([T], [130, 261], [2, 129, 1, 131, 128]):
        got = _attend(q, k, v, scale, kv_dtype=torch.bfloat16, portions=portions, bs=32, **kw)
        assert _err(got, want) < 6e-3, portions


# ------------------------------------------------------------------------------------------------ latent attention: window, sink, gate
def _latent(q, rows, C, scale, window, sink, *, kv_dtype, portions, bs=8):
    ops = _ops()
    T, H, K = q.shape
    nb = -(-T // bs) + 1
    pages = list(range(nb - 1, 0, -1))
    pool = torch.zeros(nb, 1, bs, K, dtype=kv_dtype, device=DEV)
    for p in range(T):
        pool[pages[p // bs], 0, p % bs] = rows[p].to(kv_dtype)  # a query must not see the later ones
    table = torch.zeros(3, nb, dtype=torch.int32, device=DEV)
    table[1, :len(pages)] = torch.tensor(pages, dtype=torch.int32)
    out, at = [], 0
    for n in portions:
        meta = _meta([(1, at, n)], {1: pages}, bs)
        out.append(ops.swa_sink_attn(q[at:at + n].reshape(n, -1).to(DEV), H, pool, None, table, meta, sink.to(DEV), scale, window or (1 << 30),
                                     latent_values=C).float())
        at += n
    return torch.cat(out)


@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,C,R", [(3, 20, 6), (4, 32, 16), (18, 48, 16), (1, 240, 32)])
@pytest.mark.parametrize("window", [1, 5, 33, 64, None])
def test_cached_latents_with_window_and_sink(kv_dtype, H, C, R, window):
    """Sinks from negligible to dominant per head (one left out, counted per warp or scaled would show), loud latents at window and
    tile borders, more heads than a tensor-core tile has rows."""
    from oracle.natalorn_ref import softmax_weights, window_mask

    g = torch.Generator().manual_seed(H * C + (window or 0))
    T, scale = 140, 0.3
    q = _bf16_values(T, H, C + R, g=g, scale=0.6)
    rows = _loud(_bf16_values(T, C + R, g=g, scale=0.6), (0, 31, 32, 63, 64, 90))
    sink = torch.linspace(-3, 4, H) if H > 1 else torch.tensor([1.5])

    def ref(win, sk):
        s = torch.einsum("thc,jc->htj", q.double(), rows.double()) * scale
        return torch.cat([softmax_weights(s[h], window_mask(T, win), sk[h].double()) @ rows[:, :C].double() for h in range(H)], dim=-1)

    want = ref(window, sink)
    assert _err(ref(window, sink - 50), want) > 0.1                           # the sink matters
    if window:
        assert _err(ref(window + 1, sink), want) > 0.03
    for name, portions in _cuts(T).items():
        got = _latent(q, rows, C, scale, window, sink, kv_dtype=kv_dtype, portions=portions)
        assert _err(got, want) < (2e-5 if kv_dtype == torch.float32 else 1e-2), name


def test_batched_per_head_linear_with_a_gate_per_column():
    ops = _ops()
    g = torch.Generator().manual_seed(9)
    for dtype, K, N, tol in ((torch.float32, 10, 7, 1e-5), (torch.bfloat16, 16, 24, 1e-2), (torch.bfloat16, 12, 5, 1e-2), (torch.bfloat16, 96, 150, 1e-2)):
        T, B = 37, 3
        a = torch.randn(T, B * K, generator=g).to(dtype)
        w = (torch.randn(B, N, K, generator=g) * K ** -0.5).to(dtype)
        gate = 2 * torch.randn(T, B * N + 2, generator=g)
        want = torch.einsum("tbk,bnk->tbn", a.double().view(T, B, K), w.double()).reshape(T, -1) * torch.sigmoid(gate[:, 2:].double())
        for ot in {dtype, torch.float32}:
            out = torch.zeros((T, B * N), dtype=ot, device=DEV)
            ops.batched_linear(a.to(DEV), w.to(DEV), out, a_batch_stride=K, out_batch_stride=N, gate=gate.to(DEV)[:, 2:], gate_cols=True)
            _close(out, want, tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,R,P,C,Q,dims", [(3, 10, 6, 7, 20, 12, 6), (4, 32, 16, 48, 64, 32, 16), (2, 16, 8, 24, 40, 56, 4)])
def test_latent_mixer_whole(dtype, H, D, R, P, C, Q, dims):
    """The mixer from its input rows to its output rows, in portions; fewer rotating columns than the rotated part has, too."""
    from oracle.natalorn_ref import latent_mixer

    from vllm_neuron_b200.hybrid import HybridCausalLM, HybridConfig, random_weights

    mix = {"heads": H, "dim": D, "rot_dim": R, "vdim": P, "kv_rank": C, "q_rank": Q, "scale": 0.4, "rot": {"dims": dims, "base": 70.0}, "mask": {"size": 21}}
    d = {"architecture": "Natalorn", "vocab": 20, "width": 64, "norm": {"eps": 1e-2}, "streams": 1,
         "layers": [{"type": "latent_attention", "mixer": mix, "mlp": None}]}
    cfg = HybridConfig.from_dict(d)
    weights = random_weights(cfg, seed=H)
    m = HybridCausalLM(cfg, weights, num_blocks=12, max_num_seqs=2, max_model_len=320, dtype=dtype)
    h = torch.randn(83, 64, generator=torch.Generator().manual_seed(1)).to(dtype)
    pages = [9, 2, 7]
    m.block_table[1, :3] = torch.tensor(pages, dtype=torch.int32)
    got, at = [], 0
    for n in (2, 40, 1, 1, 30, 9):
        got.append(m._latent_attention(m.layers[0], h[at:at + n].to(DEV).contiguous(), _meta([(1, at, n)], {1: pages}, 32), m.runs[0]["k_pool"]))
        at += n
    want = latent_mixer(h.double(), {k: v.double() for k, v in weights.items()}, "l0.mix.", mix, 1e-2)
    _close(torch.cat(got), want, 2e-5 if dtype == torch.float32 else 3e-2)
