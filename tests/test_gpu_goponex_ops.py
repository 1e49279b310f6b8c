"""GPU: every mechanism of the layer-norm-after-the-sum decoder (Goponex) alone, against the plain restatement in
oracle/goponex_ref.py (fp64).  Sizes are awkward on purpose (odd widths, head and state sizes that are no multiple of a warp, a
vector or a page; pages handed out in reverse), and where random numbers would hide a fault (a window's edge, a kept token, a
far key) the inputs are made so that it shows."""
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


# ------------------------------------------------------------------------------------------------ residual step, activation
@pytest.mark.parametrize("width", [7, 60, 264, 2048, 5000])
def test_residual_step_with_layer_norm(width):
    """Both branches normed, one plain branch with a bias vector, no branch (the norm alone, the stream left as it is); branches
    that are column ranges of wider rows; a stream whose mean is large beside its spread."""
    from oracle.goponex_ref import layer_norm, rms_norm

    ops = _ops()
    g = torch.Generator().manual_seed(width)
    T, eps, alpha, c = 9, 1e-5, 2.3, 0.5
    x = torch.randn(T, width, generator=g) * 2 + 20
    wide = torch.randn(T, 2 * width + 5, generator=g) * torch.logspace(-3, 2, T)[:, None]
    w, w1, w2 = (1 + 0.3 * torch.randn(width, generator=g) for _ in range(3))
    vec = torch.randn(width, generator=g)
    wd = wide.to(DEV)
    a, b = wide[:, 3:3 + width], wide[:, width + 5:]
    dbl = lambda t: t.double()  # noqa: E731
    two = alpha * dbl(x) + c * (rms_norm(dbl(a), dbl(w1), eps) + rms_norm(dbl(b), dbl(w2), eps))
    cases = [(dict(y1=wd[:, 3:3 + width], w1=w1.to(DEV), y2=wd[:, width + 5:], w2=w2.to(DEV), c=c), two),
             (dict(y1=wd[:, 3:3 + width], vec=vec.to(DEV)), alpha * dbl(x) + dbl(a) + dbl(vec)),
             (dict(y1=a.contiguous().to(DEV), c=0.25), alpha * dbl(x) + 0.25 * dbl(a))]
    for terms, u in cases:
        want = layer_norm(u, dbl(w), eps)
        for dt, tol in ((torch.float32, 3e-5), (torch.bfloat16, 6e-3)):
            xi = x.to(DEV)
            h = ops.postln_residual(xi, alpha, w.to(DEV), eps, **terms, out_dtype=dt)
            assert h.dtype == dt
            _close(xi, want, 3e-5)
            _close(h, want, tol)
    xi = x.to(DEV)
    h = ops.postln_residual(xi, 1.0, w.to(DEV), eps, out_dtype=torch.float32, store=False)
    assert torch.equal(xi.cpu(), x)
    _close(h, layer_norm(dbl(x), dbl(w), eps), 3e-5)
    assert ops.postln_residual(xi, 1.0, w.to(DEV), eps) is None
    _close(xi, layer_norm(dbl(x), dbl(w), eps), 3e-5)


@pytest.mark.parametrize("n,ld,col0", [(5, 9, 3), (64, 64, 0), (320, 336, 8), (30, 32, 2)])
def test_bias_and_squared_relu(n, ld, col0):
    ops = _ops()
    g = torch.Generator().manual_seed(n)
    src, b = torch.randn(11, ld, generator=g) * 2, torch.randn(n, generator=g)
    z = src.double()[:, col0:col0 + n]
    for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 5e-3)):
        _close(ops.bias_act(src.to(DEV), col0, n, b.to(DEV), ops.ACT_RELU2, dt), torch.relu(z + b.double()) ** 2, tol)
        _close(ops.bias_act(src.to(DEV), col0, n, None, ops.ACT_NONE, dt), z, tol)


# ------------------------------------------------------------------------------------------------ per-head norm, rotation, values = keys
@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,rot_n,lead", [(5, 1, 24, 16, 3), (4, 2, 24, 12, 4), (3, 3, 10, 10, 0), (6, 2, 128, 32, 8), (2, 1, 36, 2, 1)])
def test_head_norm_rotation_and_values_from_keys(kv_dtype, H, G, D, rot_n, lead):
    """Heads of very different magnitude (a norm over the whole projection would show), neighbour pairs with YaRN frequencies of
    all three kinds, positions across page borders; the cached values are the raw keys."""
    from oracle.goponex_ref import rms_norm, rotate_pairs
    from vllm_neuron_b200.hybrid import RotSpec

    ops = _ops()
    g = torch.Generator().manual_seed(H * D + rot_n)
    bs, pos0, n, eps = 8, 37, 13, 1e-3
    sc = {"factor": 6.0, "original": 256, "fast": 16.0, "slow": 1.0}
    rot = {"dims": rot_n, "base": 300.0, "scaling": sc}
    rows = torch.randn(n, lead + H * D + G * D + (1 if lead % 4 else 0), generator=g)
    rows[:, lead:lead + H * D] *= torch.logspace(-2, 1, H).repeat_interleave(D)
    qn, kn = 1 + 0.3 * torch.randn(D, generator=g), 1 + 0.3 * torch.randn(D, generator=g)
    cos, sin = (t.to(DEV) for t in RotSpec(rot_n, 300.0, sc).tables(64))
    pages = [6, 5, 4, 3, 2, 1, 7]
    meta = _meta([(0, pos0, n)], {0: pages}, bs)
    k_pool = torch.zeros(8, G, bs, D, dtype=kv_dtype, device=DEV)
    v_pool = torch.zeros(8, G, bs, D, dtype=kv_dtype, device=DEV)
    k0 = lead + H * D
    q = ops.qk_norm_rope_kv_write(rows.to(DEV), lead, k0, k0, H, k_pool, v_pool, meta, q_norm=qn.to(DEV), k_norm=kn.to(DEV), eps=eps,
                                  rot_n=rot_n, rot_half=False, cos=cos, sin=sin, head_norm=True)
    r = rows.double()

    def turn(u, w):
        u = rms_norm(u, w.double(), eps)
        return rotate_pairs(torch.cat([u.new_zeros(pos0, *u.shape[1:]), u]), rot)[pos0:]

    rq, rk = r[:, lead:k0].reshape(n, H, D), r[:, k0:k0 + G * D].reshape(n, G, D)
    _close(q, turn(rq, qn).reshape(n, -1), 3e-6)
    wk = turn(rk, kn)
    tol = 3e-6 if kv_dtype == torch.float32 else 5e-3
    for i in range(n):
        p = pos0 + i
        _close(k_pool[pages[p // bs], :, p % bs], wk[i], tol)
        _close(v_pool[pages[p // bs], :, p % bs], rk[i], tol)


# ------------------------------------------------------------------------------------------------ window + kept first tokens
def _attend(q, k, v, scale, window, keep, *, kv_dtype, portions, bs=8):
    """One sequence through the pools: q [T, H, D], k [T, G, D], v [T, G, P], cut into `portions`; pages in reverse order, in row 1 of
    the block table.  Returns outputs [T, H, P]."""
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
        qd = ops.qk_norm_rope_kv_write(rows[at:at + n], 0, H * D, (H + G) * D, H, k_pool, v_pool, meta)
        out.append(ops.swa_sink_attn(qd, H, k_pool, v_pool, table, meta, None, scale, window or (1 << 30), split_p=True,
                                     keep=keep).float().view(n, H, P))
        at += n
    assert at == T
    return torch.cat(out)


def _cuts(T):
    """Whole (a tensor-core prompt kernel in bf16), token by token (the decode kernels), and ragged portions down to two tokens."""
    ragged, k = [], 0
    sizes = [2, 3, 17, 2, 40, 1, 1, 29, 64, 5]
    while sum(ragged) < T:
        ragged.append(min(sizes[k % len(sizes)], T - sum(ragged)))
        k += 1
    return {"whole": [T], "single": [1] * T, "ragged": ragged}


@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window,keep", [(9, 4), (16, 1), (44, 33), (1, 1), (33, 0), (64, 40), (7, 8), (5, 100), (None, 3)])
def test_window_with_kept_tokens_at_every_edge(kv_dtype, window, keep):
    """Loud keys sit on both sides of the window's edge of late queries and on the last kept and first lost token, so a window or a
    kept range that is one position off moves the output by its whole size.  All positions, whole, token by token, ragged."""
    from oracle.goponex_ref import window_keep_attention

    g = torch.Generator().manual_seed((window or 0) * 7 + keep)
    T, H, G, scale = 150, 4, 2, 0.4
    D, P = (20, 36) if kv_dtype == torch.float32 else (32, 48)
    q, k, v = _bf16_values(T, H, D, g=g), _bf16_values(T, G, D, g=g), _bf16_values(T, G, P, g=g)
    for j in {0, max(keep - 1, 0), min(keep, T - 1), 31, 32, 64, 65, 100}:    # also at page and tile borders
        k[j] *= 4
    k = k.to(torch.bfloat16).float()
    want = window_keep_attention(q.double(), k.double(), v.double(), scale, window, keep)
    if window:
        for wk in {(window + 1, keep), (max(window - 1, 1), keep), (window, keep + 1), (window, max(keep - 1, 0))} - {(window, keep)}:
            if keep < 100:                                                    # the edges matter for these inputs
                assert _err(window_keep_attention(q.double(), k.double(), v.double(), scale, *wk), want) > 0.03, wk
    for name, portions in _cuts(T).items():
        got = _attend(q, k, v, scale, window, keep, kv_dtype=kv_dtype, portions=portions)
        assert _err(got, want) < (2e-5 if kv_dtype == torch.float32 else 6e-3), (name, _err(got, want))


@pytest.mark.parametrize("H,G,D,window,keep", [(4, 2, 64, 100, 4), (3, 3, 128, 200, 0), (6, 2, 128, 130, 130), (2, 1, 64, 37, 190), (2, 2, 128, 700, 5),
                                               (5, 1, 64, 128, 128), (1, 1, 128, 257, 1)])
def test_long_prompts_on_the_tcgen05_kernel(H, G, D, window, keep):
    """Pages of 32 tokens, head sizes with a tcgen05 kernel, portions of 128 tokens and more: windows shorter and longer than a key
    step, kept tokens that end inside, at the end of and beyond the first key step; loud keys at every edge of late queries."""
    from oracle.goponex_ref import window_keep_attention

    g = torch.Generator().manual_seed(window + keep)
    T, scale = 640, 1.5 * D ** -0.5
    q, k, v = _bf16_values(T, H, D, g=g), _bf16_values(T, G, D, g=g), _bf16_values(T, G, D, g=g)
    for j in {0, max(keep - 1, 0), keep, 127, 128, 255, 256, 300, 500}:
        k[j] *= 4
    want = window_keep_attention(q.double(), k.double(), v.double(), scale, window, keep)
    for wk in {(window, keep - 1), (window, keep + 1), (window + 1, keep), (window - 1, keep)}:
        if window < T and wk[1] >= 0:                                         # the edges matter for these inputs
            assert _err(window_keep_attention(q.double(), k.double(), v.double(), scale, *wk), want) > 0.05, wk
    ops = _ops()
    with ops.kernel_timer() as kt:
        got = _attend(q, k, v, scale, window, keep, kv_dtype=torch.bfloat16, portions=[T], bs=32)
    assert any(n.startswith("swa_sink_attn_prefill_tc") for n in kt.summary())
    assert _err(got, want) < 6e-3, _err(got, want)
    got = _attend(q, k, v, scale, window, keep, kv_dtype=torch.bfloat16, portions=[131, 2, 200, 40, 128, 1, 1, 137], bs=32)
    assert _err(got, want) < 6e-3, _err(got, want)


@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
def test_a_kept_token_among_hundreds(kv_dtype):
    """700 positions behind a window of 24: token 2 is made to win for the late queries, in prompts and in decoding; token 5, just
    as loud, is not kept and must not be seen."""
    from oracle.goponex_ref import window_keep_attention

    g = torch.Generator().manual_seed(3)
    T, H, G, scale, window, keep = 700, 6, 3, 0.3, 24, 5
    D, P = (20, 36) if kv_dtype == torch.float32 else (48, 80)
    q, k, v = _bf16_values(T, H, D, g=g), _bf16_values(T, G, D, g=g), _bf16_values(T, G, P, g=g)
    for j in (2, 5):
        k[j] = 0
        k[j, :, 0] = 8.0
    q[600:, :, 0] = 8.0
    want = window_keep_attention(q.double(), k.double(), v.double(), scale, window, keep)
    assert (want[650, 0] - v[2, 0].double()).abs().max() < 0.2 * v[2, 0].abs().max()
    for name, portions in (("whole", [T]), ("prompt then single tokens", [640] + [1] * 60), ("ragged", [3, 2, 250, 1, 300, 144])):
        got = _attend(q, k, v, scale, window, keep, kv_dtype=kv_dtype, portions=portions)
        assert _err(got, want) < (2e-5 if kv_dtype == torch.float32 else 6e-3), (name, _err(got, want))


@pytest.mark.parametrize("kv_dtype", [torch.float32, torch.bfloat16])
def test_unequal_sequences_in_one_step_see_their_own_kept_tokens(kv_dtype):
    """Three sequences in one ragged step (a long portion that continues, a short prompt, a single decoded token), each with its own
    block-table row; every output equals the sequence run alone."""
    from oracle.goponex_ref import window_keep_attention

    ops = _ops()
    g = torch.Generator().manual_seed(8)
    H, G, D, P, scale, window, keep, bs = 4, 1, 32, 16, 0.35, 12, 3, 8
    lens, done = [90, 21, 57], [40, 0, 56]
    seqs = [tuple(_bf16_values(n, h, d, g=g) for h, d in ((H, D), (G, D), (G, P))) for n in lens]
    for _, k, _ in seqs:
        k[:keep] *= 4
    k_pool = torch.zeros(40, G, bs, D, dtype=kv_dtype, device=DEV)
    v_pool = torch.zeros(40, G, bs, P, dtype=kv_dtype, device=DEV)
    pages = {0: list(range(1, 13)), 1: list(range(39, 35, -1)), 2: list(range(20, 28))}
    table = torch.zeros(3, 40, dtype=torch.int32, device=DEV)
    for r, p in pages.items():
        table[r, :len(p)] = torch.tensor(p, dtype=torch.int32)

    def step(entries):
        rows = torch.cat([torch.cat([s[i][a:a + n].reshape(n, -1) for i in range(3)], dim=1) for r, a, n in entries for s in [seqs[r]]])
        meta = _meta(entries, pages, bs)
        qd = ops.qk_norm_rope_kv_write(rows.to(DEV), 0, H * D, (H + G) * D, H, k_pool, v_pool, meta)
        return ops.swa_sink_attn(qd, H, k_pool, v_pool, table, meta, None, scale, window, split_p=True, keep=keep).float()

    for r in (0, 2):
        step([(r, 0, done[r])])
    entries = [(r, done[r], lens[r] - done[r]) for r in range(3)]
    got, at = step(entries).view(-1, H, P), 0
    for r, a, n in entries:
        want = window_keep_attention(*(t.double() for t in seqs[r]), scale, window, keep)
        assert _err(got[at:at + n], want[a:a + n]) < (2e-5 if kv_dtype == torch.float32 else 6e-3), r
        at += n


# ------------------------------------------------------------------------------------------------ recurrences over a ragged batch
def _run_steps(steps, lens, launch):
    """steps: [{sequence: tokens}] over sequences of `lens` tokens; launch(entries, [(sequence, first, count)]) -> output rows of
    the step.  Returns per-sequence outputs."""
    at, got = {s: 0 for s in lens}, {s: [] for s in lens}
    for st in steps:
        entries = [(s, at[s], c) for s, c in st.items()]
        o, k = launch(entries), 0
        for s, c in st.items():
            got[s].append(o[k:k + c])
            at[s] += c
            k += c
    assert at == lens
    return {s: torch.cat(v) for s, v in got.items()}


SHORT = ({0: 75, 2: 40}, [{0: 2, 2: 1}, {0: 33, 2: 1}, {0: 1}, {0: 3, 2: 2}, {0: 14, 2: 36}, {0: 22}])
# portions of 256 tokens and more run as chained segments: from position 0, continuing, of no multiple of the segment, beside short ones
LONG = ({0: 1000, 1: 40, 3: 300}, [{0: 333, 1: 2}, {0: 1, 1: 1, 3: 300}, {0: 410, 1: 37}, {0: 256}])
PAGES = {s: list(range(1 + 200 * s, 200 + 200 * s)) for s in range(4)}


@pytest.mark.parametrize("x_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,N,lead", [(10, 3, 1), (70, 16, 0), (244, 24, 4), (33, 64, 2), (130, 20, 0), (20, 100, 0), (17, 200, 3), (8, 256, 0), (5, 1, 0)])
@pytest.mark.parametrize("lens,steps", [SHORT, LONG], ids=["short", "segments"])
def test_selective_scan_over_portions_slots_and_reuse(C, N, lead, x_dtype, lens, steps):
    """Raw step sizes and gate -> scan with gate, for sequences cut into portions beside each other (also steps of one to three
    tokens: the kernel without staging); stale slot states are loud; then a slot is taken over by a new sequence."""
    from oracle.goponex_ref import selective_scan

    ops = _ops()
    g = torch.Generator().manual_seed(C * 300 + N)
    A = -torch.exp(torch.rand(C, N, generator=g) * 3 - 2)
    bias, D = torch.randn(C, generator=g) - 2.5, torch.randn(C, generator=g)
    a_log2 = (A.double() / torch.log(torch.tensor(2.0, dtype=torch.float64))).float().to(DEV)
    state = torch.full((5, C, N), 55.0, device=DEV)
    pad = 0 if lead % 4 == 0 else 1

    def make(n):
        x = torch.randn(n, C, generator=g).to(x_dtype)
        wide = torch.randn(n, lead + 2 * N + 2 * C + pad, generator=g)         # [.. B | C | dt | z]: bc, dt and z share rows
        wide[:, lead + 2 * N:lead + 2 * N + C] *= 2
        return x, wide

    def cols(w):
        b0 = lead
        return w[:, lead + 2 * N:lead + 2 * N + C], w[:, lead + 2 * N + C:lead + 2 * N + 2 * C], w[:, b0:b0 + N], w[:, b0 + N:b0 + 2 * N]

    def want(x, w):
        dt, z, B, Cm = cols(w.double())
        y = selective_scan(x.double(), torch.nn.functional.softplus(dt + bias.double()), A.double(), B, Cm, D.double())
        return y * torch.nn.functional.silu(z)

    data = {s: make(L) for s, L in lens.items()}

    def launch(entries, src=None):
        src = src or data
        x = torch.cat([src[s][0][a:a + n] for s, a, n in entries]).to(DEV)
        w = torch.cat([src[s][1][a:a + n] for s, a, n in entries]).to(DEV)
        dt, z, _, _ = cols(w)
        meta = _meta(entries, PAGES)
        return ops.selective_scan(x, dt, w, lead, lead + N, z, a_log2, bias.to(DEV), D.to(DEV), state, meta).float()

    tol = 2e-5 if x_dtype == torch.float32 else 6e-3                           # bf16: the output's own rounding
    for s, got in _run_steps(steps, lens, launch).items():
        _close(got, want(*data[s]), tol)
    for s in set(range(5)) - set(lens):
        assert (state[s] == 55.0).all()                                        # other slots are not touched
    fresh = {0: make(9)}
    for n in (9, 3):                                                           # both kernels start a new sequence from zero
        _close(launch([(0, 0, n)], fresh), want(fresh[0][0][:n], fresh[0][1][:n]), tol)


def test_selective_scan_keeps_a_long_memory_and_needs_no_gate():
    """Tiny steps over 1500 tokens (decays of 0.9999), single-token steps between long portions: what the first token wrote is
    still there at the end."""
    from oracle.goponex_ref import selective_scan

    ops = _ops()
    g = torch.Generator().manual_seed(1)
    C, N, T = 24, 12, 1500
    A, bias = -torch.rand(C, N, generator=g) - 0.05, torch.full((C,), -9.0)
    x, w = torch.randn(T, C, generator=g), torch.randn(T, 2 * N + C, generator=g)
    x[0] *= 300
    dtr = w[:, 2 * N:]
    want = selective_scan(x.double(), torch.nn.functional.softplus(dtr.double() + bias.double()), A.double(), w[:, :N].double(),
                          w[:, N:2 * N].double(), torch.zeros(C, dtype=torch.float64))
    state = torch.zeros(2, C, N, device=DEV)
    outs, at = [], 0
    a_log2 = (A.double() * 1.4426950408889634).float().to(DEV)
    for c in [700] + [1] * 100 + [700]:
        xd, wd = x[at:at + c].to(DEV), w[at:at + c].to(DEV)
        outs.append(ops.selective_scan(xd, wd[:, 2 * N:], wd, 0, N, None, a_log2, bias.to(DEV), torch.zeros(C, device=DEV), state,
                                       _meta([(1, at, c)], {1: list(range(1, 200))})))
        at += c
    _close(torch.cat(outs), want, 5e-5)


@pytest.mark.parametrize("H,D,P,lead", [(2, 10, 7, 3), (3, 40, 72, 0), (1, 33, 20, 1), (2, 128, 31, 4), (1, 256, 16, 8), (4, 4, 5, 0), (1, 500, 3, 0), (2, 1, 1, 0)])
@pytest.mark.parametrize("lens,steps", [SHORT, LONG], ids=["short", "segments"])
def test_matrix_memory_over_portions_slots_and_reuse(H, D, P, lead, lens, steps):
    """Projections and raw gates -> running maximum, memory, normaliser, per-head norm and output gate.  Gates that swing between
    the caps move the maximum up and down (also below zero, where exp(-m) rules the denominator)."""
    from oracle.goponex_ref import log_gates, matrix_memory

    ops = _ops()
    g = torch.Generator().manual_seed(H * D + P)
    cap, eps, scale = 6.0, 1e-3, D ** -0.5
    ib, fb = torch.randn(H, generator=g), torch.randn(H, generator=g) + 2
    w = 1 + 0.3 * torch.randn(H * P, generator=g)
    width = lead + 2 * H * D + 2 * H * P + 2 * H + (-(lead + 2 * H) % 4 if lead % 4 == 0 and (H * P) % 2 == 0 else 1)
    k0, v0 = lead + H * D, lead + 2 * H * D
    g0, i0 = v0 + H * P, v0 + 2 * H * P
    state, m_state = torch.full((5, H, P + 1, D), 55.0, device=DEV), torch.full((5, H), 55.0, device=DEV)

    def make(n):
        r = torch.randn(n, width, generator=g)
        swing = torch.sin(torch.arange(n) / 9.0)[:, None] * 8
        r[:, i0:i0 + H] = 2 * r[:, i0:i0 + H] + swing - 2
        r[:, i0 + H:i0 + 2 * H] *= 3
        return r

    def want(raw):
        r = raw.double()
        Wg = {"i": torch.eye(H, dtype=torch.float64), "i.b": ib.double(), "f": torch.eye(H, dtype=torch.float64), "f.b": fb.double()}
        i, _ = log_gates(r[:, i0:i0 + H], Wg, "", cap)
        _, f = log_gates(r[:, i0 + H:i0 + 2 * H], Wg, "", cap)
        o = matrix_memory(r[:, lead:k0].reshape(-1, H, D) * scale, r[:, k0:v0].reshape(-1, H, D), r[:, v0:g0].reshape(-1, H, P), i, f)
        u = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps)
        return u.reshape(-1, H * P) * w.double() * torch.sigmoid(r[:, g0:i0])

    data = {s: make(L) for s, L in lens.items()}

    def launch(entries, src=None):
        rows = torch.cat([(src or data)[s][a:a + n] for s, a, n in entries]).to(DEV)
        o, nq, fl = ops.matrix_memory(rows, lead, k0, v0, i0, i0 + H, ib.to(DEV), fb.to(DEV), cap, state, m_state, _meta(entries, PAGES),
                                      H, D, P)
        return ops.matrix_memory_out(o, nq, fl, scale, rows, g0, w.to(DEV), eps, H, torch.float32)

    for s, got in _run_steps(steps, lens, launch).items():
        ref = want(data[s])
        # a denominator that passes near zero (|n . q| against the floor) amplifies fp32 rounding at single positions
        assert _err(got, ref) < 2e-4 and (got.double().cpu() - ref).pow(2).mean().sqrt().item() < 2e-5 * ref.pow(2).mean().sqrt().item()
    for s in set(range(5)) - set(lens):
        assert (state[s] == 55.0).all() and (m_state[s] == 55.0).all()
    fresh = {0: make(9)}
    _close(launch([(0, 0, 9)], fresh), want(fresh[0]), 2e-4)
    got = ops.matrix_memory_out(*(t.to(DEV) for t in (torch.randn(3, H * P, generator=g), torch.randn(3, H, generator=g), torch.rand(3, H, generator=g))),
                                scale, torch.randn(3, H * P, generator=g).to(DEV), 0, w.to(DEV), eps, H, torch.bfloat16)
    assert got.dtype == torch.bfloat16


def test_matrix_memory_maximum_starts_at_zero_and_is_carried():
    """Input gates far below zero: with a maximum that started at minus infinity the first token would carry weight 1; starting at
    zero it carries exp(i) and the denominator's floor is exp(-m) of the decayed maximum.  Then one loud input gate lifts the
    maximum for the rest of the sequence, across steps."""
    from oracle.goponex_ref import log_gates, matrix_memory

    ops = _ops()
    g = torch.Generator().manual_seed(4)
    H, D, P, T, cap = 2, 6, 4, 300, 20.0
    raw = torch.randn(T, 2 * H * D + H * P + 2 * H, generator=g)
    i0 = 2 * H * D + H * P
    raw[:, i0:i0 + H] -= 7
    raw[50, i0:i0 + H] = 12
    raw[:, i0 + H:] += 6
    zero = torch.zeros(H)
    Wg = {"i": torch.eye(H, dtype=torch.float64), "i.b": zero.double(), "f": torch.eye(H, dtype=torch.float64), "f.b": zero.double()}
    r = raw.double()
    i, f = log_gates(r[:, i0:i0 + H], Wg, "", cap)[0], log_gates(r[:, i0 + H:], Wg, "", cap)[1]
    want = matrix_memory(r[:, :H * D].reshape(T, H, D), r[:, H * D:2 * H * D].reshape(T, H, D), r[:, 2 * H * D:i0].reshape(T, H, P), i, f)
    state, m_state = torch.zeros(2, H, P + 1, D, device=DEV), torch.zeros(2, H, device=DEV)
    m, ms = torch.zeros(H, dtype=torch.float64), []
    for t in range(T):
        m = torch.maximum(f[t] + m, i[t])
        ms.append(m)
    outs, floors, at = [], [], 0
    for c in [20, 1, 1, 28, 1, 1, 248]:
        o, nq, fl = ops.matrix_memory(raw[at:at + c].to(DEV), 0, H * D, 2 * H * D, i0, i0 + H, zero.to(DEV), zero.to(DEV), cap, state, m_state,
                                      _meta([(1, at, c)], {1: list(range(1, 60))}), H, D, P)
        outs.append(o.view(c, H, P) / (torch.maximum(nq.abs(), fl) + 1e-6)[:, :, None])
        floors.append(fl)
        at += c
    assert want[:10].abs().max() < 0.05 * want[51:].abs().max()                # the first tokens' weights are exp(i), not 1
    _close(torch.cat(outs), want, 1e-4)
    _close(torch.cat(floors), torch.exp(-torch.stack(ms)), 2e-5)
