"""CPU: host side of the layer-norm-after-the-sum decoder (Goponex) -- configuration reader and its refusals, tensor names and
shapes, registry, YaRN tables with neighbour pairs -- and properties of the plain restatement that the GPU tests lean on."""
import json
import math

import pytest
import torch

from vllm_neuron_b200.hybrid import (DenseSpec, DualMixerSpec, HybridConfig, MambaSpec, MatrixMemorySpec, RotAttnSpec, RotSpec,
                                     random_weights, tensor_shapes)


def _par(mask=None, scaling=None, ff=9, right=None, **left):
    lm = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 6, "scale": 0.3, "rot": {"dims": 4, "base": 100.0}}
    lm.update(left)
    if scaling:
        lm["rot"] = {**lm["rot"], "scaling": scaling}
    if mask:
        lm["mask"] = mask
    return {"type": "parallel", "mixer": {"left": lm, "right": {"inner": 10, "state": 3, "dt_rank": 5, "conv": 2, **(right or {})}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _mem(ff=None, **kw):
    return {"type": "mlstm", "mixer": {"heads": 3, "dim": 4, "vdim": 5, "gate_cap": 7.5, **kw}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _cfg(layers=None):
    yarn = {"factor": 5.0, "original": 64, "fast": 8.0, "slow": 1.0}
    return {"architecture": "Goponex", "vocab": 20, "width": 12, "norm": {"eps": 1e-5}, "postln_alpha": 1.75,
            "layers": layers if layers is not None else [_par({"size": 9, "keep_first": 2}, scaling=yarn), _mem(), _par({"size": 5}, ff=None),
                                                         _mem(ff=7), _par()]}


def test_config_reader_round_trip_and_shapes():
    d = _cfg()
    cfg = HybridConfig.from_dict(d)
    assert cfg.style == "ln_post" and cfg.postln_alpha == 1.75 and cfg.eps == 1e-5
    assert cfg.to_dict() == d and HybridConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    m0, m1, m2, m3, m4 = (L.mixer for L in cfg.layers)
    for m in (m0, m2, m4):
        assert isinstance(m, DualMixerSpec) and isinstance(m.left, RotAttnSpec) and isinstance(m.right, MambaSpec)
        assert m.left_scale == m.right_scale == 0.5 and m.branch_norm and m.left.head_norm and m.left.v_from_k and not m.left.rot.half
    assert [(m.left.window, m.left.keep) for m in (m0, m2, m4)] == [(9, 2), (5, 0), (0, 0)]
    assert (m0.right.inner, m0.right.state, m0.right.dt_rank, m0.right.conv, m0.right.rank_cols) == (10, 3, 5, 2, 8)
    assert isinstance(m1, MatrixMemorySpec) and (m1.heads, m1.dim, m1.vdim, m1.gate_cap) == (3, 4, 5, 7.5)
    assert isinstance(cfg.layers[0].mlp, DenseSpec) and cfg.layers[0].mlp == DenseSpec(9, "relu2") and cfg.layers[1].mlp is None
    sh = tensor_shapes(cfg)
    assert sh["embed"] == sh["head"] == (20, 12) and sh["final.norm"] == sh["l0.norm1"] == sh["l0.norm2"] == (12,)
    assert "l1.norm2" not in sh and "l2.norm2" not in sh and sh["l3.norm2"] == (12,) and "l0.norm1.b" not in sh
    assert sh["l0.mix.left.q"] == (24, 12) and sh["l0.mix.left.k"] == (12, 12) and "l0.mix.left.v" not in sh
    assert sh["l0.mix.left.q.norm"] == sh["l0.mix.left.k.norm"] == (6,) and sh["l0.mix.left.o"] == (12, 24)
    assert sh["l0.mix.left.out"] == sh["l0.mix.right.out"] == (12,)
    assert sh["l0.mix.right.in"] == (20, 12) and sh["l0.mix.right.conv"] == (10, 2) and sh["l0.mix.right.conv.b"] == (10,)
    assert sh["l0.mix.right.x"] == (11, 10) and sh["l0.mix.right.dt"] == (10, 5) and sh["l0.mix.right.dt.b"] == sh["l0.mix.right.D"] == (10,)
    assert sh["l0.mix.right.A_log"] == (10, 3) and sh["l0.mix.right.o"] == (12, 10)
    assert sh["l1.mix.q"] == sh["l1.mix.k"] == (12, 12) and sh["l1.mix.v"] == sh["l1.mix.g"] == (15, 12) and sh["l1.mix.norm"] == (15,)
    assert sh["l1.mix.i"] == sh["l1.mix.f"] == (3, 12) and sh["l1.mix.i.b"] == sh["l1.mix.f.b"] == (3,) and sh["l1.mix.o"] == (12, 15)
    assert sh["l0.mlp.up"] == (9, 12) and sh["l0.mlp.up.b"] == (9,) and sh["l0.mlp.down"] == (12, 9) and sh["l0.mlp.down.b"] == (12,)
    assert "l0.mlp.gate" not in sh and "l1.mlp.up" not in sh and set(random_weights(cfg)) == set(sh)


def test_config_reader_refuses_what_the_design_does_not_have():
    for bad in ({**_par(), "type": "attention"}, {"type": "mamba2", "mlp": None, "mixer": {"heads": 2, "vdim": 3, "state": 5, "groups": 1, "conv": 3}},
                _par(kv_heads=3), _par(vdim=5), _par(rot={"dims": 8, "base": 10.0}), _par(rot={"dims": 3, "base": 10.0}),
                _par({"size": 4, "keep_first": -1}), _par(right={"conv": 0}), _mem(gate_cap=0.0),
                {**_par(), "mlp": {"kind": "moe", "router": {"experts": 2, "top": 1}, "expert": {"ff": 8}}}):
        with pytest.raises(ValueError):
            HybridConfig.from_dict(_cfg(layers=[bad]))
    for other in ("Pumopel", "Kenetar", "Zudarax"):  # a layer of this design in another one
        with pytest.raises((ValueError, KeyError)):
            HybridConfig.from_dict({**_cfg([_mem()]), "architecture": other})


def test_registry_serves_it_in_both_modes():
    from vllm_neuron_b200.registry import resolve

    arch, entry = resolve(_cfg())
    assert arch == "Goponex" and entry.family == "hybrid" and set(entry.dtypes) == {torch.bfloat16, torch.float32}
    assert entry.read_config(_cfg()) == HybridConfig.from_dict(_cfg())


@pytest.mark.parametrize("dims,base,sc", [(16, 10000.0, {"factor": 8.0, "original": 64, "fast": 4.0, "slow": 1.0}),
                                          (6, 50.0, {"factor": 3.0, "original": 4000, "fast": 32.0, "slow": 1.0}),
                                          (10, 500.0, {"factor": 2.0, "original": 7, "fast": 1.0, "slow": 1.0}), (8, 300.0, None)])
def test_yarn_tables(dims, base, sc):
    from oracle.goponex_ref import yarn_frequencies

    rot = {"dims": dims, "base": base, **({"scaling": sc} if sc else {})}
    f, mag = yarn_frequencies(rot)
    assert abs(mag - (0.1 * math.log(sc["factor"]) + 1.0 if sc else 1.0)) < 1e-15
    cos, sin = RotSpec(dims, base, sc).tables(40)
    a = torch.arange(40, dtype=torch.float64)[:, None] * f
    assert (cos.double() - mag * torch.cos(a)).abs().max() < 2e-7 and (sin.double() - mag * torch.sin(a)).abs().max() < 2e-7


def test_restatement_rotation_keeps_scores_relative_and_pairs_neighbours():
    from oracle.goponex_ref import rotate_pairs

    g = torch.Generator().manual_seed(0)
    rot = {"dims": 4, "base": 30.0}
    x = torch.randn(6, generator=g, dtype=torch.float64)
    X = rotate_pairs(x.expand(9, 1, 6), rot)[:, 0]
    assert (X[:, 4:] == x[4:]).all()
    for i in (0, 1):                                                           # columns 2i and 2i + 1 keep their length together
        assert (X[:, 2 * i:2 * i + 2].norm(dim=-1) - x[2 * i:2 * i + 2].norm()).abs().max() < 1e-12
    assert abs(X[1, 0] - (x[0] * math.cos(1) - x[1] * math.sin(1))) < 1e-12 and abs(X[1, 1] - (x[1] * math.cos(1) + x[0] * math.sin(1))) < 1e-12
    assert abs(X[7] @ X[4] - X[5] @ X[2]) < 1e-12


def test_restatement_window_and_kept_tokens():
    from oracle.goponex_ref import window_keep_attention, window_mask

    m = window_mask(12, 4, 2)
    assert m[10].nonzero().flatten().tolist() == [0, 1, 7, 8, 9, 10] and m[3].nonzero().flatten().tolist() == [0, 1, 2, 3]
    assert m[0].nonzero().flatten().tolist() == [0] and m[4].nonzero().flatten().tolist() == [0, 1, 2, 3, 4]
    assert window_mask(12, None, 3).sum() == 78 == window_mask(12, 4, 12).sum()
    g = torch.Generator().manual_seed(0)
    T, H, G, D, P = 20, 4, 2, 6, 5
    q, k, v = (torch.randn(T, n, d, generator=g, dtype=torch.float64) for n, d in ((H, D), (G, D), (G, P)))
    i, h = 17, 3
    seen = [0, 1, 14, 15, 16, 17]
    w = torch.softmax((k[seen, 1] @ q[i, h]) * 0.4, 0)
    assert (window_keep_attention(q, k, v, 0.4, 4, 2)[i, h] - w @ v[seen, 1]).abs().max() < 1e-12


def test_restatement_recurrences():
    from oracle.goponex_ref import matrix_memory, selective_scan

    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    T, C, N = 9, 4, 3
    x, dt, A, B, Cm, D = r(T, C), r(T, C).exp(), -r(C, N).exp(), r(T, N), r(T, N), r(C)
    y = selective_scan(x, dt, A, B, Cm, D)
    t, c = 7, 2
    S = sum(torch.exp(A[c] * dt[s + 1:t + 1, c].sum()) * dt[s, c] * x[s, c] * B[s] for s in range(t + 1))
    assert abs(y[t, c] - (S @ Cm[t] + D[c] * x[t, c])) < 1e-12
    H, Dk, P = 2, 3, 4
    q, k, v, i, f = r(T, H, Dk), r(T, H, Dk), r(T, H, P), 2 * r(T, H), -r(T, H).exp()
    o = matrix_memory(q, k, v, i, f)
    t, h = 6, 1
    m = torch.tensor(0.0, dtype=torch.float64)
    for s in range(t + 1):
        m = torch.maximum(f[s, h] + m, i[s, h])
    w = torch.stack([torch.exp(i[s, h] + f[s + 1:t + 1, h].sum() - m) * (k[s, h] @ q[t, h]) for s in range(t + 1)])
    want = (w[:, None] * v[:t + 1, h]).sum(0) / (torch.maximum(w.sum().abs(), torch.exp(-m)) + 1e-6)
    assert (o[t, h] - want).abs().max() < 1e-12
