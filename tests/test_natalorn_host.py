"""CPU: host side of the hyper-connected decoder (Natalorn) -- configuration reader and its refusals, tensor names and shapes, layer
runs, registry, rotation tables -- and properties of the plain restatement that the GPU tests lean on."""
import json
import math

import pytest
import torch

from vllm_neuron_b200.hybrid import HybridConfig, LatentAttnSpec, MoeSpec, RotAttnSpec, RotSpec, random_weights, tensor_shapes


def _moe(**kw):
    r = {"experts": 6, "top": 2, "scale": 1.5, "groups": {"count": 3, "keep": 2}}
    r.update(kw)
    return {"kind": "moe", "router": r, "expert": {"ff": 5}, "shared": {"ff": 7}}


def _att(kind="attention", mlp=None, **kw):
    m = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "scale": 0.3, "mask": {"size": 9}}
    if kind == "attention_2":
        m["softcap"] = 12.5
    m.update(kw)
    return {"type": kind, "mixer": m, "mlp": mlp}


def _lat(mlp=None, **kw):
    m = {"heads": 3, "dim": 4, "rot_dim": 2, "vdim": 5, "kv_rank": 8, "q_rank": 10, "scale": 0.25, "rot": {"dims": 2, "base": 90.0}, "mask": {"size": 4}}
    m.update(kw)
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _cfg(layers=None, **kw):
    return {"architecture": "Natalorn", "vocab": 20, "width": 12, "norm": {"eps": 1e-5}, "streams": 3, "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": layers if layers is not None else [_att(mlp=_moe()), _att("attention_2", mlp=_moe(scale=2.0)), _lat(), _lat(_moe())], **kw}


def test_config_reader_round_trip_and_shapes():
    d = _cfg()
    cfg = HybridConfig.from_dict(d)
    assert cfg.style == "rms_hyper" and cfg.streams == 3 and cfg.eps == 1e-5
    assert cfg.to_dict() == d and HybridConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert [i for i, _ in cfg.layer_runs()] == [0, 1, 2, 1, 2, 3]
    m0, m1, m2, _ = (L.mixer for L in cfg.layers)
    assert isinstance(m0, RotAttnSpec) and m0.rot is None and (m0.window, m0.chunk, m0.softcap, m0.bias) == (9, 0, 0.0, False)
    assert isinstance(m1, RotAttnSpec) and m1.rot is None and (m1.window, m1.chunk, m1.softcap, m1.bias) == (0, 9, 12.5, True)
    assert isinstance(m2, LatentAttnSpec) and (m2.window, m2.sink, m2.gate_cols, m2.rot.half) == (4, True, True, False)
    f = cfg.layers[0].mlp
    assert isinstance(f, MoeSpec) and (f.route, f.experts, f.top, f.groups, f.keep, f.scale, f.ff, f.shared_ff) == ("softmax_grouped", 6, 2, 3, 2, 1.5, 5, 7)
    sh = tensor_shapes(cfg)
    assert sh["embed"] == sh["head"] == (20, 12) and sh["final.norm"] == sh["l0.norm1"] == sh["l0.norm2"] == (12,) and "l2.norm2" not in sh
    assert sh["l0.mix.q"] == (24, 12) and sh["l0.mix.k"] == (12, 12) and sh["l0.mix.v"] == (6, 12) and sh["l0.mix.o"] == (12, 12)
    assert "l0.mix.q.b" not in sh and sh["l1.mix.q.b"] == (24,) and sh["l1.mix.k.b"] == (12,) and sh["l1.mix.v.b"] == (6,)
    assert sh["l2.mix.dq"] == (10, 12) and sh["l2.mix.uq"] == (18, 10) and sh["l2.mix.dkv"] == (10, 12) and sh["l2.mix.uk"] == (12, 8)
    assert sh["l2.mix.uv"] == (15, 8) and sh["l2.mix.sink"] == (3,) and sh["l2.mix.g"] == (15, 12) and sh["l2.mix.o"] == (12, 15)
    assert sh["l0.hc1.in"] == sh["l0.hc2.out"] == (3,) and sh["l3.hc1.mix"] == (3, 3) and "l2.hc1.mix" in sh and "l2.hc2.mix" not in sh
    assert sh["l0.mlp.router"] == (6, 12) and sh["l0.mlp.correction"] == (6,) and sh["l0.mlp.e5.down"] == (12, 5) and sh["l0.mlp.shared.up"] == (7, 12)
    assert set(random_weights(cfg)) == set(sh)
    plain = HybridConfig.from_dict({**_cfg([_att(mlp={**_moe(), "shared": None, "router": {"experts": 4, "top": 4}}), _att(mask=None)]), "loop": None})
    f = plain.layers[0].mlp
    assert (f.groups, f.keep, f.scale, f.shared_ff) == (1, 1, 1.0, 0) and plain.layers[1].mixer.window == 0 and len(plain.layer_runs()) == 2
    assert "l0.mlp.shared.up" not in tensor_shapes(plain)


def test_config_reader_refuses_what_the_design_does_not_have():
    for bad in (_att(kv_heads=3), {**_att(), "type": "attention_3"}, {**_att(), "type": "delta"}, _lat(rot={"dims": 4, "base": 10.0}),
                _lat(rot={"dims": 1, "base": 10.0}), _att(mask={"size": -2}), _att(mlp={"kind": "dense", "ff": 8}), _att(mlp=_moe(top=5)),
                _att(mlp=_moe(groups={"count": 4, "keep": 1})), _att(mlp=_moe(groups={"count": 3, "keep": 4}))):
        with pytest.raises(ValueError):
            HybridConfig.from_dict({**_cfg([bad]), "loop": None})
    for kw in (dict(streams=33), dict(streams=-1), dict(loop={"start": 2, "stop": 5, "times": 1}), dict(loop={"start": 1, "stop": 2, "times": 0})):
        with pytest.raises(ValueError):
            HybridConfig.from_dict(_cfg(**kw))


def test_registry_serves_it_in_both_modes():
    from vllm_neuron_b200.registry import resolve

    arch, entry = resolve(_cfg())
    assert arch == "Natalorn" and entry.family == "hybrid" and set(entry.dtypes) == {torch.bfloat16, torch.float32}
    assert entry.read_config(_cfg()) == HybridConfig.from_dict(_cfg())


def test_rotation_tables_and_restatement_agree():
    from oracle.natalorn_ref import rotate_pairs

    x = torch.randn(30, 2, 8, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    cos, sin = RotSpec(6, 55.0).tables(30)
    y = rotate_pairs(x, 55.0, 6)
    for i in range(3):
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        c, s = cos[:, None, i].double(), sin[:, None, i].double()
        assert (y[..., 2 * i] - (u * c - v * s)).abs().max() < 1e-6 and (y[..., 2 * i + 1] - (v * c + u * s)).abs().max() < 1e-6
    assert (y[..., 6:] == x[..., 6:]).all() and abs(sin[1, 0].item() - math.sin(1)) < 1e-7


def test_restatement_masks_and_sink():
    from oracle.natalorn_ref import chunk_mask, softmax_weights, window_mask

    assert window_mask(12, 4)[10].nonzero().flatten().tolist() == [7, 8, 9, 10] and window_mask(12, 4)[2].sum() == 3
    assert chunk_mask(12, 5)[9].nonzero().flatten().tolist() == [5, 6, 7, 8, 9] and chunk_mask(12, 5)[10].nonzero().flatten().tolist() == [10]
    assert window_mask(12, None).sum() == chunk_mask(12, 12).sum() == 78
    s = torch.tensor([[0.3, 2.0, 9.0]], dtype=torch.float64)
    w = softmax_weights(s, torch.tensor([[True, True, False]]), torch.tensor(1.0, dtype=torch.float64))
    den = math.exp(0.3) + math.exp(2.0) + math.exp(1.0)
    assert abs(w[0, 0] - math.exp(0.3) / den) < 1e-15 and w[0, 2] == 0


def test_restatement_router_keeps_excluded_groups_out():
    from oracle.natalorn_ref import choose_experts

    z = torch.log(torch.tensor([[0.30, 0.05, 0.20, 0.15, 0.18, 0.12]], dtype=torch.float64))
    corr = torch.tensor([-2.0, -1.0, -1.1, -1.5, -1.4, -3.0], dtype=torch.float64)
    # choice scores -1.70 -0.95 | -0.90 -1.35 | -1.22 -2.88: pairs rank 2nd, 1st, 3rd
    idx, s = choose_experts(z, corr, 2, 3, 2)
    assert idx.tolist() == [[2, 1]] and (s - torch.tensor([[0.20, 0.05]], dtype=torch.float64)).abs().max() < 1e-12
    idx, _ = choose_experts(z, corr, 2, 3, 1)
    assert idx.tolist() == [[2, 3]]


def test_restatement_streams():
    from oracle.natalorn_ref import read_streams, write_streams

    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]])
    M, o, y = torch.tensor([[0.5, 2.0], [0.0, 1.0]]), torch.tensor([1.0, -1.0]), torch.tensor([[100.0, 200.0]])
    assert write_streams(X, y, M, o).tolist() == [[[100.5, 201.0]], [[-88.0, -176.0]]]
    assert read_streams(X, torch.tensor([3.0, 0.1])).tolist() == [[4.0, 8.0]]
