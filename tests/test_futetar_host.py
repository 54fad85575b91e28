"""Host-side checks of the Futetar family (no GPU): the config parser, the fused arena layout against the checkpoint
names, the registry, the rotary table, and the oracle's own consistency."""
import math

import pytest
import torch

from oracle import futetar_oracle as fo
from tests import futetar_cases as fc


def _config():
    return fc.model([fc.attention(mlp=fc.moe()), fc.cell(mlp=fc.dense()), fc.attention(heads=3, kv_from=0, mlp=fc.dense(ff=12)),
                     fc.cell(heads=2, dim=7, vdim=5), fc.attention(heads=9, kv_from=0),
                     fc.cell(mlp=fc.moe(experts=5, top=1, identity=0, groups=None, shared=0))])


def test_the_parser_reads_every_constant():
    from pipelinerl_b200.hybrid import HybridConfig
    config = _config()
    cfg = HybridConfig.from_futetar(config, fo.tensor_shapes(config))
    assert [L.kind for L in cfg.layers] == ["attention", "mlstm", "attention", "mlstm", "attention", "mlstm"]
    assert cfg.block == "one_norm" and cfg.norm_offset == 1.0 and cfg.embed_scale == 1.0 and not cfg.tied_head and cfg.logit_scale == 1.0
    a = cfg.layers[0].attn
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims, a.rot_base, a.kv_from) == (6, 3, 12, 10, 8, 30.0, -1)
    assert (a.rot_scaling_kind, a.rot_scaling, a.rot_half, a.head_norm, a.head_gain, a.gate, a.bias, a.window) == (
        "bands", (3.0, 0.5, 2.5, 40.0), True, True, True, False, False, 0)
    assert [cfg.layers[i].attn.kv_from for i in (2, 4)] == [0, 0] and cfg.layers[4].attn.heads == 9
    c = cfg.layers[1].mlstm
    assert (c.heads, c.dim, c.vdim, c.gate_cap, c.den_eps) == (3, 10, 14, 9.0, 1e-6)
    assert (cfg.layers[1].mlp.kind, cfg.layers[1].mlp.ff, cfg.layers[3].mlp) == ("geglu", 40, None)
    e = cfg.layers[0].mlp.moe
    assert (e.experts, e.identity, e.outputs, e.top, e.ff, e.groups, e.keep_groups, e.shared_ff) == (6, 2, 8, 3, 20, 4, 3, 28)
    assert e.correction and e.shared_gate and e.score == "softmax_all" and e.weight_on == "output"
    e = cfg.layers[5].mlp.moe
    assert (e.identity, e.groups, e.keep_groups, e.shared_ff, e.shared_gate) == (0, 1, 1, 0, False)


def test_every_checkpoint_tensor_has_a_place_in_the_arena():
    from pipelinerl_b200.hybrid import HybridConfig
    config = _config()
    shapes = fo.tensor_shapes(config)
    cfg = HybridConfig.from_futetar(config, shapes)
    slices, fused = cfg.checkpoint_slices(), dict(cfg.fused_shapes())
    assert set(slices) == set(shapes)
    covered = {}
    for name, (dst, r0, rn) in slices.items():
        assert (rn, *shapes[name][1:]) == (shapes[name][0], *fused[dst][1:]), name
        covered.setdefault(dst, []).append((r0, rn))
    assert set(covered) == set(fused)
    for dst, spans in covered.items():       # the slices do not overlap; only an input projection has (padding) gaps
        at = gap = 0
        for r0, rn in sorted(spans):
            assert r0 >= at
            gap += r0 - at
            at = r0 + rn
        gap += fused[dst][0] - at
        assert 0 <= gap < 15 if dst.endswith(".in") else gap == 0, dst
    for i, L in enumerate(cfg.layers):       # the column offsets the engine uses are where the loader puts the rows
        J = cfg.joint_rows(L)
        assert J.mix % 8 == 0 and J.total % 8 == 0 and fused[f"l{i}.in"] == (J.total, cfg.width)
        if L.mlp is not None and L.mlp.kind == "geglu":
            assert slices[f"l{i}.mlp.gate"][1] == J.ff and slices[f"l{i}.mlp.up"][1] == J.ff + L.mlp.ff
        elif L.mlp is not None:
            assert slices[f"l{i}.mlp.router"][1] == J.router
            if L.mlp.ff:
                assert slices[f"l{i}.mlp.shared.up"][1] == J.ff and slices[f"l{i}.mlp.shared.sg"][1] == J.shared_gate
    # a checkpoint without a correction or a shared gate parses too
    bare = {k: v for k, v in shapes.items() if not k.endswith((".correction", "shared.sg"))}
    cfg2 = HybridConfig.from_futetar(config, bare)
    assert set(cfg2.checkpoint_slices()) == set(bare) and not cfg2.layers[0].mlp.moe.correction


def test_bad_sizes_are_refused():
    from pipelinerl_b200.hybrid import HybridConfig
    A, C, M = fc.attention, fc.cell, fc.moe
    for bad in ([A(heads=5, kv_heads=2)], [A(rot_dims=7)], [A(rot_dims=14)], [C(dim=300)],
                [A(), A(kv_from=1)], [A(kv_from=1), A()], [C(), A(kv_from=0)], [A(), A(kv_from=0), A(kv_from=1)],
                [A(), A(kv_from=0, kv_heads=6)], [A(), A(kv_from=0, base=31.0)], [A(), A(kv_from=0, vdim=12)],
                [C(mlp=M(groups=(3, 1)))], [C(mlp=M(groups=(4, 5)))], [C(mlp=M(top=5, groups=(4, 2)))],
                [C(mlp=M(experts=2, identity=0, top=3, groups=None))]):
        with pytest.raises(ValueError):
            HybridConfig.from_futetar(fc.model(bad))
    odd = fc.model([A()])
    odd["layers"][0]["type"] = "convolution"
    with pytest.raises(ValueError):
        HybridConfig.from_futetar(odd)


def test_registry_knows_the_architecture(tmp_path):
    from pipelinerl_b200 import registry
    config = _config()
    fc.write_checkpoint(tmp_path, config, fc.weights(config, 1))
    fam, cfg = registry.load_config(tmp_path)
    assert fam.name == "Futetar" and torch.float32 in fam.dtypes and torch.bfloat16 in fam.dtypes
    assert cfg.vocab_size == config["vocab"] and len(cfg.layers) == 6


def test_banded_rotary_table_matches_the_oracle_and_its_limits():
    from pipelinerl_b200.hybrid import rotary_table
    for dims, base, sc in ((8, 30.0, (3.0, 0.5, 2.5, 40)), (64, 5e5, (16.0, 1.0, 4.0, 8192)), (12, 3.0, (4.0, 1.0, 2.0, 64)),
                           (2, 10.0, (2.0, 1.0, 4.0, 8)), (20, 1e4, None)):
        f, mag = rotary_table(dims, base, sc, "bands")
        rot = dict(dims=dims, base=base)
        if sc:
            rot["scaling"] = dict(factor=sc[0], low=sc[1], high=sc[2], original=sc[3])
        ref = fo.rotary_frequencies(rot)
        assert mag == 1.0 and torch.allclose(torch.tensor(f, dtype=torch.float64), torch.tensor(ref, dtype=torch.float64), rtol=1e-14, atol=0)
        for i, x in enumerate(f):
            plain = base ** (-2.0 * i / dims)
            if sc is None or 2 * math.pi / plain < sc[3] / sc[2]:       # short waves are kept
                assert x == plain
            elif 2 * math.pi / plain > sc[3] / sc[1]:                   # long ones stretched
                assert math.isclose(x, plain / sc[0], rel_tol=1e-15)
            else:
                assert plain / sc[0] * (1 - 1e-12) <= x <= plain * (1 + 1e-12)
    assert rotary_table(0, 10.0, None, "bands") == ([], 1.0)


def test_joint_cache_is_counted_once():
    from pipelinerl_b200.hybrid import HybridConfig, HybridEngine
    config = _config()
    eng = HybridEngine.__new__(HybridEngine)
    eng.cfg, eng.f32 = HybridConfig.from_futetar(config, fo.tensor_shapes(config)), False
    assert eng.kv_bytes_per_token() == 3 * (12 + 10) * 2                # three attention layers, one cache


def test_oracle_mechanisms_agree_with_their_definitions():
    g = torch.Generator().manual_seed(0)
    F64 = torch.float64
    # the choice: groups are ranked by their best score, closed groups never chosen even when all scores are negative
    score = torch.tensor([0.30, 0.05, 0.20, 0.02, 0.25, 0.18], dtype=F64)
    r = dict(top=3, groups=dict(count=3, keep=2))
    assert fo.choose(score, torch.zeros(6, dtype=F64), r) == [0, 4, 5]
    assert fo.choose(score, torch.full((6,), -2.0, dtype=F64), r) == [0, 4, 5]
    assert fo.choose(score, torch.tensor([0, 0, 0.5, 0, 0, 0], dtype=F64), r) == [2, 0, 1]
    assert fo.choose(score, torch.zeros(6, dtype=F64), dict(top=2)) == [0, 4]
    gap = []
    fo.choose(score, torch.zeros(6, dtype=F64), r, gap)
    assert math.isclose(gap[0], 0.05)                                  # between the second and the third group
    # gelu in its tanh form against torch's
    z = torch.linspace(-6, 6, 101, dtype=F64)
    assert torch.allclose(fo.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)
    # attention with one visible key returns its value; equal scores return the mean
    cfg = fc.attention(heads=2, kv_heads=1, dim=4, vdim=3, rot_dims=0)["mixer"]
    wt = {"q": torch.zeros(8, 5, dtype=F64), "q.norm": torch.ones(4, dtype=F64), "o": torch.eye(6, dtype=F64)}
    h, keys, vals = (torch.randn(*s, generator=g, dtype=F64) for s in ((7, 5), (7, 1, 4), (7, 1, 3)))
    o = fo.attention(h, keys, vals, wt, "", cfg, 1e-5)
    mean = torch.cumsum(vals[:, 0], 0) / torch.arange(1, 8, dtype=F64)[:, None]
    assert torch.allclose(o[:, :3], mean) and torch.allclose(o[:, 3:], mean)
    # the rotation keeps lengths and makes scores depend on the distance only
    rot = dict(dims=6, base=20.0, scaling=dict(factor=2.0, low=0.5, high=2.0, original=30))
    a, b = torch.randn(1, 1, 8, generator=g, dtype=F64).expand(30, 1, 8), torch.randn(1, 1, 8, generator=g, dtype=F64).expand(30, 1, 8)
    ra, rb = fo.rotate(a, rot), fo.rotate(b, rot)
    assert torch.allclose((ra[5] * rb[3]).sum(), (ra[12] * rb[10]).sum(), atol=1e-12)
    assert torch.equal(ra[7, :, 6:], a[7, :, 6:]) and torch.allclose(ra[7].norm(), a[7].norm())
    # the memory cell against its unstabilised definition S_t = f S + i k v^T (small gates, so nothing overflows)
    m = dict(heads=1, dim=3, vdim=2, gate_cap=4.0)
    W = 5
    wt = {k: torch.randn(*s, generator=g, dtype=F64) * 0.5 for k, s in dict(q=(3, W), k=(3, W), v=(2, W), i=(1, W), f=(1, W), g=(2, W)).items()}
    wt |= {"i.b": torch.zeros(1, dtype=F64), "f.b": torch.ones(1, dtype=F64), "norm": torch.ones(2, dtype=F64), "o": torch.eye(2, dtype=F64)}
    h = torch.randn(9, W, generator=g, dtype=F64)
    got = fo.matrix_lstm(h, wt, "", m, 1e-30)
    S, n = torch.zeros(3, 2, dtype=F64), torch.zeros(3, dtype=F64)
    for t in range(9):
        soft = lambda z: 4.0 * torch.tanh(z / 4.0)
        i, f = torch.exp(soft(wt["i"] @ h[t])), torch.sigmoid(soft(wt["f"] @ h[t] + 1.0))
        q, k, v = wt["q"] @ h[t] / math.sqrt(3), wt["k"] @ h[t], wt["v"] @ h[t]
        S, n = f * S + i * torch.outer(k, v), f * n + i * k
        o = S.T @ q                                                     # the head norm cancels the denominator
        want = o / o.pow(2).mean().sqrt() * torch.sigmoid(wt["g"] @ h[t])
        assert torch.allclose(got[t], want, atol=1e-8)
