"""Host-side checks of the Modadra family (no GPU): the config parser, the fused arena layout against the checkpoint names,
the registry, and the oracle's mechanisms against hand-checked cases."""
import math

import pytest
import torch

from oracle import modadra_oracle as mo
from tests import modadra_cases as mc

F64 = torch.float64


def _config():
    return mc.model([mc.parallel(mlp=mc.moe()), mc.parallel(heads=5, kv_heads=1, rot_dims=0, window=0, r_heads=3, r_kv_heads=3, conv=1),
                     mc.parallel(heads=7, kv_heads=7, dim=9, vdim=11, rot_dims=2, mlp=mc.moe(experts=4, top=4, groups=None, ff=7))])


def test_the_parser_reads_every_constant():
    from pipelinerl_b200.hybrid import HybridConfig
    config = _config()
    cfg = HybridConfig.from_modadra(config, mo.tensor_shapes(config))
    assert (cfg.block, cfg.residual_mult, cfg.logit_softcap, cfg.eps, cfg.vocab_size, cfg.width) == ("pre_norm", 0.6, 12.0, 1e-5, 96, 72)
    assert not cfg.tied_head and [L.kind for L in cfg.layers] == ["attn_delta"] * 3
    a, g, e = cfg.layers[0].attn, cfg.layers[0].gdelta, cfg.layers[0].mlp.moe
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.rot_dims, a.rot_base, a.rot_half) == (6, 3, 12, 10, 40, 8, 30.0, True)
    assert a.scale == 1.2 * 12 ** -0.5 and a.unit_sink and not a.sink and a.gate and a.gate_per_head
    assert (g.heads, g.kv_heads, g.dim, g.vdim, g.conv) == (6, 2, 10, 14, 3)
    assert (e.experts, e.top, e.ff, e.groups, e.keep_groups, e.group_top, e.weight_scale) == (10, 3, 20, 5, 3, 2, 1.4)
    assert (e.score, e.renorm, e.correction, e.act) == ("sigmoid", True, True, "gelu")
    assert cfg.layers[1].mlp is None and cfg.layers[1].attn.window == 0 and cfg.layers[1].attn.rot_dims == 0
    assert (cfg.layers[2].mlp.moe.groups, cfg.layers[2].mlp.moe.keep_groups) == (1, 1)
    assert cfg.layers[0].left_scale == cfg.layers[0].right_scale == 0.5


def test_every_checkpoint_tensor_has_a_place_in_the_arena():
    from pipelinerl_b200.hybrid import HybridConfig
    config = _config()
    shapes = mo.tensor_shapes(config)
    cfg = HybridConfig.from_modadra(config, shapes)
    slices, fused = cfg.checkpoint_slices(), dict(cfg.fused_shapes())
    assert set(slices) == set(shapes)
    covered = {}
    for name, (dst, r0, rn) in slices.items():
        assert (rn, *shapes[name][1:]) == (shapes[name][0], *fused[dst][1:]), name
        covered.setdefault(dst, []).append((r0, rn))
    assert set(covered) == set(fused)
    for dst, spans in covered.items():          # the slices tile every fused tensor, up to padding at the end of mix.in
        at = 0
        for r0, rn in sorted(spans):
            assert r0 == at
            at += rn
        assert at == fused[dst][0] or (dst.endswith("mix.in") and at <= fused[dst][0] == (at + 7) // 8 * 8), dst
    for L in cfg.layers:                        # the columns the mixers read are where the tensors' rows are
        C, p = cfg.attn_delta_rows(L), f"l{L.weights_of}.mix."
        at = {n: slices[p + n][1] for n in ("left.q", "left.k", "left.v", "left.g", "right.q", "right.g", "right.b", "right.a")}
        assert at == {"left.q": 0, "left.k": C.k, "left.v": C.v, "left.g": C.left_g, "right.q": C.right, "right.g": C.right_g,
                      "right.b": C.b, "right.a": C.a}
    assert dict(HybridConfig.from_modadra(config).fused_shapes()) == fused
    bare = {k: v for k, v in shapes.items() if not k.endswith(("correction", "left.g"))}
    cfg2 = HybridConfig.from_modadra(config, bare)
    assert set(cfg2.checkpoint_slices()) == set(bare) and not cfg2.layers[0].attn.gate and not cfg2.layers[0].mlp.moe.correction


def test_bad_sizes_are_refused():
    from pipelinerl_b200.hybrid import HybridConfig
    P, M = mc.parallel, mc.moe
    for bad in (mc.model([P(heads=5, kv_heads=2)]), mc.model([P(rot_dims=7)]), mc.model([P(rot_dims=14)]), mc.model([P(r_heads=3)]),
                mc.model([P(conv=0)]), mc.model([P(mlp=M(experts=9, groups=(2, 1)))]), mc.model([P(mlp=M(top=7))]),
                mc.model([P(mlp=M(groups=(5, 6)))]), mc.model([P(r_dim=300)]), mc.model([P()], cap=-1.0)):
        with pytest.raises(ValueError):
            HybridConfig.from_modadra(bad)
    odd = mc.model([P()])
    odd["layers"][0]["type"] = "attention"
    with pytest.raises(ValueError):
        HybridConfig.from_modadra(odd)


def test_registry_knows_the_architecture(tmp_path):
    from pipelinerl_b200 import registry
    config = _config()
    mc.write_checkpoint(tmp_path, config, mc.weights(config, 1))
    fam, cfg = registry.load_config(tmp_path)
    assert fam.name == "Modadra" and torch.float32 in fam.dtypes and torch.bfloat16 in fam.dtypes
    assert cfg.vocab_size == config["vocab"] and len(cfg.layers) == 3


def test_oracle_attention_on_small_cases():
    g = torch.Generator().manual_seed(0)
    v = torch.randn(5, 1, 3, generator=g, dtype=F64)
    q, k = torch.zeros(5, 2, 4, dtype=F64), torch.randn(5, 1, 4, generator=g, dtype=F64)
    o = mo.sink_attention(q, k, v, 0.7, 3)                  # zero scores: every visible key and the sink weigh the same
    for t in range(5):
        seen = v[max(0, t - 2):t + 1, 0]
        assert torch.allclose(o[t], (seen.sum(0) / (len(seen) + 1)).expand(2, 3), atol=1e-12)
    s = 1.3                                                 # one key: weight e^s / (1 + e^s), also for large scores
    for s in (-50.0, -1.0, 0.4, 60.0):
        o = mo.sink_attention(torch.full((1, 1, 1), s, dtype=F64), torch.ones(1, 1, 1, dtype=F64), torch.ones(1, 1, 1, dtype=F64), 1.0, 0)
        assert o.item() == pytest.approx(1.0 / (1.0 + math.exp(-s)), rel=1e-12)
    a, b = torch.randn(1, 1, 8, generator=g, dtype=F64), torch.randn(1, 1, 8, generator=g, dtype=F64)
    at = lambda x, p: mo.rotate(x, torch.tensor([p]), 6, 20.0)
    assert torch.allclose((at(a, 5) * at(b, 3)).sum(), (at(a, 12) * at(b, 10)).sum(), atol=1e-12)     # the distance decides
    assert torch.equal(at(a, 7)[..., 6:], a[..., 6:]) and torch.equal(at(a, 0), a)
    x = torch.zeros(1, 1, 4, dtype=F64)
    x[..., 0] = 1.0                                          # channel 0 turns towards its partner, channel dims / 2
    y = mo.rotate(x, torch.tensor([2]), 4, 9.0)
    assert torch.allclose(y[0, 0], torch.tensor([math.cos(2.0), 0.0, math.sin(2.0), 0.0], dtype=F64))


def test_oracle_gated_delta_on_small_cases():
    g = torch.Generator().manual_seed(1)
    keys, vals, ones = torch.eye(4, dtype=F64)[:, None, :], torch.randn(4, 1, 3, generator=g, dtype=F64), torch.ones(4, 1, dtype=F64)
    assert torch.allclose(mo.gated_delta(keys, keys, vals, ones, ones), vals, atol=1e-12)      # read back in the same token
    o = mo.gated_delta(keys[[1, 0, 0, 0]], keys[[0, 1, 2, 0]], vals, ones, ones)
    assert torch.allclose(o[0], torch.zeros(1, 3, dtype=F64)) and torch.allclose(o[1], vals[0])  # an older key's value
    assert torch.allclose(o[3], vals[3], atol=1e-12)                                           # a rewritten key: the new value
    half = torch.full((4, 1), 0.5, dtype=F64)
    o = mo.gated_delta(keys[[0, 0, 0, 0]], keys[[0, 1, 2, 3]], vals, ones, half)               # decay before the write
    assert torch.allclose(o[:, 0], vals[:1, 0] * torch.tensor([[1.0], [0.5], [0.25], [0.125]], dtype=F64), atol=1e-12)
    x, taps = torch.randn(5, 2, generator=g, dtype=F64), torch.tensor([[0.0, 0.0, 1.0], [1.0, 0.0, 0.0]], dtype=F64)
    y = mo.causal_conv(x, taps)                              # the last tap is the current token's
    assert torch.allclose(y[:, 0], mo.silu(x[:, 0])) and torch.equal(y[:2, 1], torch.zeros(2, dtype=F64))
    assert torch.allclose(y[2:, 1], mo.silu(x[:3, 1]))
    assert mo.decay(torch.tensor(0.0, dtype=F64), torch.tensor(0.0, dtype=F64), torch.tensor(0.0, dtype=F64)).item() == pytest.approx(0.5)


def test_oracle_choice_on_small_cases():
    pick = lambda s, c, **r: mo.choose(torch.tensor(s, dtype=F64), torch.tensor(c, dtype=F64), r)
    s, zero = [0.9, 0.1, 0.6, 0.5, 0.7, 0.2], [0.0] * 6
    assert pick(s, zero, top=2) == [0, 4]
    # groups of two ranked by their sum: (2, 3) 1.1, (0, 1) 1.0, (4, 5) 0.9 -- the best single output does not decide
    assert pick(s, zero, top=2, groups=dict(count=3, keep=1)) == [2, 3]
    assert pick(s, zero, top=3, groups=dict(count=3, keep=2)) == [0, 2, 3]
    # groups of three ranked by the sum of their TWO best: (0, 1, 2) 1.5, (3, 4, 5) 1.2
    assert pick(s, zero, top=3, groups=dict(count=2, keep=1)) == [0, 2, 1]
    # all choice scores negative: closed outputs lose to every open one
    assert pick(s, [-3.0] * 6, top=2, groups=dict(count=3, keep=1)) == [2, 3]
    assert pick(s, [-3.0, -3.0, -3.0, -3.0, -2.0, -2.0], top=2, groups=dict(count=3, keep=1)) == [4, 5]
    assert pick([0.5] * 6, zero, top=3) == [0, 1, 2]                                 # ties: the lower index
    assert pick(s, zero, top=2, groups=dict(count=6, keep=3)) == [0, 4]              # groups of one
