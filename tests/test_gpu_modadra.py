"""The Modadra decoders on the hybrid engine (pipelinerl_b200/hybrid.py and its kernels) against
oracle/modadra_oracle.py: each mechanism alone, whole prompts against token-by-token decoding, portions down to two
tokens, unequal batches against each request alone, pages and slots that are given back and taken again, window edges and
the constant sink, the carried memory, the choice of experts, the first tokens, long decoding, awkward sizes, the bf16
serving mode, greedy generation through the engine's scheduler, and the trace runner."""
import json
import math
import subprocess
import sys

import pytest
import torch

from oracle import modadra_oracle as mo
from tests import modadra_cases as mc

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4      # fp32 kernels against the float64 oracle
BF16_TOL = 8e-2     # bf16 operands / cache: rounding of activations dominates
P, M = mc.parallel, mc.moe


# ---- each mechanism alone ---------------------------------------------------------------------------------------
def _mechanisms():
    return {
        "both_mixers": mc.model([P()]),
        "every_head_its_own_keys_all_channels_rotated": mc.model([P(heads=4, kv_heads=4, dim=8, vdim=8, rot_dims=8, r_heads=3, r_kv_heads=3)]),
        "one_key_head_two_rotated_channels": mc.model([P(heads=5, kv_heads=1, dim=14, vdim=6, rot_dims=2, r_heads=4, r_kv_heads=1)]),
        "no_rotation_no_window": mc.model([P(rot_dims=0, window=0)]),
        "window_of_one": mc.model([P(window=1)]),
        "one_head_one_channel": mc.model([P(heads=1, kv_heads=1, dim=2, vdim=1, rot_dims=2, r_heads=1, r_kv_heads=1, r_dim=1, r_vdim=1)]),
        "wide_heads": mc.model([P(heads=2, kv_heads=1, dim=80, vdim=136, rot_dims=80, r_heads=2, r_kv_heads=1, r_dim=130, r_vdim=96)], width=40),
        "one_tap": mc.model([P(conv=1)]),
        "many_taps": mc.model([P(conv=7)]),
        "many_small_delta_heads": mc.model([P(r_heads=12, r_kv_heads=3, r_dim=4, r_vdim=8, conv=2)]),
        "routed": mc.model([P(mlp=M())]),
        "routed_one_expert": mc.model([P(mlp=M(experts=1, top=1, ff=9, groups=None))]),
        "routed_no_groups": mc.model([P(mlp=M(experts=7, top=2, ff=10, groups=None, scale=1.0))]),
        "routed_one_group_kept": mc.model([P(mlp=M(experts=12, top=3, ff=9, groups=(4, 1)))]),
        "routed_groups_of_one": mc.model([P(mlp=M(experts=6, top=2, ff=8, groups=(6, 3)))]),
        "routed_groups_of_four": mc.model([P(mlp=M(experts=12, top=5, ff=8, groups=(3, 2), scale=2.5))]),
        "routed_everything": mc.model([P(mlp=M(experts=5, top=5, ff=9, groups=(5, 5)))]),
        "routed_many": mc.model([P(mlp=M(experts=80, top=8, ff=6, groups=(8, 4)))]),
        "odd_width": mc.model([P(mlp=M()), P(heads=3, kv_heads=1)], vocab=61, width=50),
        "no_cap_whole_residual": mc.model([P(mlp=M()), P()], cap=0.0, mult=1.0),
        "three_layers": mc.model([P(mlp=M()), P(heads=3, kv_heads=3, window=9, conv=4), P(r_dim=16, r_vdim=16, mlp=M(experts=4, groups=(2, 1), top=2))]),
    }


@pytest.mark.parametrize("name", sorted(_mechanisms()))
def test_each_mechanism_matches_the_oracle_fp32(cuda_device, name):
    config = _mechanisms()[name]
    wt = mc.weights(config, seed=len(name))
    toks = mc.tokens_for(config, 150)
    res = []
    ref = mc.oracle_logits(config, wt, toks, residuals=res)
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    assert mc.rel_err(mc.stream_logits(eng, toks, [150]), ref) < F32_TOL
    assert mc.rel_err(mc.stream_logits(eng, toks, [2, 3, 61, 2, 7, 64, 2]), ref) < F32_TOL     # then one by one
    # the residual stream after every layer of a whole prompt
    s = mc.stage_stream(eng, toks[:20])
    got = []
    eng._forward_rows([(s, 0, 20)], [], trace=got)
    eng.close_stream(s)
    assert len(got) == len(res)
    for a, b in zip(got, res):
        assert (a.double().cpu() - b[:20]).abs().max().item() < 1e-4 * max(1.0, b.abs().max().item())


FULL = mc.model([P(mlp=M()), P(heads=4, kv_heads=2, dim=16, vdim=20, rot_dims=16, window=70, r_heads=4, r_kv_heads=4, r_dim=12, r_vdim=9, conv=4),
                 P(heads=3, kv_heads=1, window=65, r_heads=2, r_kv_heads=1, r_dim=24, r_vdim=16, mlp=M(experts=6, top=2, groups=(3, 2), ff=16))],
                vocab=80, width=64)


def test_prefill_against_token_by_token_decoding(cuda_device):
    wt = mc.weights(FULL, 3)
    toks = mc.tokens_for(FULL, 140, seed=5)
    ref = mc.oracle_logits(FULL, wt, toks)
    eng = mc.build_engine(FULL, wt, torch.float32, cuda_device)
    whole = mc.stream_logits(eng, toks, [140])
    single = mc.stream_logits(eng, toks, [])                                 # every token alone, through the cache / state
    assert mc.rel_err(whole, ref) < F32_TOL and mc.rel_err(single, ref) < F32_TOL
    assert mc.rel_err(whole, single) < 2e-5


@pytest.mark.parametrize("portions", [[2] * 40, [63, 2, 63, 2], [64, 64], [1, 65, 1, 2, 59], [129, 2], [39, 1, 41, 9]])
def test_portions_of_several_sizes(cuda_device, portions):
    wt = mc.weights(FULL, 4)
    toks = mc.tokens_for(FULL, 140, seed=6)
    ref = mc.oracle_logits(FULL, wt, toks)
    eng = mc.build_engine(FULL, wt, torch.float32, cuda_device, prefill_chunk=96)   # 129 is cut by the engine too
    assert mc.rel_err(mc.stream_logits(eng, toks, portions), ref) < F32_TOL


def test_unequal_batches_equal_each_request_alone(cuda_device):
    wt = mc.weights(FULL, 7)
    seqs = [mc.tokens_for(FULL, n, seed=10 + n) for n in (1, 37, 130, 66)]
    eng = mc.build_engine(FULL, wt, torch.float32, cuda_device)
    alone = [mc.stream_logits(eng, s, [len(s)]) for s in seqs]
    # together: every step brings a different mix of portion sizes; request 0 joins late, request 2 skips a step
    streams = [eng.open_stream() for _ in seqs]
    got = [[] for _ in seqs]
    at = [0] * len(seqs)
    plan = [{1: 5, 2: 64}, {0: 1, 1: 1, 2: 2, 3: 30}, {1: 31, 3: 36}, {2: 64, 3: 0}]
    for step in plan:
        entries, who = [], []
        for i, k in step.items():
            if k:
                entries.append((streams[i], seqs[i][at[i]:at[i] + k], list(range(k))))
                who.append((i, k))
                at[i] += k
        lg = eng.feed(entries).double().cpu()
        r = 0
        for i, k in who:
            got[i].append(lg[r:r + k])
            r += k
    assert at == [len(s) for s in seqs]
    for i, s in enumerate(streams):
        eng.close_stream(s)
        assert mc.rel_err(torch.cat(got[i]), alone[i]) < 2e-5, f"request {i} depends on its batch"
    assert mc.rel_err(alone[2], mc.oracle_logits(FULL, wt, seqs[2])) < F32_TOL


def test_pages_and_slots_are_reused(cuda_device):
    """Two slots and five pages for eight sequences: every later sequence runs in a slot whose memory and convolution inputs
    another one left, and on pages that held other keys and values."""
    wt = mc.weights(FULL, 8)
    eng = mc.build_engine(FULL, wt, torch.float32, cuda_device, max_batch=2, max_seq_len=192, n_pages=1 + 5)
    lens = [100, 70, 5, 128, 64, 1, 150, 65]
    for k, n in enumerate(lens):
        toks = mc.tokens_for(FULL, n, seed=40 + k)
        ref = mc.oracle_logits(FULL, wt, toks)
        held = eng.open_stream()
        eng.feed([(held, mc.tokens_for(FULL, 60 + k, seed=k), [])])          # a neighbour that dirties the other slot
        got = mc.stream_logits(eng, toks, [max(1, n // 2), 2])
        eng.close_stream(held)
        assert mc.rel_err(got, ref) < F32_TOL, f"sequence {k}"
        assert len(eng.free_pages) == 5 and len(eng.free_slots) == 2


# ---- edges made to stand out ------------------------------------------------------------------------------------------
PLANS = ([330], [63, 1, 1, 63, 2, 126], [64, 64, 64, 64], [199, 2, 54, 2], [250])       # the rest one by one


@pytest.mark.parametrize("window", [1, 33, 64, 65, 200])
def test_window_edges_and_the_constant_sink(cuda_device, window):
    """Peaked scores (a large score scale) so that single keys carry a row's weight; the oracle with a window one longer or
    one shorter, or without the one in the denominator, is far outside the tolerance, so a key that is one position off at
    the edge shows, in portions of a prompt and in single decoded tokens, at page borders and inside pages."""
    config = mc.model([P(heads=4, kv_heads=2, dim=12, vdim=10, window=window, scale=0.9)], width=40)
    wt = mc.weights(config, 19)
    wt["l0.mix.right.out"] = mc.bf16_round(wt["l0.mix.right.out"] * 0.1)                  # the attention decides
    toks = mc.tokens_for(config, 330, seed=3)
    ref = mc.oracle_logits(config, wt, toks)
    for other in ([window + 1] if window == 1 else [window - 1, window + 1]):
        wrong = mc.oracle_logits(mc.replaced(config, ["layers", 0, "mixer", "left", "mask", "size"], other), wt, toks)
        assert mc.rel_err(wrong[window:], ref[window:]) > 100 * F32_TOL
        assert ((wrong - ref).abs().amax(-1)[window:] > 1e-3).float().mean() > 0.5        # most positions, not one
    plain = mo.sink_attention
    try:
        mo.sink_attention = lambda *a: plain(*a, sink=0.0)
        assert mc.rel_err(mc.oracle_logits(config, wt, toks), ref) > 100 * F32_TOL
    finally:
        mo.sink_attention = plain
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    for portions in PLANS:
        assert mc.rel_err(mc.stream_logits(eng, toks, portions), ref) < F32_TOL
    eng16 = mc.build_engine(config, wt, torch.bfloat16, cuda_device)
    assert mc.rel_err(mc.stream_logits(eng16, toks, [199, 2, 54, 2]), ref) < BF16_TOL


def test_one_far_key_inside_the_window_stands_out(cuda_device):
    """One token whose key is long and whose queries ask for it: the positions up to window - 1 behind it see it, the next
    one does not.  The token sits at several places of a page, and the asking tokens come in portions and one by one."""
    config = mc.model([P(heads=2, kv_heads=1, dim=8, vdim=8, window=100, rot_dims=0, scale=1.0)], width=32, vocab=40)
    wt = mc.weights(config, 5)
    wt["l0.mix.left.q"] *= 0.3
    wt["l0.mix.right.out"] = mc.bf16_round(wt["l0.mix.right.out"] * 0.1)
    # token 7 is what the keys answer to, token 9 what the queries ask with
    h7 = mo.rms_unit(wt["embed"][7], 1e-5) * wt["l0.norm1"]
    h9 = mo.rms_unit(wt["embed"][9], 1e-5) * wt["l0.norm1"]
    c = torch.ones(8, dtype=torch.float64)
    wt["l0.mix.left.k"] = mc.bf16_round(wt["l0.mix.left.k"] * 0.3 + 2.0 * torch.outer(c, h7) / (h7 @ h7))
    wt["l0.mix.left.q"] = mc.bf16_round(wt["l0.mix.left.q"] + 2.0 * torch.outer(torch.cat([c, c]), h9) / (h9 @ h9))
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    for place in (0, 1, 62, 63, 64, 65):
        toks = [t if t not in (7, 9) else 3 for t in mc.tokens_for(config, 190, seed=place)]
        toks[place] = 7
        for p in (place + 50, place + 98, place + 99, place + 100, place + 101):
            toks[p] = 9
        ref = mc.oracle_logits(config, wt, toks)
        other = list(toks)
        other[place] = 3
        moved = (mc.oracle_logits(config, wt, other) - ref).abs().amax(-1)
        assert moved[place + 99] > 0.05 and moved[place + 100] < 0.5 * moved[place + 99]
        for portions in ([190], [place + 99, 2], [place + 100, 2], [place + 1], [64, 64]):
            assert mc.rel_err(mc.stream_logits(eng, toks, portions), ref) < F32_TOL


def test_rotation_follows_the_position(cuda_device):
    """Fast rotations on every channel: a key or query turned by a neighbouring position's angle, or pairs taken in another
    layout, move the scores by O(1)."""
    config = mc.model([P(heads=2, kv_heads=1, dim=12, vdim=10, rot_dims=12, base=3.0, window=90, scale=0.8)], width=40)
    wt = mc.weights(config, 23)
    toks = mc.tokens_for(config, 200, seed=2)
    ref = mc.oracle_logits(config, wt, toks)
    for path, value in ((["layers", 0, "mixer", "left", "rot", "base"], 3.3), (["layers", 0, "mixer", "left", "rot", "dims"], 10)):
        assert mc.rel_err(mc.oracle_logits(mc.replaced(config, path, value), wt, toks), ref) > 100 * F32_TOL
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    for portions in ([200], [1, 2, 62, 3, 64], [130]):
        assert mc.rel_err(mc.stream_logits(eng, toks, portions), ref) < F32_TOL


@pytest.mark.parametrize("shift,far", [(-6.0, True), (2.0, False)])
def test_far_tokens_in_the_memory(cuda_device, shift, far):
    """Decays close to 1 and keys of 64 channels (later writes hardly erase): the memory at token 300 still holds the first tokens, so a state (or the convolution's last
    inputs) that is lost, reset or not carried across portions shows at every later position.  A second model with strong
    decay exercises the other end."""
    config = mc.model([P(window=5, r_heads=4, r_kv_heads=2, r_dim=64, r_vdim=8, conv=4)], width=40)
    wt = mc.weights(config, 11)
    wt["l0.mix.right.A_log"] = mc.bf16_round(wt["l0.mix.right.A_log"] + shift)
    wt["l0.mix.left.out"] = mc.bf16_round(wt["l0.mix.left.out"] * 0.1)
    toks = mc.tokens_for(config, 300, seed=4)
    ref = mc.oracle_logits(config, wt, toks)
    if far:
        other = [(toks[0] + 1) % config["vocab"]] + toks[1:]
        assert mc.rel_err(mc.oracle_logits(config, wt, other)[250:], ref[250:]) > 20 * F32_TOL
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    assert mc.rel_err(mc.stream_logits(eng, toks, [300]), ref) < F32_TOL
    assert mc.rel_err(mc.stream_logits(eng, toks, [7, 2, 120, 2, 9]), ref) < F32_TOL      # then 160 single tokens
    assert mc.rel_err(mc.stream_logits(eng, toks, [1, 1, 1, 2, 3, 100]), ref) < F32_TOL   # portions shorter than the taps


def test_first_tokens_and_one_token_sequences(cuda_device):
    wt = mc.weights(FULL, 12)
    eng = mc.build_engine(FULL, wt, torch.float32, cuda_device)
    for n in (1, 2, 3, 4, 5):
        toks = mc.tokens_for(FULL, n, seed=70 + n)
        ref = mc.oracle_logits(FULL, wt, toks)
        assert mc.rel_err(mc.stream_logits(eng, toks, [n]), ref) < F32_TOL
        assert mc.rel_err(mc.stream_logits(eng, toks, []), ref) < F32_TOL


# ---- the choice of experts --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("shift", [0.0, -4.0])
def test_routing_follows_scores_corrections_and_groups(cuda_device, shift):
    """Scores far apart and corrections large enough to change the choice, also with every choice score negative: a closed
    group that counts as zero, a group ranked by its best output alone, a weight that sees the correction, is not divided by
    the sum or misses the constant shows at once."""
    config = mc.model([P(mlp=M(experts=12, top=3, ff=12, groups=(4, 2), scale=1.7))], width=40)
    wt = mc.weights(config, 17)
    wt["l0.mlp.router"] = mc.bf16_round(wt["l0.mlp.router"] * 2.0)
    wt["l0.mlp.correction"] = mc.bf16_round(wt["l0.mlp.correction"] * 2.0 + shift)
    toks = mc.tokens_for(config, 120, seed=4)
    gaps = []
    ref = mc.oracle_logits(config, wt, toks, margins=gaps)
    clear = torch.tensor(gaps[0]) > 1e-4
    assert clear.float().mean() > 0.9
    other = dict(wt)
    other["l0.mlp.correction"] = torch.zeros(12, dtype=torch.float64)
    assert mc.rel_err(mc.oracle_logits(config, other, toks), ref) > 50 * F32_TOL
    for path, value in ((["layers", 0, "mlp", "router", "groups"], None), (["layers", 0, "mlp", "router", "scale"], 1.6)):
        assert mc.rel_err(mc.oracle_logits(mc.replaced(config, path, value), wt, toks), ref) > 50 * F32_TOL
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    assert mc.rel_err(mc.stream_logits(eng, toks, [100, 2])[clear], ref[clear]) < F32_TOL
    eng.unfused_router = True
    assert mc.rel_err(mc.stream_logits(eng, toks, [100, 2])[clear], ref[clear]) < F32_TOL


@pytest.mark.parametrize("experts,top,groups,keep", [(12, 3, 4, 2), (8, 8, 1, 1), (6, 2, 6, 3), (96, 7, 8, 3), (33, 4, 3, 1), (1, 1, 1, 1),
                                                     (260, 5, 4, 2), (80, 40, 2, 2)])
def test_choice_kernels(cuda_device, experts, top, groups, keep):
    """prl_moe_choose and prl_moe_router_choose alone, with sigmoid scores, groups ranked by their two best and weights
    divided by their sum: choices, weights and the grouping by expert."""
    from pipelinerl_b200 import _lib
    lib, n, W = _lib.load(), 70 if experts % 3 else 700, 48
    g = torch.Generator().manual_seed(experts)
    x, wr = torch.randn(n, W, generator=g), torch.randn(experts, W, generator=g) * 0.4
    corr = torch.randn(experts, generator=g) - 2.0
    z = x.double() @ wr.double().T
    want = [mo.choose(torch.sigmoid(z[t]), corr.double(), dict(top=top, groups=dict(count=groups, keep=keep))) for t in range(n)]
    d, i32 = cuda_device, dict(dtype=torch.int32, device=cuda_device)
    xd, wd, cd, zd = x.to(d), wr.to(d), corr.to(d), z.float().to(d)
    st = _lib.stream_ptr()
    for ready in (True, False):
        sel, perm = torch.full((top, n), -1, **i32), torch.full((top * n,), -1, **i32)
        wsel, meta = torch.zeros(top, n, device=d), torch.zeros(4, **i32)
        tiles = torch.zeros(3 * int(lib.prl_moe_max_tiles(top * n, experts)), **i32)
        rule = (top, groups, keep, 2, 1, 1, 1.7, 64, sel.data_ptr(), wsel.data_ptr(), perm.data_ptr(), meta.data_ptr(), tiles.data_ptr(), st)
        if ready:
            _lib.check(lib.prl_moe_choose(zd.data_ptr(), experts, cd.data_ptr(), n, experts, experts, *rule))
        else:
            _lib.check(lib.prl_moe_router_choose(xd.data_ptr(), 1, wd.data_ptr(), 1, cd.data_ptr(), n, W, experts, experts, *rule))
        s, w = sel.cpu(), wsel.double().cpu()
        assert s.T.tolist() == want
        for t in range(n):
            sc = torch.sigmoid(z[t, want[t]])
            assert torch.allclose(w[:, t], sc / sc.sum() * 1.7, atol=1e-5)
        order = [p for e in range(experts) for p in range(top * n) if s.view(-1)[p] == e]
        assert perm.tolist() == order and meta[1].item() == top * n


# ---- the serving mode --------------------------------------------------------------------------------------------------
BIG = mc.model([P(heads=8, kv_heads=2, dim=32, vdim=32, rot_dims=16, window=100, r_heads=4, r_kv_heads=2, r_dim=64, r_vdim=32, conv=4,
                  mlp=M(experts=3, top=3, ff=64, groups=None)),
                P(heads=4, kv_heads=2, dim=48, vdim=64, rot_dims=48, window=120, r_heads=4, r_kv_heads=4, r_dim=32, r_vdim=64, conv=4),
                P(heads=4, kv_heads=4, dim=32, vdim=48, rot_dims=32, window=70, r_heads=2, r_kv_heads=1, r_dim=48, r_vdim=64, conv=3,
                  mlp=M(experts=8, top=2, ff=96, groups=(4, 2)))], vocab=200, width=128)


@pytest.mark.parametrize("plain_gemm", [False, True])
def test_bf16_serving_mode(cuda_device, plain_gemm):
    """bf16 operands and cache with the tensor-core GEMMs (and with the CUDA-core GEMM) against the float64 oracle.  Only the
    last layer's router has a choice to make, so a token whose choice is closer than bf16 rounding can tell apart touches
    only its own logits; the oracle reports the gaps and those positions are left out."""
    wt = mc.weights(BIG, 13)
    toks = mc.tokens_for(BIG, 300, seed=8)
    gaps = []
    ref = mc.oracle_logits(BIG, wt, toks, margins=gaps)
    assert min(gaps[0]) == math.inf
    clear = torch.tensor(gaps[-1]) > 0.03
    assert clear.float().mean().item() > 0.7
    eng = mc.build_engine(BIG, wt, torch.bfloat16, cuda_device, prefill_chunk=512)
    eng.force_plain_gemm = plain_gemm
    whole = mc.stream_logits(eng, toks, [300])
    assert mc.rel_err(whole[clear], ref[clear]) < BF16_TOL
    assert mc.rel_err(mc.stream_logits(eng, toks, [100, 2, 30])[clear], ref[clear]) < BF16_TOL
    # the bf16 engine is about as close to the oracle as the oracle with only its matrix products' inputs rounded
    least = mc.rel_err(mc.oracle_logits(BIG, wt, toks, round_in=mc.bf16_round)[clear], ref[clear])
    assert mc.rel_err(whole[clear], ref[clear]) < 3 * least + 1e-3


def test_grouped_tensor_core_experts_in_long_prompts(cuda_device):
    """More routed pairs per expert than the few-row grouped GEMM is for: the tcgen05 grouped GEMM with the gelu epilogue
    against the few-row kernel on the same weights."""
    config = mc.model([P(mlp=M(experts=4, top=2, ff=128, groups=(2, 2)))], width=128)
    wt = mc.weights(config, 6)
    toks = mc.tokens_for(config, 300, seed=5)
    eng = mc.build_engine(config, wt, torch.bfloat16, cuda_device, prefill_chunk=512)
    eng.moe_tc_rows = 1 << 30
    few = mc.stream_logits(eng, toks, [300])
    eng.moe_tc_rows = 1
    many = mc.stream_logits(eng, toks, [300])
    assert mc.rel_err(many, few) < 5e-3
    gaps = []
    ref = mc.oracle_logits(config, wt, toks, margins=gaps)
    clear = torch.tensor(gaps[0]) > 0.03
    assert mc.rel_err(many[clear], ref[clear]) < BF16_TOL


@pytest.mark.parametrize("dim,vdim,window", [(32, 32, 100), (64, 64, 64), (128, 128, 37), (80, 48, 90), (48, 96, 33), (16, 16, 200)])
def test_tensor_core_prompt_attention(cuda_device, dim, vdim, window):
    """bf16 with head sizes the tensor-core prompt kernel is built for, peaked scores over five page borders, against the
    CUDA-core kernel on the same cache (they differ by the bf16 rounding of the softmax weights) and against the oracle."""
    config = mc.model([P(heads=4, kv_heads=2, dim=dim, vdim=vdim, rot_dims=dim // 2, window=window, scale=1.5 * dim ** -0.5)], width=64)
    wt = mc.weights(config, 9)
    toks = mc.tokens_for(config, 330, seed=3)
    ref = mc.oracle_logits(config, wt, toks)
    eng = mc.build_engine(config, wt, torch.bfloat16, cuda_device, prefill_chunk=512)
    plans = ([330], [63, 17, 16, 130, 65, 20, 3, 2], [300])                 # the rest one by one
    eng.tc_prompt[0] = False                                                # heads of 128 have another test
    fast = [mc.stream_logits(eng, toks, p) for p in plans]
    eng.lib.prl_attn_any_tensor_cores(0)
    try:
        plain = [mc.stream_logits(eng, toks, p) for p in plans]
    finally:
        eng.lib.prl_attn_any_tensor_cores(1)
    for f, p in zip(fast, plain):
        assert 0 < mc.rel_err(f, p) < 0.25 * BF16_TOL                        # two kernels, the same result
        assert mc.rel_err(f, ref) < BF16_TOL and mc.rel_err(p, ref) < BF16_TOL


CELLS = [(4, 2, 12, 8, 3), (3, 1, 10, 13, 4), (2, 2, 32, 48, 2), (4, 2, 64, 64, 4), (2, 1, 128, 128, 4), (2, 1, 40, 132, 1), (1, 1, 200, 20, 4),
         (6, 2, 5, 40, 6)]       # heads, q / k heads, key size, value size, taps


@pytest.mark.parametrize("heads,kv,dk,dv,taps", CELLS)
def test_pieces_of_the_gated_delta_rule(cuda_device, heads, kv, dk, dv, taps):
    """Long portions as side-by-side pieces (off in fp32 unless asked for) against the oracle and the token-by-token walk: one
    piece that is not full, several, pieces of other lengths, portions that continue a state, and single tokens of another
    sequence beside them.  Memories that last (decays near one) make a wrong state at a piece's border show in every row
    behind it."""
    config = mc.model([P(window=5, r_heads=heads, r_kv_heads=kv, r_dim=dk, r_vdim=dv, conv=taps)], width=40)
    for shift in (-3.0, 1.0):
        wt = mc.weights(config, 27)
        wt["l0.mix.right.A_log"] = mc.bf16_round(wt["l0.mix.right.A_log"] + shift)
        wt["l0.mix.left.out"] = mc.bf16_round(wt["l0.mix.left.out"] * 0.1)
        toks, other = mc.tokens_for(config, 300, seed=21), mc.tokens_for(config, 20, seed=22)
        ref, oref = mc.oracle_logits(config, wt, toks), mc.oracle_logits(config, wt, other)
        eng = mc.build_engine(config, wt, torch.float32, cuda_device, prefill_chunk=320)
        walked = mc.stream_logits(eng, toks, [300])
        eng.split_scan, eng.split_min_rows = True, 2
        for step in (64, 23):
            eng.piece_tokens = step
            for portions in ([300], [64, 65, 2, 100], [130, 1, 2, 3]):
                got = mc.stream_logits(eng, toks, portions)
                assert mc.rel_err(got, ref) < F32_TOL and mc.rel_err(got, walked) < 2e-5
        a, b = eng.open_stream(), eng.open_stream()
        rows = [[], []]
        for k, (na, nb) in enumerate([(100, 5), (70, 1), (2, 1), (128, 13)]):
            at, bt = sum(x.shape[0] for x in rows[0]), sum(x.shape[0] for x in rows[1])
            lg = eng.feed([(a, toks[at:at + na], list(range(na))), (b, other[bt:bt + nb], list(range(nb)))]).double().cpu()
            rows[0].append(lg[:na]); rows[1].append(lg[na:])
        eng.close_stream(a); eng.close_stream(b)
        assert mc.rel_err(torch.cat(rows[0]), ref) < F32_TOL and mc.rel_err(torch.cat(rows[1]), oref) < F32_TOL


@pytest.mark.parametrize("heads,kv,dk,dv,taps", CELLS)
def test_token_step_of_the_gated_delta_rule(cuda_device, heads, kv, dk, dv, taps):
    """The one-kernel token step against the separate kernels and the oracle, behind a prompt, with an idle slot beside it, and
    with the state handed from one path to the other in the middle."""
    config = mc.model([P(window=5, r_heads=heads, r_kv_heads=kv, r_dim=dk, r_vdim=dv, conv=taps)], width=40)
    wt = mc.weights(config, 28)
    wt["l0.mix.left.out"] = mc.bf16_round(wt["l0.mix.left.out"] * 0.1)
    toks = mc.tokens_for(config, 60, seed=23)
    ref = mc.oracle_logits(config, wt, toks)
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    assert eng.lib.prl_gated_delta_step_fits(heads, kv, dk, dv, taps)
    assert mc.rel_err(mc.stream_logits(eng, toks, []), ref) < F32_TOL
    eng.unfused_cell = True
    separate = mc.stream_logits(eng, toks, [])
    eng.unfused_cell = False
    assert mc.rel_err(mc.stream_logits(eng, toks, []), separate) < 2e-5
    s, out, at = eng.open_stream(), [], 0
    for k in (7, 1, 1, 1, 2, 1, 1, 20):
        eng.unfused_cell = at % 2 == 0
        out.append(eng.feed([(s, toks[at:at + k], list(range(k)))]))
        at += k
    eng.close_stream(s)
    assert mc.rel_err(torch.cat(out).double().cpu(), ref[:at]) < F32_TOL


@pytest.mark.parametrize("heads,kv_heads,window", [(2, 1, 37), (4, 1, 64), (8, 1, 129), (3, 3, 200), (16, 1, 90), (4, 2, 0), (4, 2, 1), (2, 2, 128)])
def test_tcgen05_prompt_attention(cuda_device, heads, kv_heads, window):
    """Heads of 128 in bf16: the tcgen05 prompt kernel with its window, the constant sink and the head gates, against the
    CUDA-core kernel on the same cache and against the oracle.  Portions start inside a page and a key step, rows of a tile
    lose keys of the first step to the window, and steps of a tile may be hidden from some of its rows altogether."""
    config = mc.model([P(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, rot_dims=32, window=window, scale=1.5 * 128 ** -0.5)], width=64)
    wt = mc.weights(config, 9)
    toks = mc.tokens_for(config, 520, seed=3)
    ref = mc.oracle_logits(config, wt, toks)
    eng = mc.build_engine(config, wt, torch.bfloat16, cuda_device, prefill_chunk=520, max_seq_len=576)
    assert eng.tc_prompt[0]
    plans = ([520], [63, 130, 257, 3, 60], [300, 200])                     # the rest one by one
    fast = [mc.stream_logits(eng, toks, p) for p in plans]
    eng.force_plain_attn = True
    eng.lib.prl_attn_any_tensor_cores(0)
    try:
        plain = mc.stream_logits(eng, toks, [520])
    finally:
        eng.lib.prl_attn_any_tensor_cores(1)
    for f in fast:
        assert mc.rel_err(f, plain) < 0.5 * BF16_TOL and mc.rel_err(f, ref) < BF16_TOL
    assert (fast[0] != plain).any()


@pytest.mark.parametrize("shift", [0.0, -150.0, 150.0])
@pytest.mark.parametrize("heads,kv_heads,pos0,rows,window", [(4, 2, 0, 200, 37), (2, 2, 130, 300, 64), (8, 1, 77, 40, 129), (4, 4, 500, 150, 0)])
def test_tcgen05_prompt_attention_alone(cuda_device, shift, heads, kv_heads, pos0, rows, window):
    """The tcgen05 prompt kernel alone, with and without a sink and gates, on scores that are all far below (or far above) zero:
    rows of a tile that see nothing in its first steps must take their reference from the first step they do see."""
    from pipelinerl_b200 import _lib
    lib, d = _lib.load(), cuda_device
    g = torch.Generator().manual_seed(rows)
    S, R = pos0 + rows, heads // kv_heads
    c = torch.sign(torch.randn(128, generator=g))
    q = mc.bf16_round(torch.randn(rows, heads, 128, generator=g) * 0.3 + c * (0.5 if shift else 0.0))
    k = mc.bf16_round(torch.randn(S, kv_heads, 128, generator=g) * 0.3 + c * (shift / 64.0))
    v = mc.bf16_round(torch.randn(S, kv_heads, 128, generator=g))
    sink, gate = torch.randn(heads, generator=g) + shift, torch.randn(rows, heads, generator=g)
    pages = -(-S // 64)
    order = torch.randperm(pages, generator=g) + 1
    kv = torch.zeros(2, pages + 1, kv_heads, 64, 128, dtype=torch.bfloat16)
    for t in range(S):
        kv[0, order[t // 64], :, t % 64], kv[1, order[t // 64], :, t % 64] = k[t].bfloat16(), v[t].bfloat16()
    scale = 1.0                                                             # scores around `shift`
    i32 = dict(dtype=torch.int32, device=d)
    bt = order.int().view(1, -1).to(d)
    one = lambda x: torch.tensor([x], **i32)
    ss, sl, sp, slot = one(0), one(rows), one(pos0), one(0)
    qd, kvd, sd, gd = q.bfloat16().to(d), kv.to(d), sink.to(d), gate.to(d)
    for use in (False, True):
        out = torch.zeros(rows, heads, 128, dtype=torch.bfloat16, device=d)
        _lib.check(lib.prl_paged_attn_prefill_tc_gated(qd.data_ptr(), rows, kvd.data_ptr(), pages + 1, 1, 0, bt.data_ptr(), pages, ss.data_ptr(),
                                                       sl.data_ptr(), sp.data_ptr(), slot.data_ptr(), 1, rows, heads, kv_heads, 128, 64, scale,
                                                       window, sd.data_ptr() if use else None, gd.data_ptr() if use else None, heads,
                                                       out.data_ptr(), _lib.stream_ptr()))
        back = (pos0 + torch.arange(rows))[:, None] - torch.arange(S)[None, :]
        see = (back >= 0) & ((back < window) if window else torch.ones_like(back, dtype=torch.bool))
        ref = torch.zeros(rows, heads, 128, dtype=torch.float64)
        for h in range(heads):
            s = (q[:, h].double() @ k[:, h // R].double().T * scale).masked_fill(~see, -math.inf)
            if use:
                s = torch.cat([s, sink[h].double().expand(rows, 1)], 1)
            w = torch.softmax(s, 1)[:, :S]
            ref[:, h] = w @ v[:, h // R].double() * (torch.sigmoid(gate[:, h].double())[:, None] if use else 1.0)
        err = (out.double().cpu() - ref).abs().max().item()
        assert err < 0.03, (use, err)


def test_long_decoding(cuda_device):
    """A short prompt and 400 single tokens over six page borders and several windows, in fp32 against the oracle."""
    config = mc.model([P(mlp=M(), window=150), P(window=64)])
    wt = mc.weights(config, 31)
    toks = mc.tokens_for(config, 420, seed=12)
    eng = mc.build_engine(config, wt, torch.float32, cuda_device)
    assert mc.rel_err(mc.stream_logits(eng, toks, [20]), mc.oracle_logits(config, wt, toks)) < F32_TOL


def test_greedy_generation_through_the_scheduler(cuda_device):
    """add_request / run_prefill / CUDA-graph token steps / harvest, five prompts on two slots (slots and pages are reused,
    idle slots ride along in the step), greedy ids and log-probabilities of the capped logits against the oracle wherever
    its top-2 margin is not a rounding matter."""
    from pipelinerl_b200.engine import SamplingParams
    wt = mc.weights(FULL, 14)
    eng = mc.build_engine(FULL, wt, torch.float32, cuda_device, max_batch=2, max_seq_len=256, use_cuda_graph=True, prefill_chunk=64)
    prompts = [mc.tokens_for(FULL, n, seed=90 + n) for n in (1, 5, 70, 130, 64)]
    outs = eng.generate(prompts, SamplingParams(max_tokens=6, greedy=True, ignore_eos=True))
    assert len(eng.free_slots) == 2 and len(eng.free_pages) == eng.n_pages - 1
    for p, r in zip(prompts, outs):
        assert len(r.output_ids) == 6 and r.finish_reason == "length"
        seq = list(p)
        for tok, lp in zip(r.output_ids, r.output_logprobs):
            lg = mc.oracle_logits(FULL, wt, seq)[-1]
            top = torch.topk(lg, 2)
            if (top.values[0] - top.values[1]).item() > 1e-3:
                assert tok == top.indices[0].item()
            assert abs(lp - torch.log_softmax(lg, -1)[tok].item()) < 1e-3
            seq.append(tok)


def test_trace_runner_command_line(cuda_device, tmp_path):
    """bin/trace_run on a checkpoint folder: registry, safetensors loader, streams, output files, in both dtypes."""
    config = mc.model([P(mlp=M(experts=4, top=1, ff=8, groups=(2, 1))), P(window=33)], vocab=64, width=40)
    wt = mc.weights(config, 15)
    mc.write_checkpoint(tmp_path, config, wt)
    a, b = mc.tokens_for(config, 90, seed=1), mc.tokens_for(config, 20, seed=2)
    steps = [
        dict(step=0, entries=[dict(id="a", tokens=a[:50], want=[0, 49])], end=[]),
        dict(step=1, entries=[dict(id="a", tokens=a[50:52], want=[]), dict(id="b", tokens=b[:19], want=[3])], end=[]),
        dict(step=2, entries=[dict(id="b", tokens=b[19:], want=[0]), dict(id="a", tokens=a[52:], want=[37])], end=["a", "b"]),
        dict(step=3, entries=[dict(id="c", tokens=b, want=[19])], end=["c"]),
    ]
    gaps = [[], []]
    ra, rb = (mc.oracle_logits(config, wt, t, margins=m) for t, m in zip((a, b), gaps))
    expect = {0: torch.stack([ra[0], ra[49]]), 1: rb[3:4], 2: torch.stack([rb[19], ra[89]]), 3: rb[19:20]}
    root = __import__("pathlib").Path(__file__).resolve().parent.parent
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        out = tmp_path / dtype
        p = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=900)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(4)]
        import numpy as np
        for i, ref in expect.items():
            got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, config["vocab"])
            assert got.shape == ref.shape and mc.rel_err(got, ref) < tol
