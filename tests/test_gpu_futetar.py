"""The Futetar decoders on the hybrid engine (pipelinerl_b200/hybrid.py and its kernels) against
oracle/futetar_oracle.py: each mechanism alone, whole prompts against token-by-token decoding, portions down to two
tokens, unequal batches against each request alone, pages and slots that are given back and taken again, keys far away
and at page borders, caches that several layers read, the choice of experts, the carried memory, the first tokens, long
decoding, awkward sizes, the bf16 serving mode, greedy generation through the engine's scheduler, and the trace runner."""
import json
import subprocess
import sys

import pytest
import torch

from oracle import futetar_oracle as fo
from tests import futetar_cases as fc

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4      # fp32 kernels against the float64 oracle
BF16_TOL = 8e-2     # bf16 operands / cache: rounding of activations dominates
C, A, D, M = fc.cell, fc.attention, fc.dense, fc.moe


# ---- each mechanism alone ---------------------------------------------------------------------------------------
def _mechanisms():
    return {
        "cell": fc.model([C()]),
        "cell_one_head_values_smaller_than_keys": fc.model([C(heads=1, dim=24, vdim=5, gate_cap=3.0)]),
        "cell_many_small_heads": fc.model([C(heads=12, dim=4, vdim=8)]),
        "cell_wide_head": fc.model([C(heads=2, dim=130, vdim=96)], width=40),
        "cell_one_channel": fc.model([C(heads=5, dim=1, vdim=1)]),
        "cell_high_cap": fc.model([C(gate_cap=30.0)]),
        "attention": fc.model([A()]),
        "attention_every_head_its_own_keys_plain_rotation": fc.model([A(heads=4, kv_heads=4, dim=8, vdim=8, rot_dims=8, scaling=None)]),
        "attention_one_key_head_two_rotated_channels": fc.model([A(heads=5, kv_heads=1, dim=14, vdim=6, rot_dims=2)]),
        "attention_without_rotation": fc.model([A(rot_dims=0)]),
        "attention_wide_heads": fc.model([A(heads=2, kv_heads=1, dim=80, vdim=136, rot_dims=80, base=1e4, scaling=(8.0, 1.0, 4.0, 64))], width=40),
        "shared_cache": fc.model([A(), A(kv_from=0), A(heads=3, kv_from=0)]),
        "shared_cache_across_cells": fc.model([C(), A(), A(heads=3, kv_heads=1), C(), A(heads=9, kv_from=1), A(kv_heads=1, kv_from=2)]),
        "dense": fc.model([C(mlp=D())]),
        "dense_beside_attention": fc.model([A(mlp=D(ff=7))]),
        "routed": fc.model([A(mlp=M())]),
        "routed_top1_no_groups_no_identity_no_shared": fc.model([C(mlp=M(experts=7, top=1, ff=10, identity=0, groups=None, shared=0))]),
        "routed_one_group_kept": fc.model([C(mlp=M(experts=9, top=3, ff=9, identity=3, groups=(4, 1)))]),
        "routed_groups_of_one": fc.model([C(mlp=M(experts=5, top=2, ff=8, identity=1, groups=(6, 3), shared=1))]),
        "routed_everything": fc.model([C(mlp=M(experts=3, top=5, ff=9, identity=2, groups=(5, 5)))]),
        "routed_mostly_identity": fc.model([A(mlp=M(experts=1, top=4, ff=9, identity=7, groups=(2, 2)))]),
        "routed_many_outputs": fc.model([C(mlp=M(experts=70, top=8, ff=6, identity=10, groups=(8, 4)))]),
        "odd_width": fc.model([A(mlp=M()), C(mlp=D(ff=11)), C()], vocab=61, width=50),
        "every_kind_in_another_order": fc.model([C(mlp=M()), A(mlp=D()), C(mlp=D()), A(kv_from=1, mlp=M(experts=4, identity=0)), A(heads=3, kv_heads=3),
                                                 A(heads=6, kv_heads=3, kv_from=4)]),
    }


@pytest.mark.parametrize("name", sorted(_mechanisms()))
def test_each_mechanism_matches_the_oracle_fp32(cuda_device, name):
    config = _mechanisms()[name]
    wt = fc.weights(config, seed=len(name))
    toks = fc.tokens_for(config, 150)
    res = []
    ref = fc.oracle_logits(config, wt, toks, residuals=res)
    eng = fc.build_engine(config, wt, torch.float32, cuda_device)
    assert fc.rel_err(fc.stream_logits(eng, toks, [150]), ref) < F32_TOL
    assert fc.rel_err(fc.stream_logits(eng, toks, [2, 3, 61, 2, 7, 64, 2]), ref) < F32_TOL     # then one by one
    # the residual stream after every layer of a whole prompt
    s = fc.stage_stream(eng, toks[:20])
    got = []
    eng._forward_rows([(s, 0, 20)], [], trace=got)
    eng.close_stream(s)
    assert len(got) == len(res)
    for a, b in zip(got, res):
        assert (a.double().cpu() - b[:20]).abs().max().item() < 1e-4 * max(1.0, b.abs().max().item())


FULL = fc.model([C(mlp=D()), A(mlp=M()), C(heads=2, dim=12, vdim=9, mlp=M(experts=5, top=2, identity=1, groups=(3, 2), ff=16)),
                 A(heads=3, kv_from=1, mlp=D(ff=24)), A(heads=4, kv_heads=2, dim=16, vdim=20, rot_dims=16), C()], vocab=80, width=64)


def test_prefill_against_token_by_token_decoding(cuda_device):
    wt = fc.weights(FULL, 3)
    toks = fc.tokens_for(FULL, 140, seed=5)
    ref = fc.oracle_logits(FULL, wt, toks)
    eng = fc.build_engine(FULL, wt, torch.float32, cuda_device)
    whole = fc.stream_logits(eng, toks, [140])
    single = fc.stream_logits(eng, toks, [])                                 # every token alone, through the cache / state
    assert fc.rel_err(whole, ref) < F32_TOL and fc.rel_err(single, ref) < F32_TOL
    assert fc.rel_err(whole, single) < 2e-5


@pytest.mark.parametrize("portions", [[2] * 40, [63, 2, 63, 2], [64, 64], [1, 65, 1, 2, 59], [129, 2], [39, 1, 41, 9]])
def test_portions_of_several_sizes(cuda_device, portions):
    wt = fc.weights(FULL, 4)
    toks = fc.tokens_for(FULL, 140, seed=6)
    ref = fc.oracle_logits(FULL, wt, toks)
    eng = fc.build_engine(FULL, wt, torch.float32, cuda_device, prefill_chunk=96)   # 129 is cut by the engine too
    assert fc.rel_err(fc.stream_logits(eng, toks, portions), ref) < F32_TOL


def test_unequal_batches_equal_each_request_alone(cuda_device):
    wt = fc.weights(FULL, 7)
    seqs = [fc.tokens_for(FULL, n, seed=10 + n) for n in (1, 37, 130, 66)]
    eng = fc.build_engine(FULL, wt, torch.float32, cuda_device)
    alone = [fc.stream_logits(eng, s, [len(s)]) for s in seqs]
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
        assert fc.rel_err(torch.cat(got[i]), alone[i]) < 2e-5, f"request {i} depends on its batch"
    assert fc.rel_err(alone[2], fc.oracle_logits(FULL, wt, seqs[2])) < F32_TOL


def test_pages_and_slots_are_reused(cuda_device):
    """Two slots and five pages for eight sequences: every later sequence runs in a slot whose memory, normaliser and
    running maximum another one left, and on pages that held other keys and values."""
    wt = fc.weights(FULL, 8)
    eng = fc.build_engine(FULL, wt, torch.float32, cuda_device, max_batch=2, max_seq_len=192, n_pages=1 + 5)
    lens = [100, 70, 5, 128, 64, 1, 150, 65]
    for k, n in enumerate(lens):
        toks = fc.tokens_for(FULL, n, seed=40 + k)
        ref = fc.oracle_logits(FULL, wt, toks)
        held = eng.open_stream()
        eng.feed([(held, fc.tokens_for(FULL, 60 + k, seed=k), [])])          # a neighbour that dirties the other slot
        got = fc.stream_logits(eng, toks, [max(1, n // 2), 2])
        eng.close_stream(held)
        assert fc.rel_err(got, ref) < F32_TOL, f"sequence {k}"
        assert len(eng.free_pages) == 5 and len(eng.free_slots) == 2


# ---- faults made to stand out ------------------------------------------------------------------------------------------
PLANS = ([330], [63, 1, 1, 63, 2, 126], [64, 64, 64, 64], [199, 2, 54, 2], [250])       # the rest one by one


@pytest.mark.parametrize("far", [0, 1, 63, 64, 127, 128, 191])
def test_a_far_key_stands_out(cuda_device, far):
    """One early token's key is the only one that matches the late tokens' queries (its direction is planted in the
    embedding), so at far positions nearly all the weight lies on that one key: a key that is lost, misplaced at a page
    border or read from another layer's cache changes those logits by O(1).  The second layer reads the same cache with
    queries of its own."""
    config = fc.model([A(heads=2, kv_heads=1, dim=8, vdim=10, rot_dims=0, scale=4.0), A(heads=4, kv_heads=1, dim=8, vdim=10, rot_dims=0,
                                                                                        scale=4.0, kv_from=0)], width=40, vocab=64)
    wt = fc.weights(config, 19)
    mark, ask = 1, 2                                            # the far token, and the token that every late position holds
    hk = fo.offset_norm(wt["embed"], wt["l0.norm1"], 1e-5)
    kdir = wt["l0.mix.k"] @ hk[mark]
    for name, heads in (("l0.mix.q", 2), ("l1.mix.q", 4)):      # queries of `ask` point at the key of `mark`
        q = wt[name].view(heads, 8, -1)
        wt[name] = fc.bf16_round(0.05 * q + kdir[None, :, None] * (hk[ask] / hk[ask].norm() ** 2)[None, None, :] * 4.0).reshape(heads * 8, -1)
    toks = [3 + t % 50 for t in fc.tokens_for(config, 260, seed=3)]
    toks[far] = mark
    for t in range(far + 3, 260, 2):
        toks[t] = ask
    late = [t for t in range(200, 260) if toks[t] == ask]
    ref = fc.oracle_logits(config, wt, toks)
    other = list(toks)
    other[far] = 7
    assert fc.rel_err(fc.oracle_logits(config, wt, other)[late], ref[late]) > 300 * F32_TOL
    eng = fc.build_engine(config, wt, torch.float32, cuda_device)
    for portions in ([260], [far + 1, 2, 62, 3, 64], [64, 64, 64], [130]):
        assert fc.rel_err(fc.stream_logits(eng, toks, portions), ref) < F32_TOL
    eng16 = fc.build_engine(config, wt, torch.bfloat16, cuda_device)
    assert fc.rel_err(fc.stream_logits(eng16, toks, [199, 2, 54, 2]), ref) < 2 * BF16_TOL


def test_rotation_follows_the_position(cuda_device):
    """Fast rotations: a key or query turned by a neighbouring position's angle, pairs taken in the wrong layout, or a
    scaling whose bands are misread move the scores by O(1); the shared cache holds turned keys."""
    config = fc.model([A(heads=2, kv_heads=1, dim=12, vdim=10, rot_dims=12, base=6.0, scaling=(4.0, 1.0, 3.0, 24), scale=1.0),
                       A(heads=3, kv_heads=1, dim=12, vdim=10, rot_dims=12, base=6.0, scaling=(4.0, 1.0, 3.0, 24), scale=1.2, kv_from=0)], width=40)
    wt = fc.weights(config, 23)
    toks = fc.tokens_for(config, 200, seed=2)
    ref = fc.oracle_logits(config, wt, toks)
    for key, value in (("base", 6.6), ("dims", 10)):
        wrong = fc.replaced(fc.replaced(config, ["layers", 0, "mixer", "rot", key], value), ["layers", 1, "mixer", "rot", key], value)
        assert fc.rel_err(fc.oracle_logits(wrong, wt, toks), ref) > 100 * F32_TOL
    for key, value in (("factor", 3.0), ("low", 1.6), ("high", 2.2), ("original", 30)):
        wrong = fc.replaced(fc.replaced(config, ["layers", 0, "mixer", "rot", "scaling", key], value), ["layers", 1, "mixer", "rot", "scaling", key], value)
        assert fc.rel_err(fc.oracle_logits(wrong, wt, toks), ref) > 100 * F32_TOL
    eng = fc.build_engine(config, wt, torch.float32, cuda_device)
    for portions in ([200], [1, 2, 62, 3, 64], [130]):
        assert fc.rel_err(fc.stream_logits(eng, toks, portions), ref) < F32_TOL


def test_layers_read_the_cache_they_name(cuda_device):
    """Two caches of one geometry: taking the other one, or the layer's own (absent) projections, shows at once."""
    config = fc.model([A(), A(), C(), A(kv_from=0), A(kv_from=1), A(kv_from=0)], width=48)
    wt = fc.weights(config, 29)
    toks = fc.tokens_for(config, 100, seed=7)
    ref = fc.oracle_logits(config, wt, toks)
    for layer in (3, 4, 5):
        wrong = fc.replaced(config, ["layers", layer, "mixer", "kv_from"], 1 if layer != 4 else 0)
        assert fc.rel_err(fc.oracle_logits(wrong, wt, toks), ref) > 100 * F32_TOL
    eng = fc.build_engine(config, wt, torch.float32, cuda_device)
    assert eng.k_pool[3] is eng.k_pool[0] and eng.k_pool[4] is eng.k_pool[1] and eng.v_pool[5] is eng.v_pool[0]
    for portions in ([100], [30, 2, 5], []):
        assert fc.rel_err(fc.stream_logits(eng, toks, portions), ref) < F32_TOL


def test_far_tokens_in_the_memory_cell(cuda_device):
    """Forget gates close to one: the memory at token 300 still holds the first tokens, so a state, normaliser or running
    maximum that is lost, reset or not carried across portions shows at every later position.  Then input gates that jump
    by several units (the maximum moves), and forgetting gates."""
    config = fc.model([C(heads=2, dim=12, vdim=9, gate_cap=11.0)], width=40)
    for fb, ib, spread, far in ((9.0, 0.0, 1.0, True), (6.0, -3.0, 4.0, False), (-1.0, 2.0, 2.0, False)):
        wt = fc.weights(config, 11)
        wt["l0.mix.f.b"] = fc.bf16_round(torch.full((2,), fb, dtype=torch.float64))
        wt["l0.mix.i.b"] = fc.bf16_round(torch.full((2,), ib, dtype=torch.float64))
        wt["l0.mix.i"] = fc.bf16_round(wt["l0.mix.i"] * spread)
        toks = fc.tokens_for(config, 300, seed=4)
        ref = fc.oracle_logits(config, wt, toks)
        if far:
            other = [(toks[0] + 1) % config["vocab"]] + toks[1:]
            assert fc.rel_err(fc.oracle_logits(config, wt, other)[250:], ref[250:]) > 20 * F32_TOL
        eng = fc.build_engine(config, wt, torch.float32, cuda_device)
        assert fc.rel_err(fc.stream_logits(eng, toks, [300]), ref) < F32_TOL
        assert fc.rel_err(fc.stream_logits(eng, toks, [7, 2, 120, 2, 9]), ref) < F32_TOL      # then 160 single tokens
        eng.split_scan, eng.split_min_rows, eng.piece_tokens = True, 16, 16                   # side-by-side pieces, as the bf16 mode runs them
        assert fc.rel_err(fc.stream_logits(eng, toks, [140, 33, 64, 63]), ref) < F32_TOL


@pytest.mark.parametrize("heads,dim,vdim", [(3, 10, 14), (2, 128, 256), (1, 256, 40), (4, 4, 330)])
def test_one_kernel_token_step_equals_the_separate_kernels(cuda_device, heads, dim, vdim):
    """The cell's token step in one kernel against gates, scan and output kernels: the same sums in the same order."""
    config = fc.model([C(heads=heads, dim=dim, vdim=vdim)], width=48)
    wt = fc.weights(config, 5)
    toks = fc.tokens_for(config, 40, seed=6)
    eng = fc.build_engine(config, wt, torch.float32, cuda_device)
    fused = fc.stream_logits(eng, toks, [3])
    eng.unfused_cell = True
    assert fc.rel_err(fused, fc.stream_logits(eng, toks, [3])) < 1e-6
    assert fc.rel_err(fused, fc.oracle_logits(config, wt, toks)) < F32_TOL


def test_choice_of_experts(cuda_device):
    """Choice scores that are never a close call and all negative (closed groups must count as minus infinity, not zero),
    corrections large enough to change the choice: a wrong group rule, a correction inside the weights, renormalised
    weights, a forgotten identity output or a forgotten shared gate shows at once."""
    spec = M(experts=13, top=4, ff=12, identity=5, groups=(6, 3), shared=16)
    config = fc.model([C(mlp=spec)], width=40)
    wt = fc.weights(config, 17)
    wt["l0.mlp.correction"] = fc.bf16_round(wt["l0.mlp.correction"] * 3.0 - 2.0)
    toks = fc.tokens_for(config, 120, seed=4)
    gaps = []
    ref = fc.oracle_logits(config, wt, toks, margins=gaps)
    clear = torch.tensor(gaps[0]) > 1e-5
    assert clear.float().mean() > 0.95
    score = torch.softmax(fo._mm(fo.offset_norm(wt["embed"][torch.tensor(toks)], wt["l0.norm1"], 1e-5), wt["l0.mlp.router"]), -1)
    chosen = [fo.choose(s, wt["l0.mlp.correction"], spec["router"]) for s in score]
    assert {e for c in chosen for e in c} > {13, 14} and len({tuple(c) for c in chosen}) > 10
    for path, value in ((["groups", "keep"], 6), (["groups", "keep"], 2), (["groups", "count"], 9), (["top"], 3)):
        wrong = fc.replaced(config, ["layers", 0, "mlp", "router", *path], value)
        assert fc.rel_err(fc.oracle_logits(wrong, wt, toks), ref) > 50 * F32_TOL
    flat = dict(wt)
    flat["l0.mlp.correction"] = torch.full((18,), -2.0, dtype=torch.float64)
    assert fc.rel_err(fc.oracle_logits(config, flat, toks), ref) > 50 * F32_TOL
    shut = dict(wt)
    shut["l0.mlp.shared.sg"] = torch.zeros(1, 40, dtype=torch.float64)
    assert fc.rel_err(fc.oracle_logits(config, shut, toks), ref) > 50 * F32_TOL
    eng = fc.build_engine(config, wt, torch.float32, cuda_device)
    for portions in ([100, 2], [120], [2, 3, 33]):
        assert fc.rel_err(fc.stream_logits(eng, toks, portions)[clear], ref[clear]) < F32_TOL


@pytest.mark.parametrize("n", [1, 5, 70])
def test_choice_kernel_against_the_oracle(cuda_device, n):
    """prl_moe_choose alone: choices, weights, and the grouping (no identity pair among the sorted rows)."""
    from pipelinerl_b200 import _lib
    lib = _lib.load()
    g = torch.Generator().manual_seed(n)
    for experts, identity, top, groups, keep in ((6, 2, 3, 4, 3), (40, 8, 6, 8, 2), (1, 0, 1, 1, 1), (3, 4, 7, 1, 1), (60, 4, 5, 64, 9), (900, 100, 12, 10, 4)):
        E = experts + identity
        z = (torch.randn(n, E + 3, generator=g) * 2.0).float()
        corr = torch.randn(E, generator=g) * 0.3 - 1.0
        i32 = dict(dtype=torch.int32, device=cuda_device)
        sel, perm = torch.full((top, n), -1, **i32), torch.full((top * n,), -1, **i32)
        wsel, meta = torch.zeros(top, n, device=cuda_device), torch.zeros(4, **i32)
        tiles = torch.zeros(3 * int(lib.prl_moe_max_tiles(top * n, experts)), **i32)
        zd, cd = z.to(cuda_device), corr.to(cuda_device)
        _lib.check(lib.prl_moe_choose(zd.data_ptr(), E + 3, cd.data_ptr(), n, experts, E, top, groups, keep, 1, 0, 0, 1.0, 64, sel.data_ptr(), wsel.data_ptr(),
                                      perm.data_ptr(), meta.data_ptr(), tiles.data_ptr(), _lib.stream_ptr()))
        torch.cuda.synchronize()
        score = torch.softmax(z[:, :E].double(), -1)
        sel, wsel, perm, tiles = sel.cpu(), wsel.cpu(), perm.cpu(), tiles.cpu().view(-1, 3)[:int(meta[0])]
        for t in range(n):
            gap = []
            want = fo.choose(score[t], corr.double(), dict(top=top, groups=dict(count=groups, keep=keep)), gap)
            if gap[0] > 1e-6:
                assert set(sel[:, t].tolist()) == set(want)
            assert torch.allclose(wsel[:, t].double(), score[t, sel[:, t].long()], rtol=2e-6)
        rows = []
        for e, at, m in tiles.tolist():
            assert 1 <= m <= 64
            rows += perm[at:at + m].tolist()
            assert all(int(sel.view(-1)[p]) == e for p in perm[at:at + m].tolist())
        assert sorted(rows) == [p for p in range(top * n) if int(sel.view(-1)[p]) < experts]


def test_first_tokens_and_one_token_sequences(cuda_device):
    wt = fc.weights(FULL, 12)
    eng = fc.build_engine(FULL, wt, torch.float32, cuda_device)
    for n in (1, 2, 3, 4, 5):
        toks = fc.tokens_for(FULL, n, seed=70 + n)
        ref = fc.oracle_logits(FULL, wt, toks)
        assert fc.rel_err(fc.stream_logits(eng, toks, [n]), ref) < F32_TOL
        assert fc.rel_err(fc.stream_logits(eng, toks, []), ref) < F32_TOL


# ---- the bf16 serving mode --------------------------------------------------------------------------------------------
BIG = fc.model([C(heads=4, dim=32, vdim=48, mlp=D(ff=256)), A(heads=8, kv_heads=2, dim=32, vdim=32, rot_dims=16, mlp=M(experts=3, top=4, ff=64, identity=1, groups=(2, 2), shared=128)),
                A(heads=4, kv_heads=2, dim=32, vdim=32, rot_dims=16, kv_from=1, mlp=D(ff=128)),
                C(heads=2, dim=64, vdim=64, mlp=M(experts=6, top=2, ff=96, identity=2, groups=(4, 2), shared=64))], vocab=200, width=128)


@pytest.mark.parametrize("mode", ["tensor_cores", "unfused_glu", "plain_gemm"])
def test_bf16_serving_mode(cuda_device, mode):
    """bf16 operands and cache with the tensor-core GEMMs (with and without the activation in the GEMM's epilogue, and with
    the CUDA-core GEMM) against the float64 oracle.  Only the last layer's router has a choice to make (the other one takes
    every output), so a token whose choice is closer than bf16 rounding can tell apart touches only its own logits; the
    oracle reports how close they are and those positions are left out."""
    wt = fc.weights(BIG, 13)
    toks = fc.tokens_for(BIG, 300, seed=8)
    gaps = []
    ref = fc.oracle_logits(BIG, wt, toks, margins=gaps)
    assert len(gaps) == 2 and min(gaps[0]) == float("inf")
    clear = torch.tensor(gaps[1]) > 0.02
    assert clear.float().mean().item() > 0.6
    eng = fc.build_engine(BIG, wt, torch.bfloat16, cuda_device, prefill_chunk=512)
    eng.force_plain_gemm, eng.unfused_glu = mode == "plain_gemm", mode == "unfused_glu"
    whole = fc.stream_logits(eng, toks, [300])
    assert fc.rel_err(whole[clear], ref[clear]) < BF16_TOL
    assert fc.rel_err(fc.stream_logits(eng, toks, [100, 2, 30])[clear], ref[clear]) < BF16_TOL
    assert fc.rel_err(fc.stream_logits(eng, toks, [130, 129])[clear], ref[clear]) < BF16_TOL
    eng.moe_tc_rows = 1 << 20                                # the routed products of the prompt on the few-row kernel
    assert fc.rel_err(fc.stream_logits(eng, toks, [300])[clear], ref[clear]) < BF16_TOL
    # the bf16 engine is about as close to the oracle as the oracle with only its matrix products' inputs rounded
    least = fc.rel_err(fc.oracle_logits(BIG, wt, toks, round_in=fc.bf16_round)[clear], ref[clear])
    assert fc.rel_err(whole[clear], ref[clear]) < 3 * least + 1e-3


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 128, 128), (8, 1, 128, 128), (4, 4, 64, 64), (6, 2, 48, 80), (5, 5, 40, 48)])
def test_attention_kernels_agree(cuda_device, heads, kv_heads, dim, vdim):
    """Head sizes that the tensor-core kernels are built for (128 with the paged decode kernel, others with the prompt
    kernel for any size) and one they are not, a cache that two layers read, portions and single tokens over five page
    borders: against the CUDA-core kernel on the same cache, and against the oracle."""
    config = fc.model([A(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot_dims=dim // 2, scale=2.0 * dim ** -0.5),
                       A(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot_dims=dim // 2, scale=dim ** -0.5, kv_from=0, mlp=D(ff=64))], width=64)
    wt = fc.weights(config, 9)
    toks = fc.tokens_for(config, 330, seed=3)
    ref = fc.oracle_logits(config, wt, toks)
    eng = fc.build_engine(config, wt, torch.bfloat16, cuda_device, prefill_chunk=512)
    assert eng.tc_attn[0] == (dim == 128) and eng.tc_attn[1] == (dim == 128)
    plans = ([330], [63, 17, 16, 130, 65, 20, 3, 2], [300])                 # the rest one by one
    fast = [fc.stream_logits(eng, toks, p) for p in plans]
    eng.force_plain_attn = True
    eng.lib.prl_attn_any_tensor_cores(0)
    try:
        plain = [fc.stream_logits(eng, toks, p) for p in plans]
    finally:
        eng.lib.prl_attn_any_tensor_cores(1)
    for f, p in zip(fast, plain):
        assert fc.rel_err(f, p) < 0.25 * BF16_TOL                            # two kernels, the same result
        assert fc.rel_err(f, ref) < BF16_TOL and fc.rel_err(p, ref) < BF16_TOL


@pytest.mark.parametrize("M_,N,K1,K2", [(1, 40, 64, 72), (33, 300, 200, 64), (128, 256, 128, 1000), (129, 130, 72, 64), (300, 520, 512, 136)])
def test_dual_product_gemm(cuda_device, M_, N, K1, K2):
    """C = A1 B1^T + A2 B2^T in one accumulation, token-step form (split K) and many-row form, against fp32 torch."""
    from pipelinerl_b200 import _lib
    lib = _lib.load()
    g = torch.Generator().manual_seed(1)
    t = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16).to(cuda_device)
    A1, B1, A2, B2 = t(M_, K1), t(N, K1), t(M_, K2), t(N, K2)
    ref = A1.double() @ B1.double().T + A2.double() @ B2.double().T
    st = _lib.stream_ptr()
    if M_ <= 128:
        for k in (1, int(lib.prl_gemm_dual_split_k(M_, N, K1, K2)), 3):
            out = torch.full((k, M_, N), float("nan"), device=cuda_device)
            _lib.check(lib.prl_gemm_bf16_dual(B1.data_ptr(), A1.data_ptr(), K1, B2.data_ptr(), A2.data_ptr(), K2, M_, N, k, out.data_ptr(), st))
            assert (out.sum(0).double() - ref).abs().max().item() < 1e-4
    else:
        for k in (1, int(lib.prl_gemm_tn_dual_split_k(M_, N, K1, K2, 4)), 3):
            out = torch.full((k, M_, N), float("nan"), device=cuda_device)
            _lib.check(lib.prl_gemm_tn_dual(A1.data_ptr(), B1.data_ptr(), K1, A2.data_ptr(), B2.data_ptr(), K2, M_, N, k, out.data_ptr(), st))
            assert (out.sum(0).double() - ref).abs().max().item() < 1e-4


@pytest.mark.parametrize("n,W,ff,experts,identity,top", [(300, 64, 64, 3, 1, 2), (700, 136, 200, 5, 3, 3), (129, 256, 520, 2, 0, 1), (1024, 64, 72, 40, 8, 6)])
def test_grouped_gemm_of_many_rows(cuda_device, n, W, ff, experts, identity, top):
    """The tcgen05 grouped GEMM over gathered rows (row tiles of 256, expert sizes that are no multiple of a tile, choices
    that belong to no expert) against fp32 torch, for both products."""
    from pipelinerl_b200 import _lib
    lib = _lib.load()
    g = torch.Generator().manual_seed(n)
    bf = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16).to(cuda_device)
    x, up, down = bf(n, W) * 4, bf(experts * ff, W), bf(experts * W, ff)
    E = experts + identity
    z = torch.randn(n, E, generator=g).to(cuda_device)
    i32 = dict(dtype=torch.int32, device=cuda_device)
    sel, perm, meta = torch.zeros(top, n, **i32), torch.zeros(top * n, **i32), torch.zeros(4, **i32)
    wsel, tiles = torch.zeros(top, n, device=cuda_device), torch.zeros(3 * int(lib.prl_moe_max_tiles(top * n, experts)), **i32)
    st = _lib.stream_ptr()
    table = (perm.data_ptr(), meta.data_ptr(), tiles.data_ptr())
    _lib.check(lib.prl_moe_choose(z.data_ptr(), E, None, n, experts, E, top, 1, 1, 1, 0, 0, 1.0, 256, sel.data_ptr(), wsel.data_ptr(), *table, st))
    xs, act = torch.zeros(top * n, W, dtype=torch.bfloat16, device=cuda_device), torch.zeros(top * n, ff, dtype=torch.bfloat16, device=cuda_device)
    out = torch.full((top * n, W), float("nan"), device=cuda_device)
    _lib.check(lib.prl_moe_gather(x.data_ptr(), *table[:2], n, top * n, W, xs.data_ptr(), st))
    _lib.check(lib.prl_moe_gemm_tc(xs.data_ptr(), top * n, up.data_ptr(), experts, ff, W, *table, wsel.data_ptr(), 1, act.data_ptr(), ff, st))
    _lib.check(lib.prl_moe_gemm_tc(act.data_ptr(), top * n, down.data_ptr(), experts, W, ff, *table, None, 0, out.data_ptr(), W, st))
    torch.cuda.synchronize()
    assert int(meta[1]) == int((sel < experts).sum())
    for k in range(top):
        for e in range(E):
            rows = (sel[k] == e).nonzero().view(-1)
            got = out[k * n + rows]
            if e >= experts:
                assert torch.isnan(got).all()                        # handed through elsewhere, not written here
                continue
            a = torch.relu(x[rows].float() @ up[e * ff:(e + 1) * ff].float().T) ** 2 * wsel[k, rows, None]
            want = a.to(torch.bfloat16).float() @ down[e * W:(e + 1) * W].float().T
            assert (got - want).abs().max().item() < 2e-2 * max(1.0, want.abs().max().item()) if len(rows) else True


def test_long_decoding(cuda_device):
    """A short prompt and 400 single tokens over six page borders, in fp32 against the oracle."""
    config = fc.model([C(mlp=M()), A(), C(), A(kv_from=1, mlp=D())])
    wt = fc.weights(config, 31)
    toks = fc.tokens_for(config, 420, seed=12)
    eng = fc.build_engine(config, wt, torch.float32, cuda_device)
    assert fc.rel_err(fc.stream_logits(eng, toks, [20]), fc.oracle_logits(config, wt, toks)) < F32_TOL


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_greedy_generation_through_the_scheduler(cuda_device, dtype):
    """add_request / run_prefill / CUDA-graph token steps / harvest, five prompts on two slots (slots and pages are
    reused, idle slots ride along in the step), greedy ids against the oracle wherever its top-2 margin is not a
    rounding matter (fp32); bf16: against the engine's own stream of the same tokens."""
    from pipelinerl_b200.engine import SamplingParams
    config = FULL if dtype == torch.float32 else fc.model([C(heads=4, dim=32, vdim=48, mlp=D(ff=256)),
                                                            A(heads=4, kv_heads=1, dim=128, vdim=128, rot_dims=64, mlp=D(ff=128)),
                                                            A(heads=2, kv_heads=1, dim=128, vdim=128, rot_dims=64, kv_from=1)], vocab=100, width=128)
    wt = fc.weights(config, 14)
    eng = fc.build_engine(config, wt, dtype, cuda_device, max_batch=2, max_seq_len=256, use_cuda_graph=True, prefill_chunk=64)
    prompts = [fc.tokens_for(config, n, seed=90 + n) for n in (1, 5, 70, 130, 64)]
    outs = eng.generate(prompts, SamplingParams(max_tokens=6, greedy=True, ignore_eos=True))
    assert len(eng.free_slots) == 2 and len(eng.free_pages) == eng.n_pages - 1
    clear, gap = (1e-3, 1e-3) if dtype == torch.float32 else (0.2, 0.1)
    for p, r in zip(prompts, outs):
        assert len(r.output_ids) == 6 and r.finish_reason == "length"
        lg = fc.oracle_logits(config, wt, p + r.output_ids)
        for j, (tok, lp) in enumerate(zip(r.output_ids, r.output_logprobs)):
            row = lg[len(p) - 1 + j]
            top = torch.topk(row, 2)
            if (top.values[0] - top.values[1]).item() > clear:
                assert tok == top.indices[0].item()
            assert abs(lp - torch.log_softmax(row, -1)[tok].item()) < gap


def test_trace_runner_command_line(cuda_device, tmp_path):
    """bin/trace_run on a checkpoint folder: registry, safetensors loader, streams, output files, in both dtypes."""
    config = fc.model([A(mlp=M(experts=4, top=6, ff=8, identity=2, groups=(3, 3))), C(mlp=D(ff=24)), A(kv_from=0)], vocab=64, width=40)
    wt = fc.weights(config, 15)
    fc.write_checkpoint(tmp_path, config, wt)
    a, b = fc.tokens_for(config, 90, seed=1), fc.tokens_for(config, 20, seed=2)
    steps = [
        dict(step=0, entries=[dict(id="a", tokens=a[:50], want=[0, 49])], end=[]),
        dict(step=1, entries=[dict(id="a", tokens=a[50:52], want=[]), dict(id="b", tokens=b[:19], want=[3])], end=[]),
        dict(step=2, entries=[dict(id="b", tokens=b[19:], want=[0]), dict(id="a", tokens=a[52:], want=[37])], end=["a", "b"]),
        dict(step=3, entries=[dict(id="c", tokens=b, want=[19])], end=["c"]),
    ]
    ra, rb = fc.oracle_logits(config, wt, a), fc.oracle_logits(config, wt, b)
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
            assert got.shape == ref.shape and fc.rel_err(got, ref) < tol
