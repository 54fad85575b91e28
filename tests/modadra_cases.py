"""Small Modadra configurations and helpers for the tests (random weights, sizes chosen to be awkward)."""
import copy

import torch

from oracle import modadra_oracle as mo
from tests.belelorn_cases import rel_err, stream_logits, tokens_for, write_checkpoint  # noqa: F401  (model-independent helpers)
from tests.futetar_cases import replaced  # noqa: F401
from tests.pametar_cases import bf16_round, stage_stream  # noqa: F401


def parallel(heads=6, kv_heads=3, dim=12, vdim=10, window=40, rot_dims=8, base=30.0, scale=None, r_heads=6, r_kv_heads=2, r_dim=10,
             r_vdim=14, conv=3, mlp=None):
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else 1.2 * dim ** -0.5)
    if rot_dims:
        left["rot"] = dict(base=base, dims=rot_dims)
    if window:
        left["mask"] = dict(size=window)
    right = dict(heads=r_heads, kv_heads=r_kv_heads, dim=r_dim, vdim=r_vdim, conv=conv)
    return dict(type="parallel", mixer=dict(left=left, right=right), mlp=mlp)


def moe(experts=10, top=3, ff=20, groups=(5, 3), scale=1.4):
    r = dict(experts=experts, top=top, scale=scale)
    if groups is not None:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", router=r, expert=dict(ff=ff))


def model(layers, vocab=96, width=72, eps=1e-5, mult=0.6, cap=12.0):
    return dict(architecture="Modadra", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, logit_softcap=cap,
                layers=copy.deepcopy(layers))


def weights(config, seed=0):
    return mo.random_weights(config, seed)


def build_engine(config, wt, dtype, device, **kw):
    from pipelinerl_b200.hybrid import HybridConfig, HybridEngine
    from pipelinerl_b200.model import ParamArena
    cfg = HybridConfig.from_modadra(config, {k: tuple(v.shape) for k, v in wt.items()})
    arena = ParamArena(cfg, device, dtype=dtype)
    arena.load_hf_state_dict(wt)
    args = dict(max_batch=4, max_seq_len=512, max_new_tokens=32, prefill_chunk=256, use_cuda_graph=False, device=device)
    args.update(kw)
    return HybridEngine(cfg, arena, **args)


def oracle_logits(config, wt, tokens, **kw):
    return mo.forward(config, wt, tokens, **kw)
