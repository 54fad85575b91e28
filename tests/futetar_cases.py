"""Small Futetar configurations and helpers for the tests (random weights, sizes chosen to be awkward)."""
import copy

import torch

from oracle import futetar_oracle as fo
from tests.belelorn_cases import rel_err, stream_logits, tokens_for, write_checkpoint  # noqa: F401  (model-independent helpers)
from tests.pametar_cases import bf16_round, stage_stream  # noqa: F401


def cell(heads=3, dim=10, vdim=14, gate_cap=9.0, mlp=None):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap), mlp=mlp)


def attention(heads=6, kv_heads=3, dim=12, vdim=10, rot_dims=8, base=30.0, scaling=(3.0, 0.5, 2.5, 40), scale=None, kv_from=None,
              mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else dim ** -0.5)
    if rot_dims:
        m["rot"] = dict(base=base, dims=rot_dims)
        if scaling is not None:
            m["rot"]["scaling"] = dict(factor=scaling[0], low=scaling[1], high=scaling[2], original=scaling[3])
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=mlp)


def dense(ff=40):
    return dict(kind="dense", ff=ff)


def moe(experts=6, top=3, ff=20, identity=2, groups=(4, 3), shared=28):
    r = dict(experts=experts, top=top, identity=identity)
    if groups is not None:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    out = dict(kind="moe", router=r, expert=dict(ff=ff))
    if shared:
        out["shared"] = dict(ff=shared)
    return out


def model(layers, vocab=96, width=72, eps=1e-5):
    return dict(architecture="Futetar", vocab=vocab, width=width, norm=dict(eps=eps), layers=copy.deepcopy(layers))


def weights(config, seed=0):
    return fo.random_weights(config, seed)


def build_engine(config, wt, dtype, device, **kw):
    from pipelinerl_b200.hybrid import HybridConfig, HybridEngine
    from pipelinerl_b200.model import ParamArena
    cfg = HybridConfig.from_futetar(config, {k: tuple(v.shape) for k, v in wt.items()})
    arena = ParamArena(cfg, device, dtype=dtype)
    arena.load_hf_state_dict(wt)
    args = dict(max_batch=4, max_seq_len=512, max_new_tokens=32, prefill_chunk=256, use_cuda_graph=False, device=device)
    args.update(kw)
    return HybridEngine(cfg, arena, **args)


def oracle_logits(config, wt, tokens, **kw):
    return fo.forward(config, wt, tokens, **kw)


def replaced(config, path, value):
    """A copy of the config with one nested key replaced (None: taken out)."""
    out = copy.deepcopy(config)
    node = out
    for k in path[:-1]:
        node = node[k]
    if value is None:
        node.pop(path[-1])
    else:
        node[path[-1]] = value
    return out
