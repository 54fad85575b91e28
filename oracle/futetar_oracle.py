"""Oracle for the "Futetar" decoders (pipelinerl_b200/hybrid.py, `HybridConfig.from_futetar`): a plain, slow,
whole-sequence implementation.

TEST INFRASTRUCTURE (see oracle/__init__.py).  Torch float64 on CPU, one function per mechanism, every recurrence an
explicit loop over time, no cache, no chunks, no batching, nothing shared with the product path.  The reference has no
model code of its own (it serves through vLLM, pipelinerl/launch.py:191-247), so these functions restate the design's
equations and are the yardstick for the CUDA kernels.

Notation: T tokens, W the model width, h [T, W] a layer's normed input, weights stored [out, in] and applied as h @ M.T.
`wt` maps a checkpoint tensor name to a float64 tensor, `p` is the prefix of a sublayer's tensors, `cfg` the dict of
config.json.  `round_in`, when given, is applied to both operands of every matrix product (tests use it to measure the
least error a bf16 product can have).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def _mm(a, w, round_in=None):
    if round_in is not None:
        a, w = round_in(a), round_in(w)
    return a @ w.T


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """Root-mean-square norm whose stored weight is the gain minus one."""
    return unit_rms(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- mixers ---------------------------------------------------------------------------------------------------------
def matrix_lstm(h, wt, p, m, eps, round_in=None):
    """One d x dv matrix per head.  With log gates i_t and f_t and the stabiliser m_t = max(f_t + m_(t-1), i_t), m_0 = 0:
    S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k v^T, n_t the same with k alone."""
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (_mm(h, wt[p + "q"], round_in) / math.sqrt(d)).view(T, H, d)
    k = _mm(h, wt[p + "k"], round_in).view(T, H, d)
    v = _mm(h, wt[p + "v"], round_in).view(T, H, dv)
    soft = lambda z: cap * torch.tanh(z / cap)
    log_in = soft(_mm(h, wt[p + "i"], round_in) + wt[p + "i.b"])
    log_keep = -torch.nn.functional.softplus(-soft(_mm(h, wt[p + "f"], round_in) + wt[p + "f.b"]))
    o = torch.zeros(T, H, dv, dtype=F64)
    S, n, stab = torch.zeros(H, d, dv, dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)
    for t in range(T):
        new = torch.maximum(log_keep[t] + stab, log_in[t])
        keep, take = torch.exp(log_keep[t] + stab - new), torch.exp(log_in[t] - new)
        stab = new
        for a in range(H):
            S[a] = keep[a] * S[a] + take[a] * torch.outer(k[t, a], v[t, a])
            n[a] = keep[a] * n[a] + take[a] * k[t, a]
            o[t, a] = (q[t, a] @ S[a]) / (max(abs(float(n[a] @ q[t, a])), math.exp(-float(new[a]))) + 1e-6)
    y = unit_rms(o, eps).reshape(T, H * dv) * wt[p + "norm"] * torch.sigmoid(_mm(h, wt[p + "g"], round_in))
    return _mm(y, wt[p + "o"], round_in)


def rotary_frequencies(rot):
    """base^(-2i/dims); with a scaling block, wavelengths above original/low are stretched by `factor`, those below
    original/high kept, and in between the two are mixed linearly in the number of turns over `original` positions."""
    dims, out = rot["dims"], []
    sc = rot.get("scaling")
    for i in range(dims // 2):
        f = rot["base"] ** (-2.0 * i / dims)
        if sc:
            turns = sc["original"] * f / (2.0 * math.pi)        # original / wavelength
            if turns < sc["low"]:
                f = f / sc["factor"]
            elif turns <= sc["high"]:
                s = (turns - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, rot):
    """x [T, heads, dim]: channel i < dims/2 turns with channel i + dims/2 by position * frequency."""
    if not rot:
        return x
    half = rot["dims"] // 2
    ang = torch.arange(x.shape[0], dtype=F64)[:, None, None] * torch.tensor(rotary_frequencies(rot), dtype=F64)
    y = x.clone()
    u, v = x[..., :half], x[..., half:2 * half]
    y[..., :half] = u * torch.cos(ang) - v * torch.sin(ang)
    y[..., half:2 * half] = v * torch.cos(ang) + u * torch.sin(ang)
    return y


def attention_keys(h, wt, p, a, eps, round_in=None):
    """(keys [T, G, dim] normed and turned, values [T, G, vdim]) of a layer that projects its own."""
    T, G = h.shape[0], a["kv_heads"]
    k = _mm(h, wt[p + "k"], round_in).view(T, G, a["dim"])
    return rotate(unit_rms(k, eps) * wt[p + "k.norm"], a.get("rot")), _mm(h, wt[p + "v"], round_in).view(T, G, a["vdim"])


def attention(h, keys, values, wt, p, a, eps, round_in=None):
    T, H, G = h.shape[0], a["heads"], a["kv_heads"]
    q = rotate(unit_rms(_mm(h, wt[p + "q"], round_in).view(T, H, a["dim"]), eps) * wt[p + "q.norm"], a.get("rot"))
    out = torch.zeros(T, H, values.shape[2], dtype=F64)
    for t in range(T):
        for head in range(H):
            g = head // (H // G)
            w = torch.softmax((keys[:t + 1, g] @ q[t, head]) * a["scale"], dim=0)
            out[t, head] = w @ values[:t + 1, g]
    return _mm(out.reshape(T, -1), wt[p + "o"], round_in)


# ---- feed-forward ---------------------------------------------------------------------------------------------------
def gated_ff(h, wt, p, round_in=None):
    return _mm(gelu_tanh(_mm(h, wt[p + "gate"], round_in)) * _mm(h, wt[p + "up"], round_in), wt[p + "down"], round_in)


def squared_relu_ff(h, wt, p, round_in=None):
    return _mm(torch.relu(_mm(h, wt[p + "up"], round_in)) ** 2, wt[p + "down"], round_in)


def choose(score, correction, r, margins=None):
    """Chosen outputs of one token: the `top` best by score + correction among the outputs whose group is one of the
    `keep` groups with the best maximum.  `margins` receives how close the closest of the two choices was."""
    n = score.numel()
    c = score + correction
    groups = r.get("groups") or {"count": 1, "keep": 1}
    size = n // groups["count"]
    best = [float(c[g * size:(g + 1) * size].max()) for g in range(groups["count"])]
    order = sorted(range(groups["count"]), key=lambda g: (-best[g], g))
    open_groups = set(order[:groups["keep"]])
    ranked = sorted((e for e in range(n) if e // size in open_groups), key=lambda e: (-float(c[e]), e))
    if margins is not None:
        gap = math.inf
        if groups["keep"] < groups["count"]:
            gap = best[order[groups["keep"] - 1]] - best[order[groups["keep"]]]
        if r["top"] < len(ranked):
            gap = min(gap, float(c[ranked[r["top"] - 1]] - c[ranked[r["top"]]]))
        margins.append(gap)
    return ranked[:r["top"]]


def routed_ff(h, wt, p, f, round_in=None, margins=None):
    """Weighted sum of the chosen outputs, a weight being the output's share of the softmax over all of them (as it is,
    without the correction); outputs past the experts hand the input through.  A shared expert joins every token's sum
    behind a sigmoid of one logit."""
    r = f["router"]
    score = torch.softmax(_mm(h, wt[p + "router"], round_in), dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(score[t], wt[p + "correction"], r, margins):
            y = squared_relu_ff(h[t:t + 1], wt, f"{p}e{e}.", round_in)[0] if e < r["experts"] else h[t]
            out[t] += score[t, e] * y
    if f.get("shared") is not None:
        out = out + torch.sigmoid(_mm(h, wt[p + "shared.sg"], round_in)) * squared_relu_ff(h, wt, p + "shared.", round_in)
    return out


# ---- the model --------------------------------------------------------------------------------------------------------
def forward(cfg, wt, tokens, residuals=None, round_in=None, margins=None):
    """Logits [T, vocab] of a whole sequence; `residuals` collects the stream after every layer, `margins` the closeness
    of the expert choices of every routed layer (one list of T gaps per layer)."""
    eps = cfg["norm"]["eps"]
    x = wt["embed"][torch.tensor(tokens)]
    cache = {}
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        h = offset_norm(x, wt[p + "norm1"], eps)
        if L["type"] == "mlstm":
            y = matrix_lstm(h, wt, p + "mix.", m, eps, round_in)
        elif L["type"] == "attention":
            if m.get("kv_from") is None:
                cache[i] = attention_keys(h, wt, p + "mix.", m, eps, round_in)
            y = attention(h, *cache[m["kv_from"] if m.get("kv_from") is not None else i], wt, p + "mix.", m, eps, round_in)
        else:
            raise ValueError(L["type"])
        if f is not None:
            if f["kind"] == "dense":
                y = y + gated_ff(h, wt, p + "mlp.", round_in)
            else:
                gaps = [] if margins is not None else None
                y = y + routed_ff(h, wt, p + "mlp.", f, round_in, gaps)
                if margins is not None:
                    margins.append(gaps)
        x = x + y
        if residuals is not None:
            residuals.append(x.clone())
    return _mm(offset_norm(x, wt["final.norm"], eps), wt["head"], round_in)


def tensor_shapes(cfg):
    """Checkpoint tensor names and shapes of a config."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        out[p + "norm1"] = (W,)
        if L["type"] == "mlstm":
            nq, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({p + "mix.q": (nq, W), p + "mix.k": (nq, W), p + "mix.v": (nv, W), p + "mix.g": (nv, W),
                        p + "mix.o": (W, nv), p + "mix.norm": (nv,), p + "mix.i": (m["heads"], W),
                        p + "mix.i.b": (m["heads"],), p + "mix.f": (m["heads"], W), p + "mix.f.b": (m["heads"],)})
        else:
            nq = m["heads"] * m["dim"]
            out.update({p + "mix.q": (nq, W), p + "mix.q.norm": (m["dim"],), p + "mix.o": (W, m["heads"] * m["vdim"])})
            if m.get("kv_from") is None:
                out.update({p + "mix.k": (m["kv_heads"] * m["dim"], W), p + "mix.k.norm": (m["dim"],),
                            p + "mix.v": (m["kv_heads"] * m["vdim"], W)})
        if f is None:
            continue
        if f["kind"] == "dense":
            out.update({p + "mlp.gate": (f["ff"], W), p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
        else:
            r, F = f["router"], f["expert"]["ff"]
            for e in range(r["experts"]):
                out.update({f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
            n = r["experts"] + r.get("identity", 0)
            out.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
            if f.get("shared") is not None:
                S = f["shared"]["ff"]
                out.update({p + "mlp.shared.up": (S, W), p + "mlp.shared.down": (W, S), p + "mlp.shared.sg": (1, W)})
    return out


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random tensors, rounded to `dtype` so that the engine and the oracle see the same numbers.  Matrices have unit
    row gain (std 1/sqrt(fan_in)), gains are spread around their neutral value, gate biases favour remembering."""
    g = torch.Generator().manual_seed(seed)
    wt = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        noise = torch.randn(shape, generator=g)
        if name == "embed":
            t = noise
        elif leaf == "norm1" or name == "final.norm":
            t = noise * 0.2                                              # offsets from one
        elif leaf == "norm":
            t = 1.0 + noise * 0.2
        elif name.endswith("f.b"):
            t = 2.0 + noise
        elif leaf == "b":
            t = noise * 0.5
        elif leaf == "router":
            t = noise * 3.0 / math.sqrt(shape[-1])                       # well separated scores
        elif leaf == "correction":
            t = noise * 0.1
        else:
            t = noise / math.sqrt(shape[-1])
        wt[name] = t.to(dtype).to(F64)
    return wt
