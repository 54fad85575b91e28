"""Float64 oracle of the "Modadra" decoder: one function per mechanism, whole sequences, no cache, no batching.

Every layer is pre-normed with a scaled residual: x <- x + m mixer(rms(x) w1), x <- x + m ff(rms(x) w2), m one constant of
the model.  The mixer is two mixers side by side on the same input h, each RMS-normed over the width with a gain of its
own, and averaged:

  left    softmax attention (grouped heads, value size of its own, rotate-half rotary on the leading channels, sliding
          window); the softmax denominator has one more term exp(0) = 1; head j's output times sigmoid(w_j . h)
  right   gated delta rule: short causal convolutions + SiLU on q, k, v, unit q and k, S <- g S, u = beta (v - S^T k),
          S <- S + k u^T, o = S^T q, per-head RMS norm with one gain of head size times a SiLU gate

Feed-forward: routed experts W_down gelu(W_up h) (gelu with the error function).  Scores are sigmoids of the router
logits; a correction joins them for the choice only; the outputs form equal groups of neighbours ranked by the sum of
their two best choice scores, and only the best groups are open; the chosen experts' scores are divided by their sum
and multiplied by a constant.  Logits are capped: c tanh(logits / c).

`forward(cfg, weights, tokens)` takes the parsed config.json (a dict), a {name: tensor} dict with the checkpoint's tensor
names and a list of token ids.  `round_in` is applied to the inputs of every matrix product (a bf16 rounding gives the
least error a bf16 engine can have); everything else stays float64.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ---- norms and activations ----------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def unit_length(x, eps=1e-6):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_erf(x):
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


# ---- left: windowed softmax attention with a constant sink --------------------------------------------------------------
def rotate(x, positions, dims, base):
    """x [T, heads, d]: of the first `dims` channels i pairs with i + dims / 2 and turns by position * base^(-2i/dims)."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = positions.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def window_mask(T, window):
    """[T, T] bool: query i sees key j when 0 <= i - j < window (window 0: every earlier key)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & ((back < window) if window else torch.ones_like(back, dtype=torch.bool))


def sink_attention(q, k, v, scale, window, sink=1.0):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]: weights exp(s_j) / (sink + sum_j exp(s_j)) over the window."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    see = window_mask(T, window)
    heads = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T * scale).masked_fill(~see, -math.inf)
        m = s.amax(-1, keepdim=True).clamp_min(0.0)
        e = torch.exp(s - m)
        heads.append(e @ v[:, h // per] / (sink * torch.exp(-m) + e.sum(-1, keepdim=True)))
    return torch.stack(heads, 1)


def left_mixer(lin, p, m, h, positions):
    T = h.shape[0]
    H, G, d, e = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])
    q, k, v = lin(h, p + "q").view(T, H, d), lin(h, p + "k").view(T, G, d), lin(h, p + "v").view(T, G, e)
    rot = m.get("rot") or {}
    if rot.get("dims", 0):
        q, k = (rotate(t, positions, rot["dims"], rot["base"]) for t in (q, k))
    o = sink_attention(q, k, v, m["scale"], (m.get("mask") or {}).get("size", 0))
    o = o * torch.sigmoid(lin(h, p + "g"))[:, :, None]
    return lin(o.reshape(T, H * e), p + "o")


# ---- right: gated delta rule ------------------------------------------------------------------------------------------
def causal_conv(x, taps):
    """x [T, C], taps [C, n]: sum_j taps[:, n - 1 - j] x_(t - j), zeros before the start, then SiLU."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=F64), x])
    return silu(sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(n)))


def gated_delta(q, k, v, beta, g):
    """q, k [T, K, d], v [T, H, e], beta, g [T, H] -> [T, H, e]; value head h reads q / k head h // (H / K).  The read-out
    of a token sees its own write."""
    T, H, e = v.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, e, dtype=F64)
    for h in range(H):
        S = torch.zeros(k.shape[2], e, dtype=F64)
        for t in range(T):
            kt = k[t, h // per]
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ kt)
            S = S + torch.outer(kt, u)
            out[t, h] = S.T @ q[t, h // per]
    return out


def decay(a, A_log, dt_bias):
    """exp(-exp(A_log) softplus(a + dt_bias))."""
    return torch.exp(-torch.exp(A_log) * torch.nn.functional.softplus(a + dt_bias))


def right_mixer(lin, w, p, m, h, eps):
    T = h.shape[0]
    H, K, d, e = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    q, k, v = (causal_conv(lin(h, p + n), w[p + n + ".conv"]) for n in "qkv")
    q, k = unit_length(q.view(T, K, d)) / math.sqrt(d), unit_length(k.view(T, K, d))
    o = gated_delta(q, k, v.view(T, H, e), torch.sigmoid(lin(h, p + "b")), decay(lin(h, p + "a"), w[p + "A_log"], w[p + "dt_bias"]))
    o = rms_unit(o, eps) * w[p + "norm"] * silu(lin(h, p + "g").view(T, H, e))
    return lin(o.reshape(T, H * e), p + "o")


def parallel_mixer(lin, w, p, m, h, positions, eps):
    a = rms_unit(left_mixer(lin, p + "left.", m["left"], h, positions), eps) * w[p + "left.out"]
    b = rms_unit(right_mixer(lin, w, p + "right.", m["right"], h, eps), eps) * w[p + "right.out"]
    return 0.5 * (a + b)


# ---- routed feed-forward --------------------------------------------------------------------------------------------------
def choose(scores, correction, r, margins=None):
    """Chosen experts of one token, best first (ties: the lower index).  `margins` receives how close the closer of the
    two choices (groups, experts) was."""
    c = scores + correction
    n, top = scores.numel(), r["top"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    size = n // groups["count"]
    rank = [float(torch.sort(c[g * size:(g + 1) * size], descending=True).values[:2].sum()) for g in range(groups["count"])]
    order = sorted(range(groups["count"]), key=lambda g: (-rank[g], g))
    kept = set(order[:groups["keep"]])
    ranked = sorted((e for e in range(n) if e // size in kept), key=lambda e: (-float(c[e]), e))
    if margins is not None:
        gap = math.inf
        if groups["keep"] < groups["count"]:
            gap = rank[order[groups["keep"] - 1]] - rank[order[groups["keep"]]]
        if top < len(ranked):
            gap = min(gap, float(c[ranked[top - 1]] - c[ranked[top]]))
        margins.append(gap)
    return ranked[:top]


def routed(lin, w, p, f, h, margins=None):
    r = f["router"]
    scores = torch.sigmoid(lin(h, p + "router"))
    corr = w.get(p + "correction", torch.zeros(r["experts"], dtype=F64))
    rows = {}                                   # expert -> [(token, weight)]
    for t in range(h.shape[0]):
        picked = choose(scores[t], corr, r, margins)
        total = sum(float(scores[t, e]) for e in picked) + 1e-20
        for e in picked:
            rows.setdefault(e, []).append((t, float(scores[t, e]) / total * r.get("scale", 1.0)))
    y = torch.zeros_like(h)
    for e, pairs in rows.items():
        at = torch.tensor([t for t, _ in pairs])
        wt = torch.tensor([x for _, x in pairs], dtype=F64)
        y.index_add_(0, at, wt[:, None] * lin(gelu_erf(lin(h[at], f"{p}e{e}.up")), f"{p}e{e}.down"))
    return y


# ---- the model ------------------------------------------------------------------------------------------------------------
def forward(cfg, weights, tokens, residuals=None, round_in=None, margins=None):
    """Logits [T, vocab]; `residuals` receives the residual stream after every layer, `margins` one list per routed layer
    with a gap per token (see choose)."""
    w = {k: v.to(F64) for k, v in weights.items()}
    rnd = round_in if round_in is not None else (lambda x: x)
    lin = lambda x, name: rnd(x) @ w[name].T
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    positions = torch.arange(len(tokens))
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        if L["type"] != "parallel":
            raise ValueError(f"layer {i}: unknown mixer {L['type']!r}")
        x = x + m * parallel_mixer(lin, w, p + "mix.", L["mixer"], rms_unit(x, eps) * w[p + "norm1"], positions, eps)
        if L.get("mlp") is not None:
            gaps = None if margins is None else []
            x = x + m * routed(lin, w, p + "mlp.", L["mlp"], rms_unit(x, eps) * w[p + "norm2"], gaps)
            if margins is not None:
                margins.append(gaps)
        if residuals is not None:
            residuals.append(x.clone())
    z = lin(rms_unit(x, eps) * w["final.norm"], "head")
    cap = cfg.get("logit_softcap") or 0.0
    return soft_cap(z, cap) if cap else z


# ---- random checkpoints for the tests ---------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """{tensor name: shape} of a checkpoint of this config."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, L in enumerate(cfg["layers"]):
        a, r, p = L["mixer"]["left"], L["mixer"]["right"], f"l{i}.mix."
        H, G, d, e = a["heads"], a.get("kv_heads", a["heads"]), a["dim"], a.get("vdim", a["dim"])
        out.update({p + "left.q": (H * d, W), p + "left.k": (G * d, W), p + "left.v": (G * e, W), p + "left.g": (H, W),
                    p + "left.o": (W, H * e), p + "left.out": (W,), p + "right.out": (W,)})
        H, K, d, e, taps = r["heads"], r.get("kv_heads", r["heads"]), r["dim"], r["vdim"], r["conv"]
        for name, n in (("q", K * d), ("k", K * d), ("v", H * e)):
            out[p + "right." + name], out[f"{p}right.{name}.conv"] = (n, W), (n, taps)
        out.update({p + "right.b": (H, W), p + "right.a": (H, W), p + "right.A_log": (H,), p + "right.dt_bias": (H,),
                    p + "right.norm": (e,), p + "right.g": (H * e, W), p + "right.o": (W, H * e), f"l{i}.norm1": (W,)})
        f = L.get("mlp")
        if f is not None:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            out.update({f"l{i}.norm2": (W,), f"l{i}.mlp.router": (E, W), f"l{i}.mlp.correction": (E,)})
            for k in range(E):
                out.update({f"l{i}.mlp.e{k}.up": (ff, W), f"l{i}.mlp.e{k}.down": (W, ff)})
    return out


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random tensors, rounded to `dtype` so that the engine and the oracle see the same numbers.  Matrices have unit
    row gain (std 1/sqrt(fan_in)), gains are spread around one, decays favour remembering, router rows are scaled so that
    a choice is rarely a close call."""
    g = torch.Generator().manual_seed(seed)
    wt = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        noise = torch.randn(shape, generator=g)
        if name == "embed":
            t = noise
        elif leaf in ("norm1", "norm2", "norm", "out"):
            t = 1.0 + noise * 0.2
        elif leaf == "A_log":
            t = torch.log(0.05 + 0.5 * torch.rand(shape, generator=g))
        elif leaf == "dt_bias":
            t = noise
        elif leaf == "conv":
            t = noise * 0.6
        elif leaf == "correction":
            t = noise * 0.3
        elif leaf == "router":
            t = noise * 2.0 / math.sqrt(shape[-1])
        elif name == "head":
            t = noise * 4.0 / math.sqrt(shape[-1])
        else:
            t = noise / math.sqrt(shape[-1])
        wt[name] = t.to(dtype).to(F64)
    return wt
