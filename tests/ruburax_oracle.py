"""Plain, slow Ruburax: one function per mechanism, whole sequences, no cache, no batching, float64.

The oracle of the tests of the attention / parallel / gated-recurrence model.  It shares no code with the package: weights come
as a dictionary ``name -> tensor`` under the checkpoint's names, the configuration as the parsed ``config.json``.
"""
import math

import torch

F = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


# ---- attention -------------------------------------------------------------------------------------------------------
def frequencies(base, dims, scaling=None):
    """One frequency per rotated pair; ``scaling``: long wavelengths stretched by ``factor``, short ones kept, a linear blend (in
    turns per original context) between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            turns = scaling["original"] * f / (2.0 * math.pi)          # original / wavelength
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate_halves(x, freqs, sign=1.0):
    """Rotary positions for ``x [T, heads, dim]``: channels i and i + n turn together, n = len(freqs) pairs; the rest pass."""
    T, n = x.shape[0], len(freqs)
    out = x.clone()
    for i, f in enumerate(freqs):
        a = sign * torch.arange(T, dtype=F) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + n]
        out[..., i] = u * c - v * s
        out[..., i + n] = v * c + u * s
    return out


def causal_attention(q, k, v, scale, sink=None):
    """``q [T, H, dk]``, ``k [T, G, dk]``, ``v [T, G, dv]`` (groups by integer division): softmax over all keys up to the query;
    ``sink [H]``: one extra term exp(sink) in the denominator."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    of = torch.arange(H) // (H // k.shape[1])
    kh, vh = k[:, of], v[:, of]
    for i in range(T):
        s = torch.einsum("hd,jhd->hj", q[i], kh[:i + 1]) * scale
        top = s.max(-1).values
        if sink is not None:
            top = torch.maximum(top, sink)
        e = torch.exp(s - top[:, None])
        den = e.sum(-1)
        if sink is not None:
            den = den + torch.exp(sink - top)
        out[i] = torch.einsum("hj,jhd->hd", e, vh[:i + 1]) / den[:, None]
    return out


def attention_keys(h, w, p, m, eps):
    """Normed, rotated keys and plain values of a layer that projects them."""
    T, G = h.shape[0], m["kv_heads"]

    def lin(n):
        y = h @ w[p + n].T
        return y + w[p + n + ".b"] if p + n + ".b" in w else y
    k = rms(lin("k").reshape(T, G, m["dim"]), eps) * w[p + "k.norm"]
    return rotate_halves(k, frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))), lin("v").reshape(T, G, m["vdim"])


def attention_mixer(h, w, p, m, eps, kv):
    """``kv``: keys and values of the layer that owns them."""
    q = h @ w[p + "q"].T
    if p + "q.b" in w:
        q = q + w[p + "q.b"]
    q = rms(q.reshape(h.shape[0], m["heads"], m["dim"]), eps) * w[p + "q.norm"]
    q = rotate_halves(q, frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling")))
    o = causal_attention(q, kv[0], kv[1], m["scale"], w.get(p + "sink"))
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


# ---- matrix memory ---------------------------------------------------------------------------------------------------
def memory_core(q, k, v, i, f):
    """``q, k [T, H, dk]``, ``v [T, H, dv]``, log gates ``i, f [T, H]``: state, normaliser and running maximum token by token; the
    maximum starts at 0."""
    T, H, dk = q.shape
    S, n, m = torch.zeros(H, dk, v.shape[-1], dtype=F), torch.zeros(H, dk, dtype=F), torch.zeros(H, dtype=F)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        mt = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - mt), torch.exp(i[t] - mt)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        m = mt
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / den[:, None]
    return out


def memory_gates(h, w, p, cap):
    """Log input and log forget gates from capped pre-activations."""
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    return i, -softplus(-cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))


def memory_mixer(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = (h @ w[p + "q"].T).reshape(T, H, m["dim"]) * m["dim"] ** -0.5
    k, v = (h @ w[p + "k"].T).reshape(T, H, m["dim"]), (h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o = memory_core(q, k, v, *memory_gates(h, w, p, m["gate_cap"]))
    return (rms(o, eps).reshape(T, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- gated linear recurrence -------------------------------------------------------------------------------------------
def causal_conv(x, taps, bias):
    """``x [T, C]``, ``taps [C, K]`` (last column: the current token), zeros before the start."""
    K = taps.shape[1]
    full = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=F), x])
    return sum(full[j:j + x.shape[0]] * taps[:, j] for j in range(K)) + bias


def recurrence_core(u, ra, rab, ri, rib, lam):
    """``u [T, C]``; ``ra, ri [B, n, n]`` act on the B equal parts of u, as ``[out, in]``."""
    T, C = u.shape
    parts = u.reshape(T, ra.shape[0], -1)
    r = sigmoid(torch.einsum("tbn,bmn->tbm", parts, ra) + rab).reshape(T, C)
    i = sigmoid(torch.einsum("tbn,bmn->tbm", parts, ri) + rib).reshape(T, C)
    log_a = -8.0 * r * softplus(lam)
    S, out = torch.zeros(C, dtype=F), torch.zeros(T, C, dtype=F)
    for t in range(T):
        a = torch.exp(log_a[t])
        S = a * S + torch.sqrt(1.0 - a * a) * i[t] * u[t]
        out[t] = S
    return out


def rglru_mixer(h, w, p, m, eps):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    s = recurrence_core(u, w[p + "ra"], w[p + "ra.b"], w[p + "ri"], w[p + "ri.b"], w[p + "lam"])
    return (s * y) @ w[p + "o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------------
def glu(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(scores, correction, top, groups):
    """Chosen experts of one token: best ``keep`` groups by their two largest corrected scores, then the best experts in them."""
    c = scores + correction
    if groups is not None:
        per = c.numel() // groups["count"]
        rank = [sum(sorted(c[g * per:(g + 1) * per].tolist(), reverse=True)[:2]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: -rank[g])[:groups["keep"]]
        open_ = [e for g in kept for e in range(g * per, (g + 1) * per)]
    else:
        open_ = range(c.numel())
    return sorted(open_, key=lambda e: -float(c[e]))[:top]


def margin(scores, correction, top, groups):
    """How far the choice of one token is from another one: the smaller of the two gaps, between groups and between experts."""
    c, gap = scores + correction, math.inf
    per = c.numel() // groups["count"] if groups is not None else c.numel()
    if groups is not None and groups["keep"] < groups["count"]:
        g = sorted((sum(sorted(c[i:i + per].tolist(), reverse=True)[:2]) for i in range(0, c.numel(), per)), reverse=True)
        gap = g[groups["keep"] - 1] - g[groups["keep"]]
    picked = route(scores, correction, top, groups)
    rest = set(route(scores, correction, c.numel(), groups)) - set(picked)
    if rest:
        gap = min(gap, min(float(c[e]) for e in picked) - max(float(c[e]) for e in rest))
    return gap


def moe(h, w, p, m, margins=None):
    r, out = m["router"], torch.zeros_like(h)
    s = sigmoid(h @ w[p + "router"].T)
    if margins is not None:
        margins.append(torch.tensor([margin(x, w[p + "correction"], r["top"], r.get("groups")) for x in s]))
    for t in range(h.shape[0]):
        for e in route(s[t], w[p + "correction"], r["top"], r.get("groups")):
            out[t] += s[t, e] * r["scale"] * glu(h[t], w, f"{p}e{e}.")
    if m.get("shared") is not None:
        out = out + glu(h, w, p + "shared.") * sigmoid(h @ w[p + "shared.sg"].T)
    return out


# ---- the layer's frame -------------------------------------------------------------------------------------------------
def token_input(x, w, p, tokens, i, dim, eps):
    e = w["side.embed"][torch.as_tensor(tokens)][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return rms(y, eps) * w[p + "side.norm"]


def forward(cfg, weights, tokens, layers_out=None, margins=None):
    """Logits ``[T, vocab]``; ``layers_out`` (a list) receives the residual stream after every layer, ``margins`` every expert
    layer's margins of choice."""
    w = {n: t.to(F) for n, t in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x, keys = w["embed"][torch.as_tensor(tokens)], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            keys[i] = keys[m["kv_from"]] if m.get("kv_from") is not None else attention_keys(x, w, p + "mix.", m, eps)
            y = attention_mixer(x, w, p + "mix.", m, eps, keys[i])
        elif layer["type"] == "parallel":
            left = attention_mixer(x, w, p + "mix.left.", m["left"], eps, attention_keys(x, w, p + "mix.left.", m["left"], eps))
            y = m["left_scale"] * left + m["right_scale"] * memory_mixer(x, w, p + "mix.right.", m["right"], eps)
        else:
            y = rglru_mixer(x, w, p + "mix.", m, eps)
        x = x + mult * rms(y, eps) * w[p + "norm1"]
        if layer["mlp"] is not None:
            y = glu(x, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else moe(x, w, p + "mlp.", layer["mlp"], margins)
            x = x + mult * rms(y, eps) * w[p + "norm2"]
        if cfg.get("token_side") is not None:
            x = x + mult * token_input(x, w, p, tokens, i, cfg["token_side"]["dim"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T * cfg["logit_scale"]


def shapes(cfg):
    W, s = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    side = cfg.get("token_side")
    if side is not None:
        s["side.embed"] = (cfg["vocab"], side["dim"] * len(cfg["layers"]))

    def glu_shapes(p, ff):
        return {p + "gate": (ff, W), p + "up": (ff, W), p + "down": (W, ff)}

    def attention_shapes(x, m, bias, sink):
        H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        r = {x + "q": (H * d, W), x + "q.norm": (d,), x + "o": (W, H * v)}
        if m.get("kv_from") is None:
            r |= {x + "k": (G * d, W), x + "k.norm": (d,), x + "v": (G * v, W)}
        if bias:
            r |= {n + ".b": r[n][:1] for n in (x + "q", x + "k", x + "v") if n in r}
        return r | ({x + "sink": (H,)} if sink else {})
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        s[p + "norm1"] = (W,)
        if layer["type"] == "attention":
            s |= attention_shapes(x, m, True, True)
        elif layer["type"] == "parallel":
            s |= attention_shapes(x + "left.", m["left"], False, False)
            r, x = m["right"], x + "right."
            H, d, v = r["heads"], r["dim"], r["vdim"]
            s |= {x + "q": (H * d, W), x + "k": (H * d, W), x + "v": (H * v, W), x + "g": (H * v, W), x + "o": (W, H * v),
                  x + "norm": (H * v,), x + "i": (H, W), x + "i.b": (H,), x + "f": (H, W), x + "f.b": (H,)}
        else:
            C, B = m["width"], m["blocks"]
            s |= {x + "y": (C, W), x + "y.b": (C,), x + "x": (C, W), x + "x.b": (C,), x + "conv": (C, m["conv"]), x + "conv.b": (C,),
                  x + "lam": (C,), x + "o": (W, C)}
            s |= {x + n: (B, C // B, C // B) for n in ("ra", "ri")} | {x + n + ".b": (B, C // B) for n in ("ra", "ri")}
        f, x = layer["mlp"], p + "mlp."
        if f is not None:
            s[p + "norm2"] = (W,)
            if f["kind"] == "dense":
                s |= glu_shapes(x, f["ff"])
            else:
                for e in range(f["router"]["experts"]):
                    s |= glu_shapes(f"{x}e{e}.", f["expert"]["ff"])
                s |= {x + "router": (f["router"]["experts"], W), x + "correction": (f["router"]["experts"],)}
                if f.get("shared") is not None:
                    s |= glu_shapes(x + "shared.", f["shared"]["ff"]) | {x + "shared.sg": (1, W)}
        if side is not None:
            s |= {p + "side.gate": (side["dim"], W), p + "side.proj": (W, side["dim"]), p + "side.norm": (W,)}
    return s


def random_weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        r, last = torch.randn(shape, generator=g, dtype=torch.float32), name.rsplit(".", 1)[-1]
        if last.startswith("norm"):
            r = 1.0 + 0.2 * r
        elif name.endswith("f.b"):
            r = 4.0 + r
        elif last == "b":
            r = r * 0.5
        elif last == "correction":
            r = r * 1.2 - 1.0             # most choice scores are negative, and few choices are close
        elif last == "sink":
            r = 1.0 + r
        elif last == "lam":
            r = r - 4.0
        elif last == "router":
            r = r * shape[-1] ** -0.5 * 0.7
        elif name in ("embed", "side.embed"):
            r = r
        else:
            r = r * shape[-1] ** -0.5 * 1.5
        out[name] = r
    return out
