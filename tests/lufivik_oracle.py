"""Plain, slow Lufivik: one function per mechanism, whole sequences, no cache, no batching, float64.

The oracle of the tests of the windowed latent-attention model with experts.  It shares no code with the package: weights come as a
dictionary ``name -> tensor`` under the checkpoint's names, the configuration as the parsed ``config.json``.
"""
import torch

F = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    """Mean off, divided by the root of the mean squared deviation, weight and bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


# ---- embedding -------------------------------------------------------------------------------------------------------
def bigram_rows(seq, mul_prev, mul_cur, buckets):
    """Row of the bigram table for every token; the first token of a sequence has the row past the buckets."""
    return [buckets] + [(a * mul_prev + b * mul_cur) % buckets for a, b in zip(seq, seq[1:])]


def embedding(seq, cfg, w, eps):
    g = cfg["embedding"]["bigram"]
    x = w["embed"][list(seq)] + w["bigram"][bigram_rows(list(seq), g["mul_prev"], g["mul_cur"], g["buckets"])]
    return layer_norm(x, w["embed.norm"], w["embed.norm.b"], eps)


# ---- what surrounds a sublayer -----------------------------------------------------------------------------------------
def causal_conv(h, taps):
    """``h [T, C]``, ``taps [C, K]`` (last column: the current token), zeros before the start."""
    K = taps.shape[1]
    full = torch.cat([torch.zeros(K - 1, h.shape[1], dtype=F), h])
    return sum(full[j:j + h.shape[0]] * taps[:, j] for j in range(K))


def residual_gate(h, w, b):
    return sigmoid(h @ w.T + b)


# ---- latent attention --------------------------------------------------------------------------------------------------
def rotate_halves(x, base, sign=1.0):
    """Rotary positions for all channels of ``x [T, heads, dim]``: channels i and i + dim / 2 turn together."""
    T, half = x.shape[0], x.shape[-1] // 2
    out = x.clone()
    for i in range(half):
        a = sign * torch.arange(T, dtype=F) * base ** (-2.0 * i / (2 * half))
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def latent_keys(c, kr, uk, heads):
    """``c [T, rank]`` normed, ``kr [T, rot]`` turned: ``[T, heads, dim + rot]``."""
    k = (c @ uk.T).reshape(c.shape[0], heads, -1)
    return torch.cat([k, kr[:, None].expand(-1, heads, -1)], -1)


def window_attention(q, k, v, scale, window):
    """``q, k [T, H, dk]``, ``v [T, H, dv]``: softmax over the last ``window`` keys up to the query."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for i in range(T):
        a = max(0, i - window + 1)
        s = torch.einsum("hd,jhd->hj", q[i], k[a:i + 1]) * scale
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhd->hd", e, v[a:i + 1]) / e.sum(-1)[:, None]
    return out


def latent_mixer(h, w, p, m, eps):
    T, H, rot = h.shape[0], m["heads"], m["rot_dim"]
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(T, H, m["dim"] + rot)
    q = torch.cat([q[..., :m["dim"]], rotate_halves(q[..., m["dim"]:], m["rot"]["base"])], -1)
    y = h @ w[p + "dkv"].T
    c = rms(y[:, :m["kv_rank"]], eps) * w[p + "dkv.norm"]
    kr = rotate_halves(y[:, None, m["kv_rank"]:], m["rot"]["base"])[:, 0]
    o = window_attention(q, latent_keys(c, kr, w[p + "uk"], H), (c @ w[p + "uv"].T).reshape(T, H, m["vdim"]), m["scale"], m["mask"]["size"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T


# ---- experts -----------------------------------------------------------------------------------------------------------
def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def choose(z, top):
    """Softmax over all experts: indices of the largest scores and the scores themselves, with the gap to the next logit."""
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    order = z.sort(dim=-1, descending=True, stable=True)
    gap = order.values[:, top - 1] - order.values[:, top] if top < z.shape[1] else torch.full((z.shape[0],), float("inf"), dtype=F)
    return order.indices[:, :top], s.gather(1, order.indices[:, :top]), gap


def experts(h, w, p, f, margins=None):
    ids, weights, gap = choose(h @ w[p + "router"].T, f["router"]["top"])
    if margins is not None:
        margins.append(gap)
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, c = (ids == e).nonzero(as_tuple=True)
        n = f"{p}e{e}."
        y = clamped_glu(h[t] @ w[n + "gate"].T, h[t] @ w[n + "up"].T, f["expert"]["limit"]) @ w[n + "down"].T
        out[t] += weights[t, c][:, None] * y
    return out


# ---- the model ---------------------------------------------------------------------------------------------------------
def order_of_runs(cfg):
    """Which layer's weights every run uses."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def run_layer(x, w, p, l, eps, margins=None):
    h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
    y = latent_mixer(h + causal_conv(h, w[p + "canon1"]), w, p + "mix.", l["mixer"], eps)
    y = y * residual_gate(h, w[p + "rg1"], w[p + "rg1.b"])
    x = x + w[p + "ls1"] * layer_norm(y, w[p + "norm1b"], w[p + "norm1b.b"], eps)
    if l.get("mlp") is None:
        return x
    h = layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps)
    y = experts(h, w, p + "mlp.", l["mlp"], margins) * residual_gate(h, w[p + "rg2"], w[p + "rg2.b"])
    return x + w[p + "ls2"] * layer_norm(y, w[p + "norm2b"], w[p + "norm2b.b"], eps)


def forward(cfg, weights, seq, seen=None, margins=None):
    """Token ids -> logits ``[T, vocab]``.  ``seen`` collects the residual after every layer run, ``margins`` how far the last chosen
    expert's logit is above the next, per run and token."""
    w = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(seq, cfg, w, eps)
    for i in order_of_runs(cfg):
        x = run_layer(x, w, f"l{i}.", cfg["layers"][i], eps, margins)
        if seen is not None:
            seen.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


def shapes(cfg):
    """Checkpoint name -> shape."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, W), "head": (V, W)}

    def norm(n):
        s[n], s[n + ".b"] = (W,), (W,)
    norm("embed.norm")
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l.get("mlp")
        H, q = m["heads"], p + "mix."
        s |= {p + "canon1": (W, cfg["canon"]["taps"]), q + "dq": (m["q_rank"], W), q + "dq.norm": (m["q_rank"],),
              q + "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]), q + "dkv": (m["kv_rank"] + m["rot_dim"], W), q + "dkv.norm": (m["kv_rank"],),
              q + "uk": (H * m["dim"], m["kv_rank"]), q + "uv": (H * m["vdim"], m["kv_rank"]), q + "g": (H, W), q + "o": (W, H * m["vdim"])}
        for k in "12" if f is not None else "1":
            norm(f"{p}norm{k}")
            norm(f"{p}norm{k}b")
            s |= {f"{p}ls{k}": (W,), f"{p}rg{k}": (W, W), f"{p}rg{k}.b": (W,)}
        if f is not None:
            s[p + "mlp.router"] = (f["router"]["experts"], W)
            for e in range(f["router"]["experts"]):
                for n, sh in (("gate", (f["expert"]["ff"], W)), ("up", (f["expert"]["ff"], W)), ("down", (W, f["expert"]["ff"]))):
                    s[f"{p}mlp.e{e}.{n}"] = sh
    return s


def random_weights(cfg, seed=0):
    """fp32 weights that let every mechanism show: loud gates and routers, biases and layer scales of every size, norm weights
    around 1."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in shapes(cfg).items():
        r = torch.randn(*s, generator=g)
        last = n.rsplit(".", 1)[-1]
        if last.startswith("norm"):
            r = 1.0 + 0.3 * r
        elif last == "b":
            r = 0.4 * r
        elif last in ("ls1", "ls2"):
            r = 0.5 + 0.3 * r
        elif last == "canon1":
            r = 0.5 * r
        elif last in ("embed", "bigram"):
            r = r * 0.7
        else:
            r = r * {"router": 2.5, "g": 2.0, "uq": 1.8, "uk": 1.5, "gate": 1.5, "up": 1.5}.get(last, 1.0) * s[-1] ** -0.5
        out[n] = r
    return out
