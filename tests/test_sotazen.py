"""Sotazen through the framework against the plain implementation of ``sotazen_oracle``: every mechanism alone, whole
prompts, portions, mixed batches, reused pages and slots, long decoding, greedy generation.  The same tests run the
operators' CPU form and, on a GPU, the kernels in true 32-bit and in bf16."""
import json
import random

import pytest
import torch

import sotazen_oracle as O
from b200fw import ops
from b200fw.infer import InferenceConfig, InferenceEngine
from b200fw.infer.hybrid import build_portions
from b200fw.model import registry
from b200fw.model.sotazen import SotazenConfig
from b200fw.ops.portions import pad8

GPU = pytest.mark.gpu
CPU_RUN = ("cpu", torch.float32)
RUNS = [pytest.param(CPU_RUN, id="cpu"), pytest.param(("cuda", torch.float32), id="gpu-f32", marks=GPU),
        pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=GPU)]


def lightning(heads, dim, vdim, ff=24):
    return {"type": "lightning", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": [1.0 - 2.0 ** -(2 + 7 * h) for h in range(heads)]}}


def differential(heads, kv, dim, vdim, window, rot, diff=0.3, scale=0.3, cap=20.0, base=900.0, ff=24):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "diff": diff,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot}}}


def latent(heads, dim, rot, vdim, rank, scale=0.2, base=700.0, ff=24):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                      "rot": {"base": base, "dims": rot}}}


def config(width, vocab, layers, eps=1e-5, alpha=1.7, scale=3.0):
    return {"architecture": "Sotazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": scale}, "layers": layers}


# odd sizes on purpose: nothing a multiple of eight, sizes of q / k and v apart, groups, partial rotation, missing feed-forwards
ODD = config(42, 67, [latent(3, 11, 6, 13, 20), lightning(3, 20, 12, ff=None), differential(6, 2, 18, 10, 23, 10),
                      latent(5, 20, 10, 9, 37, ff=None), differential(3, 1, 10, 21, 5, 2, diff=0.8, ff=None)])
# a differential layer first, every head with its own key, a window of one page; unit constants
PLAIN = config(64, 96, [differential(4, 4, 32, 16, 16, 32, diff=0.1, cap=5.0), latent(4, 32, 16, 32, 48), lightning(2, 32, 32)],
               eps=1e-3, alpha=1.0, scale=1.0)
# heads as wide as a real model's, windows across several tiles, more heads than a tensor-core tile has rows
WIDE = config(96, 80, [lightning(2, 128, 64, ff=40), differential(4, 2, 128, 96, 150, 64, scale=0.08, cap=30.0, ff=40),
                       latent(18, 128, 64, 128, 256, scale=0.07, ff=40), lightning(1, 64, 128, ff=40)])
CONFIGS = {"odd": ODD, "plain": PLAIN, "wide": WIDE}


def bf16_exact(weights):
    return {k: v.bfloat16().float() for k, v in weights.items()}


_cache = {}


def case(name, seed=1):
    if (name, seed) not in _cache:
        _cache[name, seed] = (CONFIGS[name], bf16_exact(O.random_weights(CONFIGS[name], seed)))
    return _cache[name, seed]


def expected(name, seq):
    key = (name, tuple(seq))
    if key not in _cache:
        _cache[key] = O.forward(*case(name), seq)
    return _cache[key]


def build(cfg, weights, run):
    m = registry.build_model(SotazenConfig.from_dict(cfg), dtype=run[1], device=run[0])
    registry.load_slots(m, weights.items())
    return m


def engine(model, tokens=640, seqs=4, **kw):
    c = InferenceConfig.from_model_config(model.cfg, num_blocks=tokens // 16, max_num_sequences=seqs,
                                          **{"inference_mode": "kv_cache", "temperature": 0.0, **kw})
    return InferenceEngine(c, model).initialize()


def close(got, want, run, what=""):
    """Difference of logits with their mean taken off, relative to the size of the logits.  In bf16 a few positions amplify
    rounding (heads whose two maps cancel, or whose state answers a query with almost nothing, are normed up again): one in
    fifty may be further off, none by much."""
    got, want = got.double().cpu(), want.double().cpu()
    d = (got - got.mean(-1, keepdim=True)) - (want - want.mean(-1, keepdim=True))
    e = d.pow(2).mean(-1).sqrt() / want.std()
    if run[1] == torch.bfloat16:
        assert int((e > 0.06).sum()) <= max(1, len(e) // 50) and e.max() < 0.2, f"{what}: {e.topk(min(4, len(e)))}"
    else:
        assert e.max() < 2e-4, f"{what}: {float(e.max()):.6f} at {int(e.argmax())}"


def toks(n, vocab, seed=0):
    r = random.Random(seed)
    return [r.randrange(vocab) for _ in range(n)]


def feed_cuts(eng, rid, seq, cuts):
    assert sum(cuts) == len(seq)
    out, at = [], 0
    for c in cuts:
        out.append(eng.feed([(rid, seq[at:at + c])])[rid])
        at += c
    eng.release(rid)
    return torch.cat(out)


# ---- mechanisms alone -------------------------------------------------------------------------------------------
def layout(starts, counts, run, pages_each=24, seed=0):
    """A step's row layout with scattered pages and slots."""
    r = random.Random(seed)
    n = len(counts)
    ids, slots = list(range(n * pages_each)), list(range(n))
    r.shuffle(ids)
    r.shuffle(slots)
    tables = [ids[i * pages_each:(i + 1) * pages_each] for i in range(n)]
    dev = lambda a: torch.from_numpy(a).to(run[0])  # noqa: E731
    p, order, _ = build_portions(starts, counts, tables, slots, run[1] == torch.float32, dev)
    return p, order, n * pages_each


def steps_of(counts_per_seq):
    """[[portions of sequence 0], ...] -> per step (starts, counts) with every sequence present."""
    for k in range(len(counts_per_seq[0])):
        yield [sum(c[:k]) for c in counts_per_seq], [c[k] for c in counts_per_seq]


def P8(t):
    return torch.nn.functional.pad(t, (0, pad8(t.shape[-1]) - t.shape[-1]))


def packed(parts, run):
    """Side by side in one matrix, every head padded to eight: parts [(tensor [M, H, d])] -> slices."""
    M = parts[0].shape[0]
    flat = [P8(t).reshape(M, -1) for t in parts]
    y = torch.cat(flat, 1).to(run[1]).to(run[0])
    out, at = [], 0
    for f in flat:
        out.append(y[:, at:at + f.shape[1]])
        at += f.shape[1]
    return out


def near(got, ref, run):
    """``[rows, heads, size]``: every head of every row, relative to the size of the outputs."""
    assert torch.isfinite(got).all()
    e = ((got - ref).pow(2).mean(-1).sqrt() / ref.std()).max()
    assert e < (0.06 if run[1] == torch.bfloat16 else 5e-4), float(e)


def randn(*s, seed=0, run=None):
    t = torch.randn(*s, generator=torch.Generator().manual_seed(seed))
    return t.bfloat16().float() if run is None or run[1] == torch.bfloat16 else t


COUNTS = [[1, 5, 40, 1, 1], [17, 2, 64, 70, 1], [65, 130, 1, 16, 33]]


def rows_of(data, order, starts, cnt):
    """The step's rows of every per-sequence tensor, in the kernels' order."""
    return [torch.cat([data[s][i][starts[s]:starts[s] + cnt[s]] for s in order]) for i in range(len(data[0]))]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dk,dv", [(3, 20, 12), (2, 128, 64), (1, 8, 136), (2, 64, 128)])
def test_lightning_state(run, H, dk, dv):
    """The recurrence, and the norm over all heads that is split between it and the sum after the output projection."""
    eps, decay = 1e-6, [0.5, 0.97, 0.9995][:H]
    T = [sum(c) for c in COUNTS]
    nw = (1 + 0.3 * randn(H, dv, seed=3)).bfloat16().float()
    data = [[randn(t, H, d, seed=10 * s + i, run=run) for i, d in enumerate((dk, dk, dv, dv))] for s, t in enumerate(T)]
    want = []
    for q, k, v, g in data:
        o = O.lightning_core(q.double(), k.double(), v.double(), decay).reshape(-1, H * dv)
        want.append((O.rms(o, eps) * nw.double().reshape(-1) * O.sigmoid(g.double().reshape(-1, H * dv))).reshape(-1, H, dv))
    state = torch.full((len(T), H, pad8(dk), pad8(dv)), 7.0, device=run[0])     # slots hold another request's leftovers
    w = P8(nw).reshape(-1).to(run[1]).to(run[0])
    for starts, cnt in steps_of(COUNTS):
        p, order, _ = layout(starts, cnt, run)
        q, k, v, g = packed(rows_of(data, order, starts, cnt), run)
        out = torch.full((p.rows, H * pad8(dv)), 9.0, dtype=run[1], device=run[0])
        ss = torch.full((p.rows, H), float("nan"), device=run[0])
        ops.retention(q, k, v, g, out, state, p, torch.tensor(decay, device=run[0]), dk, dv, None, None, 1.0, eps, w, ss)
        got = out.float() / torch.sqrt(ss.sum(-1, keepdim=True) / (H * dv) + eps)
        near(got.cpu().reshape(p.rows, H, -1)[:, :, :dv], torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float(), run)


def loud_keys(T, window, seed):
    """For some queries a key that should stand out: around the window's edge, on page and tile borders, the query itself."""
    r, pick = random.Random(seed), {}
    for i in range(0, T, 3):
        e = i - window + 1
        j = r.choice([e, e - 1, e + 1, i, i - 1, i // 16 * 16, i // 16 * 16 - 1, e // 16 * 16, i // 128 * 128, 0, 1])
        pick[i] = min(max(j, 0), i)
    return pick


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,window,rot,cap", [
    (6, 2, 12, 20, 24, 8, 20.0), (5, 1, 9, 7, 37, 6, 3.0), (4, 2, 128, 96, 150, 64, 30.0), (4, 1, 96, 128, 128, 96, 8.0),
    (8, 1, 64, 64, 17, 2, 45.0), (2, 2, 160, 24, 40, 12, 15.0), (3, 3, 128, 128, 1, 128, 35.0), (2, 1, 64, 128, 1000, 32, 100.0),
    (1, 1, 24, 72, 129, 24, 6.0), (2, 1, 24, 136, 30, 8, 25.0), (9, 1, 32, 40, 33, 16, 9.0)])
def test_differential_attention(run, H, G, dk, dv, window, rot, cap):
    """One loud key per query and map at a time, the two maps' apart.  A key that is wrongly seen, or missed, takes the whole
    softmax with it; a cap that is left out sharpens every score."""
    eps, scale, diff = 1e-6, 9.0 / dk, 0.35
    T = [sum(c) for c in COUNTS]
    wq, wk = ((1 + 0.3 * randn(dk, seed=i)).bfloat16().float() for i in (5, 6))
    lams = [(0.3 * randn(dk, seed=20 + i)).bfloat16().float() for i in range(4)]
    bias = [(0.4 * randn(n, d, seed=30 + i)).bfloat16().float() for i, (n, d) in enumerate(((2 * H, dk), (2 * G, dk), (G, dv)))]
    lam = O.diff_lambda(*(t.double() for t in lams), diff)
    data, want = [], []
    for s, t in enumerate(T):
        q, k, v = randn(t, H, 2, dk, seed=40 * s), randn(t, G, 2, dk, seed=40 * s + 1), randn(t, G, dv, seed=40 * s + 2, run=run)
        for m in range(2):
            keys = O.rotate_pairs((O.rms(k[:, :, m] + bias[1].reshape(G, 2, dk)[:, m], eps) * wk).double(), 500.0, rot)
            for i, j in loud_keys(t, window, 7 * s + m).items():
                # the query that meets key j head on: the key as the score sees it, turned back by the query's own position
                back = keys[j].clone()
                for c in range(rot // 2):
                    a = torch.tensor(i * 500.0 ** (-2.0 * c / rot), dtype=torch.float64)
                    u, z = back[:, 2 * c].clone(), back[:, 2 * c + 1].clone()
                    back[:, 2 * c] = u * torch.cos(a) + z * torch.sin(a)
                    back[:, 2 * c + 1] = z * torch.cos(a) - u * torch.sin(a)
                raw = back.float().repeat_interleave(H // G, 0) / wq
                q[i, :, m] = raw * 2 - bias[0].reshape(H, 2, dk)[:, m]
        if run[1] == torch.bfloat16:
            q, k = q.bfloat16().float(), k.bfloat16().float()
        gate = randn(t, H, dv, seed=40 * s + 3, run=run)
        data.append((q.reshape(t, 2 * H, dk), k.reshape(t, 2 * G, dk), v, gate))
        qn = O.rms(data[-1][0].double() + bias[0].double(), eps) * wq.double()
        kn = O.rms(data[-1][1].double() + bias[1].double(), eps) * wk.double()
        qn, kn = O.rotate_pairs(qn, 500.0, rot).reshape(t, H, 2, dk), O.rotate_pairs(kn, 500.0, rot).reshape(t, G, 2, dk)
        o = O.differential_core(qn, kn, v.double() + bias[2].double(), lam, diff, scale, window, cap, eps)
        want.append(o * O.sigmoid(gate.double()))
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    turns = ops.rope_turns(500.0, rot, run[0])
    b = on(torch.cat([P8(x).reshape(-1) for x in bias]))
    l4 = on(torch.stack([P8(x) for x in lams]))
    kc = vc = None
    for starts, cnt in steps_of(COUNTS):
        p, order, pages = layout(starts, cnt, run)
        if kc is None:
            # the tiled kernel may read, masked, what a page holds past its sequence: finite leftovers there
            junk = 3.0 if run[1] == torch.bfloat16 else float("nan")
            kc = torch.full((pages, 16, 2 * G, pad8(dk)), junk, dtype=run[1], device=run[0])
            vc = torch.full((pages, 16, G, pad8(dv)), junk, dtype=run[1], device=run[0])
        q, k, v, g = packed(rows_of(data, order, starts, cnt), run)
        cs, sn = ops.rope_rows(p.positions, turns)
        qn = ops.qk_norm_store(q, k, v, kc, vc, p, 2 * H, dk, True, eps, on(P8(wq)), on(P8(wk)), b, cs, sn)
        out = torch.full((p.rows, H * pad8(dv)), 9.0, dtype=run[1], device=run[0])
        ops.differential_attention(qn, kc, vc, out, p, H, scale, l4, diff, dv, eps, g, window, cap)
        near(out.float().cpu().reshape(p.rows, H, -1)[:, :, :dv],
             torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float(), run)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dim,rot,dv,rank", [(3, 11, 6, 13, 20), (4, 72, 24, 64, 80), (2, 128, 64, 128, 512), (18, 96, 32, 64, 128),
                                               (1, 160, 32, 24, 40), (2, 40, 24, 136, 72), (5, 128, 8, 128, 264), (2, 24, 2, 8, 600),
                                               (2, 180, 20, 32, 16)])
def test_latent_attention(run, H, dim, rot, dv, rank):
    """One loud key per query: far away, on page borders, the first token, the query's own; and a sink that weighs in."""
    eps, base = 1e-6, 300.0
    scale = 3.0 / (dim + rot) ** 0.5
    T = [sum(c) for c in COUNTS]
    nw = (1 + 0.2 * randn(rank, seed=2)).bfloat16().float()
    uk, uv = (randn(H * d, rank, seed=i).mul(rank ** -0.5).bfloat16().float() for i, d in ((3, dim), (4, dv)))
    sink = (2.0 + randn(H, seed=6)).bfloat16().float()
    data, want = [], []
    for s, t in enumerate(T):
        q, c, kr = randn(t, H, dim + rot, seed=50 * s), randn(t, 1, rank, seed=50 * s + 1), randn(t, 1, rot, seed=50 * s + 2)
        cn = O.rms(c[:, 0].double(), eps) * nw.double()
        kt = O.rotate_pairs(kr.double(), base, rot)[:, 0]
        keys = O.latent_keys(cn, kt, uk.double(), H)
        for i, j in loud_keys(t, t + 1, 3 * s).items():
            q[i, :, :dim] = keys[j, :, :dim].float()
        q = q.bfloat16().float() if run[1] == torch.bfloat16 else q
        data.append((q, c, kr))
        qt = torch.cat([q[..., :dim].double(), O.rotate_pairs(q[..., dim:].double(), base, rot)], -1)
        want.append(O.sink_attention(qt, keys, (cn @ uv.double().T).reshape(t, H, dv), scale, sink.double()))
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    Cp, Rp, dqp = pad8(rank), pad8(rank) + pad8(rot), pad8(dim + rot)
    w_key, w_value = torch.zeros(H, dqp, Rp), torch.zeros(H, pad8(dv), Cp)
    w_key[:, :dim, :rank], w_value[:, :dv, :rank] = uk.reshape(H, dim, rank), uv.reshape(H, dv, rank)
    for i in range(rot):
        w_key[:, dim + i, Cp + i] = 1.0
    w_key, w_value, norm, snk = on(w_key), on(w_value), on(P8(nw)), on(sink)
    pages = None
    for starts, cnt in steps_of(COUNTS):
        p, order, n = layout(starts, cnt, run)
        if pages is None:
            pages = torch.full((n, 16, 1, Rp), 3.0 if run[1] == torch.bfloat16 else float("nan"), dtype=run[1], device=run[0])
        q, c, kr = packed(rows_of(data, order, starts, cnt), run)
        cs, sn = ops.rope_rows(p.positions, ops.rope_turns(base, rot, run[0]))
        ops.latent_store(q, c, kr, pages, p, H, dim, rank, rot, norm, cs, sn, eps)
        out = torch.full((p.rows, H * pad8(dv)), 9.0, dtype=run[1], device=run[0])
        ops.latent_attention(q, pages, out, p, w_key, w_value, scale, snk)
        near(out.float().cpu().reshape(p.rows, H, -1)[:, :, :dv],
             torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float(), run)


@pytest.mark.gpu
@pytest.mark.parametrize("rows,longest", [(1, 900), (3, 40), (300, 500), (1100, 90)])
def test_decoded_rows_of_ragged_lengths(rows, longest):
    """One token for each of many sequences, padding rows among them: the work split over the SMs cuts rows anywhere.  Against the
    32-bit kernels on the same numbers."""
    r = random.Random(rows)
    lens = [r.choice([1, 2, 15, 16, 17, 31, 32, 33, 64, 65, r.randrange(1, longest)]) for _ in range(rows)]
    lens[-1] = longest
    pads = [i for i in range(rows - 1) if i % 7 == 3]
    need = [-(-n // 16) for n in lens]
    ids, tables = list(range(sum(need))), []
    r.shuffle(ids)
    for n in need:
        tables.append(ids[:n])
        ids = ids[n:]
    slots = [-1 if i in pads else i for i in range(rows)]
    p, _, _ = build_portions([n - 1 for n in lens], [1] * rows, tables, slots, False, lambda a: torch.from_numpy(a).to("cuda"))
    bf = lambda *s, seed: randn(*s, seed=seed).bfloat16().to("cuda")  # noqa: E731
    live = torch.tensor([i for i in range(rows) if i not in pads], device="cuda")

    def same(f, width):
        outs = []
        for dt in (torch.bfloat16, torch.float32):
            out = torch.full((rows, width), 9.0, dtype=dt, device="cuda")
            f(out, lambda t: t.to(dt))
            outs.append(out.float()[live])
        assert torch.isfinite(outs[0]).all()
        d = (outs[0] - outs[1]).pow(2).mean(-1).sqrt() / outs[1].std()
        assert d.max() < 0.05, float(d.max())
    for H, G, d, dv, window, cap in ((8, 4, 128, 128, 0, 40.0), (6, 2, 24, 40, 37, 2.0), (20, 1, 64, 64, 100, 30.0)):
        q, kc, vc = bf(rows, 2 * H * d, seed=1) * 2, bf(sum(need), 16, 2 * G, d, seed=2), bf(sum(need), 16, G, dv, seed=3)
        lam, gate = bf(4, d, seed=4) * 0.1, bf(rows, H * dv, seed=5)
        same(lambda o, c: ops.differential_attention(c(q), c(kc), c(vc), o, p, H, d ** -0.5, c(lam), 0.4, dv, 1e-6, c(gate), window, cap),
             H * dv)
    for H, R, C in ((8, 576, 512), (3, 80, 64), (18, 336, 264), (16, 24, 16)):
        q, pages, sink = bf(rows, H * R, seed=1), bf(sum(need), 16, 1, R, seed=2), bf(H, seed=3) + 2
        same(lambda o, c: ops.latent_rows(c(q), c(pages), o, p, H, C, 2 * R ** -0.5, c(sink)), H * C)


@pytest.mark.gpu
def test_latent_contexts_in_groups(monkeypatch):
    """Contexts too large to expand at once are expanded in groups of sequences, or not at all."""
    from b200fw.ops import latent as L
    H, dim, rot, dv, rank, run = 2, 32, 16, 24, 40, ("cuda", torch.bfloat16)
    starts, counts = [30, 0, 64, 5, 0], [40, 1, 100, 17, 33]
    p, _, n = layout(starts, counts, run)
    on = lambda *s, seed: randn(*s, seed=seed).bfloat16().to("cuda")  # noqa: E731
    q, pages = on(p.rows, H * (dim + rot), seed=1), on(n, 16, 1, rank + rot, seed=2)
    wk, wv, sink = on(H, dim + rot, rank + rot, seed=3), on(H, dv, rank, seed=4), on(H, seed=5)
    outs = []
    row = H * (dim + rot + dv) * 2
    for limit in (1 << 30, 16 * row * 12, 16 * row * 11, 0):
        monkeypatch.setattr(L, "MAX_EXPANDED_BYTES", limit)
        out = torch.empty(p.rows, H * dv, dtype=torch.bfloat16, device="cuda")
        ops.latent_attention(q, pages, out, p, wk, wv, 0.05, sink)
        outs.append(out.float())
    assert torch.equal(outs[0], outs[1]) and torch.equal(outs[0], outs[2])
    assert (outs[0] - outs[3]).abs().max() < 0.05 * outs[0].abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("window,cap", [(0, 0.0), (40, 0.0), (0, 4.0), (130, 4.0)])
def test_window_and_cap_on_plain_heads(window, cap):
    """The two options without differential heads."""
    H, G, d, run = 4, 2, 64, ("cuda", torch.bfloat16)
    starts, counts = [100, 0, 64, 200], [1, 130, 90, 16]
    p, _, n = layout(starts, counts, run)
    q, kc, vc = (randn(*s, seed=i).bfloat16().to("cuda") for i, s in enumerate(((p.rows, H * d), (n, 16, G, d), (n, 16, G, d))))
    out = torch.empty(p.rows, H * d, dtype=torch.bfloat16, device="cuda")
    ops.paged_attention(q, kc, vc, out, p, H, 0.3, window=window, softcap=cap)
    pc, _, _ = layout(starts, counts, ("cpu", torch.bfloat16))
    ref = torch.empty(p.rows, H * d)
    ops.paged_attention(q.cpu(), kc.cpu(), vc.cpu(), ref, pc, H, 0.3, window=window, softcap=cap)
    near(out.float().cpu().reshape(-1, H, d), ref.reshape(-1, H, d), run)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("M,N,K,cols", [(1, 8, 8, 8), (3, 40, 24, 24), (130, 200, 72, 200), (257, 1000, 640, 520), (300, 512, 128, 448)])
def test_products_with_activation(run, M, N, K, cols):
    a, b = randn(M, K, seed=1), randn(N, K, seed=2) * K ** -0.5 * 3
    b = b.bfloat16().float()
    z = a.double() @ b.double().t()
    for act, f in (("silu", O.silu), ("relu2", O.relu2)):
        want = z.clone()
        want[:, :cols] = f(z[:, :cols])
        got = ops.linear_act(a.to(run[1]).to(run[0]), b.to(run[1]).to(run[0]), act, cols).double().cpu()
        tol = dict(rtol=1e-2, atol=1e-2) if run[1] == torch.bfloat16 else dict(rtol=1e-5, atol=1e-4)
        torch.testing.assert_close(got, want, **tol)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,N,K", [(1, 8, 8), (3, 40, 24), (4, 192, 72), (2, 64, 328)])
def test_product_per_head(run, H, N, K):
    for M in (1, 5, 130):
        x, w = randn(M, H * K, seed=1), randn(H, N, K, seed=2)
        on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
        wide = on(torch.cat([x, x], 1))
        out = torch.zeros(M, H * N + 8, dtype=run[1], device=run[0])
        want = torch.einsum("mhk,hnk->mhn", x.double().reshape(M, H, K), w.double()).reshape(M, -1)
        for t, wt in ((False, w), (True, w.transpose(1, 2).contiguous())):
            ops.head_linear(wide[:, :H * K], on(wt), out[:, 8:], transposed=t)
            assert (out[:, 8:].double().cpu() - want).abs().max() < (0.02 if run[1] == torch.bfloat16 else 1e-4) * want.abs().max()
            assert not out[:, :8].any()


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("n", [8, 42, 200, 9000])
def test_sum_then_norm(run, n):
    ld, M, eps, alpha = pad8(n), 5, 1e-5, 2.3
    x, y, w, b = (P8(randn(*s, seed=i)) for i, s in enumerate(((M, n), (M, n), (n,), (n,))))
    ss = randn(M, 3, seed=9) ** 2 * 20
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    for bias, sums in ((None, None), (b, None), (None, ss), (b, ss)):
        z = y.double() if sums is None else y.double() / torch.sqrt(sums.double().sum(-1, keepdim=True) / 12 + eps)
        z = alpha * x.double() + z + (0 if bias is None else bias.double())
        want = O.rms(z[:, :n], eps) * w[:n].double()
        xs = x.clone().to(run[0])
        h = ops.post_norm(xs, y.to(run[0]), on(w), alpha, n, eps, None if bias is None else on(bias),
                          None if sums is None else sums.to(run[0]), 12)
        torch.testing.assert_close(xs[:, :n].double().cpu(), want, rtol=1e-5, atol=1e-5)
        assert h.dtype == run[1] and not xs[:, n:].any()
        torch.testing.assert_close(h[:, :n].double().cpu(), want, rtol=1e-2 if run[1] == torch.bfloat16 else 1e-5, atol=1e-5)
    table = on(P8(randn(11, n, seed=4)))
    x0, h0 = ops.embedding_f32(torch.tensor([3, 0, 10], device=run[0]), table, 11, 12.5, h=True)
    torch.testing.assert_close(x0.cpu(), table.float().cpu()[[3, 0, 10]] * 12.5, rtol=1e-6, atol=0)
    assert h0.dtype == run[1] and torch.equal(h0, x0.to(run[1]))


# ---- the whole model ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_layers_and_logits(run, name):
    cfg, w = case(name)
    seq, seen = toks(45, cfg["vocab"]), []
    want = O.forward(cfg, w, seq, seen)
    eng = engine(build(cfg, w, run))
    eng.kv.allocate_for_sequence("a", 45)
    ctx, got = eng.runner.prepare_prefill(["a"], [0], [45]), []
    out = eng.runner.forward(torch.tensor(seq, device=run[0]), ctx, all_rows=True,
                             on_layer=lambda i, x: got.append(x[:, :cfg["width"]].double().cpu().clone()))
    assert len(got) == len(seen)
    for i, (a, b) in enumerate(zip(got, seen)):
        assert (a - b).pow(2).mean().sqrt() / b.std() < (0.03 if run[1] == torch.bfloat16 else 2e-5), f"layer {i}"
    close(out, want, run)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_decoding(run, name):
    """The logits of every position do not depend on where the prompt was cut, down to two tokens and to one."""
    cfg, w = case(name)
    T = 210
    seq = toks(T, cfg["vocab"], 3)
    want = expected(name, seq)
    eng = engine(build(cfg, w, run))
    r = random.Random(5)
    win = [l["mixer"]["mask"]["size"] for l in cfg["layers"] if l["type"] == "attention"]
    cuts = [[T], [2] * (T // 2), [100] + [1] * 110, [17, 64, 65, 63, 1], [win[0], 1, T - win[0] - 2, 1],
            [win[-1] - 1, 2, T - win[-1] - 1]]
    rnd = []
    while sum(rnd) < T:
        rnd.append(min(r.choice([1, 2, 3, 16, 31, 48, 80]), T - sum(rnd)))
    for c in cuts + [rnd]:
        close(feed_cuts(eng, "a", seq, c), want, run, f"{c[:8]}...")
    assert eng.kv.pool.num_used_blocks == 0 and eng.kv.state.num_free_slots == 4


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_unequal_batches_and_reused_slots(run, name):
    """Requests of different lengths come and go in one small pool; portions beside decoded tokens, requests left out of steps."""
    cfg, w = case(name)
    r = random.Random(11)
    lens = [3, 150, 33, 90, 1, 64, 17, 129, 47]
    seqs = [toks(n, cfg["vocab"], 40 + i) for i, n in enumerate(lens)]
    want = [expected(name, s) for s in seqs]
    eng = engine(build(cfg, w, run), tokens=160 + 96 + 144 + 64)
    at, live, waiting, got = {}, [], list(range(len(seqs))), {i: [] for i in range(len(seqs))}
    while waiting or live:
        while waiting and len(live) < 4 and sum(-(-lens[i] // 16) for i in live + waiting[:1]) <= eng.kv.pool.num_blocks:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        step = [i for i in live if r.random() < 0.8] or live[:1]
        r.shuffle(step)
        entries = []
        for i in step:
            n = min(r.choice([1, 1, 2, 5, 20, 64, 70]), lens[i] - at[i])
            entries.append((f"q{i}", seqs[i][at[i]:at[i] + n]))
            at[i] += n
        out = eng.feed(entries)
        for i in step:
            got[i].append(out[f"q{i}"])
            if at[i] == lens[i]:
                eng.release(f"q{i}")
                live.remove(i)
    for i in range(len(seqs)):
        close(torch.cat(got[i]), want[i], run, f"request {i}")
    assert eng.kv.pool.num_used_blocks == 0 and eng.kv.state.num_free_slots == 4


@pytest.mark.parametrize("run", RUNS)
def test_long_decoding_remembers(run):
    """A decay close to one and a latent cache: the first token still moves the last logits after hundreds of decoded tokens."""
    cfg, w = case("plain")
    T = 400
    a, b = toks(T, cfg["vocab"], 8), toks(T, cfg["vocab"], 8)
    b[0] = (b[0] + 1) % cfg["vocab"]
    eng = engine(build(cfg, w, run))
    wa, wb = expected("plain", a), expected("plain", b)
    ga = feed_cuts(eng, "a", a, [5] + [1] * (T - 5))
    close(ga, wa, run)
    if run[1] == torch.float32:
        gb = feed_cuts(eng, "b", b, [T])
        moved = (wa[-1] - wb[-1]).norm()
        assert moved > 1e-3 and ((ga[-1] - gb[-1]).double().cpu() - (wa[-1] - wb[-1])).norm() < 0.05 * moved


# ---- generation through the scheduler -------------------------------------------------------------------------------
def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(O.forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("run", RUNS[:2])
def test_greedy_generation(run):
    cfg, w = case("odd")
    prompts = [toks(n, cfg["vocab"], 60 + n) for n in (5, 41, 1, 60, 23, 30)]
    if "greedy" not in _cache:
        _cache["greedy"] = [greedy(cfg, w, p, 8) for p in prompts]
    want = _cache["greedy"]
    m = build(cfg, w, run)
    # more requests than slots, chunked prompts beside decoding ones, too few pages for all (preemption)
    for kw in (dict(seqs=3, chunk_size=16, max_prefill_tokens=32), dict(seqs=6, tokens=192, chunk_size=24),
               dict(seqs=6, enable_cuda_graph=True), dict(seqs=4, async_decode="force", chunk_size=32)):
        eng = engine(m, **kw)
        assert eng.generate(prompts, max_tokens=8) == want, kw
        assert eng.kv.pool.num_used_blocks == 0 and eng.kv.state.num_free_slots == kw["seqs"], kw
    assert engine(m, inference_mode="eager").generate(prompts[:2], max_tokens=4) == [x[:4] for x in want[:2]]


@pytest.mark.gpu
def test_graph_decoding_matches_plain_bf16():
    cfg, w = case("wide")
    m = build(cfg, w, ("cuda", torch.bfloat16))
    prompts = [toks(n, cfg["vocab"], 80 + n) for n in (40, 3, 130, 64, 77)]
    outs = [engine(m, tokens=1600, seqs=5, enable_cuda_graph=g).generate(prompts, max_tokens=24) for g in (False, True)]
    assert outs[0] == outs[1]


# ---- loading ----------------------------------------------------------------------------------------------------------
def test_checkpoint_round_trip_and_registry(tmp_path):
    cfg, w = case("odd")
    m = build(cfg, w, CPU_RUN)
    registry.save_checkpoint(m, str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    assert registry.architecture_at(str(tmp_path)).name == "Sotazen"
    eng = InferenceEngine(InferenceConfig.from_model_config(registry.read_config(str(tmp_path)), num_blocks=16,
                                                            model_path=str(tmp_path), dtype="float32", max_num_sequences=2,
                                                            inference_mode="kv_cache", temperature=0.0)).initialize()
    if eng.device.type == "cpu":
        for (n, a), (n2, b) in zip(m.named_checkpoint_tensors(), eng.model.named_checkpoint_tensors()):
            assert n == n2 and torch.equal(a, b) and torch.equal(a, w[n])
        seq = toks(30, cfg["vocab"])
        close(eng.feed([("a", seq)])["a"], expected("odd", seq), CPU_RUN)
        # new weights in place, through the engine's update path
        w2 = bf16_exact(O.random_weights(cfg, 9))
        assert eng.load_weights(w2) == len(w2)
        eng.release("a")
        close(eng.feed([("a", seq)])["a"], O.forward(cfg, w2, seq), CPU_RUN)


def test_bad_checkpoints_and_configs():
    cfg, w = case("odd")
    m = build(cfg, w, CPU_RUN)
    before = m.embed_tokens.clone()
    for change in ({"l0.norm1": None}, {"l9.norm1": torch.zeros(42)}, {"l0.mix.dkv": torch.zeros(3, 3)}):
        items = {**w, **change, "embed": torch.zeros_like(w["embed"])}
        with pytest.raises(ValueError, match="nothing was loaded"):
            registry.load_slots(m, [(k, v) for k, v in items.items() if v is not None])
        assert torch.equal(m.embed_tokens, before)
    bad = [({"type": "other", "mixer": {}}, "unknown type"), ({"type": "lightning", "mixer": {"heads": 1}}, "missing"),
           ({**latent(1, 8, 4, 8, 8), "mlp": {"kind": "sparse"}}, "feed-forward kind")]
    for layer, why in bad:
        with pytest.raises(ValueError, match=why):
            SotazenConfig.from_dict(config(8, 8, [layer]))
    wrong = latent(1, 8, 4, 8, 8)
    wrong["mixer"]["rot"] = {"base": 10.0, "dims": 2}
    with pytest.raises(ValueError, match="rotated size"):
        SotazenConfig.from_dict(config(8, 8, [wrong]))
    with pytest.raises(ValueError, match="missing required"):
        SotazenConfig.from_dict({"vocab": 8})
    with pytest.raises(ValueError, match="do not divide"):
        build(*(lambda c: (c, O.random_weights(c)))(config(8, 8, [differential(3, 2, 8, 8, 4, 2)])), CPU_RUN)
    for kw in (dict(speculative_enabled=True), dict(kv_cache_dtype="fp8")):
        with pytest.raises(ValueError, match="recurrent state"):
            engine(m, **kw)
    for name in ("sotazen-tiny", "sotazen-0.6b"):
        assert registry.PRESETS[name].num_params() > 0
