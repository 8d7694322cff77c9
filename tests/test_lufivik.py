"""Lufivik through the framework against the plain implementation of ``lufivik_oracle``: every mechanism alone, whole prompts,
portions, mixed batches, reused pages and slots, windows and loops, long decoding, greedy generation.  The same tests run the
operators' CPU form and, on a GPU, the kernels in true 32-bit and in bf16."""
import copy
import json
import random

import pytest
import torch

import lufivik_oracle as O
import test_sotazen as S
from b200fw import ops
from b200fw.infer import InferenceConfig, InferenceEngine
from b200fw.infer.hybrid import build_portions
from b200fw.model import registry
from b200fw.model.lufivik import LufivikConfig
from b200fw.ops.portions import pad8
from test_ruburax import close
from test_sotazen import COUNTS, CPU_RUN, P8, RUNS, bf16_exact, engine, feed_cuts, layout, loud_keys, near, packed, randn, rows_of, steps_of, toks


# ---- configurations -------------------------------------------------------------------------------------------------------
def latent(heads, dim, rot, vdim, q_rank, rank, window, ff=None, scale=0.3, base=700.0):
    return {"type": "latent_attention", "mlp": ff, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": rank, "scale": scale, "mask": {"size": window},
        "rot": {"base": base, "dims": rot}}}


def moe(experts, top, ff, limit=0.8):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, loop=None, taps=3, buckets=31, mul=(5, 3), eps=1e-5):
    return {"architecture": "Lufivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}},
            **({} if loop is None else {"loop": dict(zip(("start", "stop", "times"), loop))})}


# odd sizes on purpose: nothing a multiple of eight, sizes and windows that differ from layer to layer, a missing feed-forward, a loop
# that starts with the first layer
ODD = config(42, 67, [latent(3, 11, 6, 13, 19, 20, 23, moe(6, 3, 10)), latent(5, 20, 10, 9, 27, 37, 5), latent(1, 10, 2, 21, 12, 12, 40, moe(9, 1, 12, 0.4))],
             loop=(0, 2, 2))
# unit constants: one tap, one bucket, no loop, as many experts as are chosen, a window longer than any sequence, a limit that is never met
PLAIN = config(64, 96, [latent(4, 32, 16, 32, 48, 48, 1000, moe(4, 4, 24, 50.0), 0.2), latent(2, 16, 32, 16, 64, 32, 16, moe(8, 2, 40), 0.25)], taps=1,
               buckets=1, mul=(1, 1), eps=1e-3)
# heads as wide as a real model's and more of them than a tensor-core tile has rows, a window across several tiles, many experts, a loop
# of the last layer
WIDE = config(96, 80, [latent(18, 128, 64, 128, 200, 256, 150, moe(16, 4, 72), 0.05, 5e4), latent(2, 96, 32, 64, 72, 512, 64, moe(80, 6, 40, 1.5), 0.08),
                       latent(8, 64, 8, 128, 96, 128, 129, moe(12, 3, 48), 0.1)], loop=(2, 3, 3), taps=4, buckets=1009, mul=(48271, 16807))
CONFIGS = {"odd": ODD, "plain": PLAIN, "wide": WIDE}
_cache = {}


def case(name, seed=1):
    if (name, seed) not in _cache:
        _cache[name, seed] = (CONFIGS[name], bf16_exact(O.random_weights(CONFIGS[name], seed)))
    return _cache[name, seed]


def expected(name, seq):
    """Logits, and which positions choose their experts by a narrow margin in some run."""
    key = (name, tuple(seq))
    if key not in _cache:
        margins = []
        out = O.forward(*case(name), seq, margins=margins)
        _cache[key] = out, torch.stack(margins).min(0).values < 0.05
    return _cache[key]


def build(cfg, weights, run):
    m = registry.build_model(LufivikConfig.from_dict(cfg), dtype=run[1], device=run[0])
    registry.load_slots(m, weights.items())
    return m


def on_run(run):
    return lambda t: t.to(run[1]).to(run[0])


def tolerance(run):
    return dict(rtol=1e-2, atol=1e-2) if run[1] == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)


# ---- mechanisms alone -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("n,buckets,mul", [(8, 1, (1, 1)), (42, 31, (5, 3)), (200, 499, (11, 1)), (2560, 97, (10 ** 9 + 7, 998244353)), (9000, 11, (3, 0))])
def test_embedding_of_pairs(run, n, buckets, mul):
    """Portions cut anywhere: the token before a portion comes from the sequence's slot, the first token of a sequence has a row of its
    own even where the slot holds another request's token."""
    V, eps, on = 53, 1e-5, on_run(run)
    W = {k: randn(*s, seed=i).bfloat16().float() for i, (k, s) in enumerate((("embed", (V, n)), ("bigram", (buckets + 1, n)), ("w", (n,)), ("b", (n,)),
                                                                              ("nw", (n,)), ("nb", (n,))))}
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}}}
    seqs = [toks(sum(c), V, 7 + i) for i, c in enumerate(COUNTS)]
    D = {k: v.double() for k, v in W.items()}
    want = [O.embedding(s, cfg, {**D, "embed.norm": D["w"], "embed.norm.b": D["b"]}, eps) for s in seqs]
    last = torch.full((len(seqs),), 17, dtype=torch.int32, device=run[0])
    table, pairs, w, b, nw, nb = (on(P8(W[k])) for k in ("embed", "bigram", "w", "b", "nw", "nb"))
    for starts, cnt in steps_of(COUNTS):
        p, order, _ = layout(starts, cnt, run)
        ids = torch.tensor([t for s in order for t in seqs[s][starts[s]:starts[s] + cnt[s]]], device=run[0])
        x, h = ops.embedding_pairs(ids, table, pairs, last, p, V, mul[0], mul[1], (w, b), n, eps, (nw, nb))
        ref = torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order])
        torch.testing.assert_close(x.double().cpu()[:, :n], ref, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(h.double().cpu()[:, :n], O.layer_norm(ref, D["nw"], D["nb"], eps), **tolerance(run))
        assert h.dtype == run[1] and not x[:, n:].any() and not h[:, n:].any()


@pytest.mark.gpu
def test_embedding_of_padding_rows():
    """Rows of a graph batch without a sequence: any id, no slot."""
    bf = lambda *s, seed: randn(*s, seed=seed).bfloat16().to("cuda")  # noqa: E731
    p, _, _ = build_portions([4, 0, 9], [1, 1, 1], [[0], [1], [2]], [1, -1, -1], False, lambda a: torch.from_numpy(a).to("cuda"))
    last = torch.tensor([5, 6], dtype=torch.int32, device="cuda")
    x, h = ops.embedding_pairs(torch.tensor([3, 10 ** 12, -4], device="cuda"), bf(11, 16, seed=1), bf(8, 16, seed=2), last, p, 11, 3, 2,
                               (bf(16, seed=3), bf(16, seed=4)), 16, 1e-5, (bf(16, seed=5), bf(16, seed=6)))
    assert torch.isfinite(x).all() and torch.isfinite(h).all() and last.tolist() == [5, 3]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("C,K", [(8, 1), (42, 3), (264, 4), (96, 2), (520, 17)])
def test_input_convolution(run, C, K):
    on = on_run(run)
    taps = randn(C, K, seed=1).bfloat16().float() * 0.5
    data = [[randn(sum(c), C, seed=20 + i, run=run)] for i, c in enumerate(COUNTS)]
    want = [h[0].double() + O.causal_conv(h[0].double(), taps.double()) for h in data]
    state = torch.full((len(data), pad8(C), K - 1), 7.0, device=run[0])
    tp = on(torch.nn.functional.pad(taps, (0, 0, 0, pad8(C) - C)))
    for starts, cnt in steps_of(COUNTS):
        p, order, _ = layout(starts, cnt, run)
        h = on(P8(rows_of(data, order, starts, cnt)[0]))
        u = ops.causal_conv(h, None, tp, None, state, p, add_input=True)
        ref = torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order])
        torch.testing.assert_close(u.double().cpu()[:, :C], ref, **tolerance(run))


def unturned(k, i, base):
    """The query part that a turn by position i makes equal to ``k [heads, rot]`` (halves paired)."""
    out, half = k.clone(), k.shape[-1] // 2
    for c in range(half):
        a = torch.tensor(i * base ** (-2.0 * c / (2 * half)), dtype=torch.float64)
        u, v = k[..., c], k[..., c + half]
        out[..., c] = u * torch.cos(a) + v * torch.sin(a)
        out[..., c + half] = v * torch.cos(a) - u * torch.sin(a)
    return out


def neighbours(t):
    """Channels paired as halves, as they are stored: pairs next to each other."""
    half = t.shape[-1] // 2
    return torch.stack([t[..., :half], t[..., half:]], -1).flatten(-2)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dim,rot,dv,q_rank,rank,window", [
    (3, 11, 6, 13, 19, 20, 23), (4, 72, 24, 64, 96, 80, 16), (2, 128, 64, 128, 512, 512, 150), (18, 96, 32, 64, 40, 128, 17), (1, 160, 32, 24, 24, 40, 64),
    (2, 40, 24, 136, 33, 72, 1), (5, 128, 8, 128, 8, 264, 128), (2, 24, 2, 8, 50, 600, 31), (2, 180, 20, 32, 16, 16, 100), (2, 16, 16, 16, 64, 24, 1000),
    (1, 8, 8, 8, 8, 8, 2), (16, 128, 64, 128, 64, 512, 65)])
def test_windowed_latent_attention(run, H, dim, rot, dv, q_rank, rank, window):
    """Queries from a latent, one loud key per query: just inside and just outside the window, on page borders, the query's own; half of
    them loud through the rotated part alone.  A gate per head."""
    eps, base, on = 1e-6, 300.0, on_run(run)
    scale = 3.0 / (dim + rot) ** 0.5
    T = [sum(c) for c in COUNTS]
    nw, nq = ((1 + 0.2 * randn(n, seed=i)).bfloat16().float() for i, n in ((2, rank), (7, q_rank)))
    uk, uv = (randn(H * d, rank, seed=i).mul(rank ** -0.5).bfloat16().float() for i, d in ((3, dim), (4, dv)))
    data, want = [], []
    for s, t in enumerate(T):
        cq, c, kr, g = (randn(t, 1, d, seed=50 * s + i, run=run) for i, d in enumerate((q_rank, rank, rot, H)))
        cn = O.rms(c[:, 0].double(), eps) * nw.double()
        keys = O.latent_keys(cn, O.rotate_halves(kr.double(), base)[:, 0], uk.double(), H)
        q = randn(t, H, dim + rot, seed=50 * s + 9)
        for i, j in loud_keys(t, window, 3 * s).items():
            if i % 2 and rot >= 8:
                q[i, :, :dim] = 0
                q[i, :, dim:] = unturned(keys[j, :, dim:], i, base).float() * 2 * (dim / rot) ** 0.5
            else:
                q[i, :, :dim] = keys[j, :, :dim].float()
        q = q.bfloat16().float() if run[1] == torch.bfloat16 else q
        stored = torch.cat([q[..., :dim], neighbours(q[..., dim:])], -1)
        data.append((cq, c, neighbours(kr), g, stored))
        qt = torch.cat([q[..., :dim].double(), O.rotate_halves(q[..., dim:].double(), base)], -1)
        o = O.window_attention(qt, keys, (cn @ uv.double().T).reshape(t, H, dv), scale, window)
        want.append((o * O.sigmoid(g[:, 0].double())[:, :, None], O.rms(cq[:, 0].double(), eps) * nq.double()))
    Cp, Rp, dqp = pad8(rank), pad8(rank) + pad8(rot), pad8(dim + rot)
    w_key, w_value = torch.zeros(H, dqp, Rp), torch.zeros(H, pad8(dv), Cp)
    w_key[:, :dim, :rank], w_value[:, :dv, :rank] = uk.reshape(H, dim, rank), uv.reshape(H, dv, rank)
    for i in range(rot):
        w_key[:, dim + i, Cp + i] = 1.0
    w_key, w_value, norm, norm_q = on(w_key), on(w_value), on(P8(nw)), on(P8(nq))
    pages = None
    for starts, cnt in steps_of(COUNTS):
        p, order, n = layout(starts, cnt, run)
        if pages is None:
            pages = torch.full((n, 16, 1, Rp), 3.0 if run[1] == torch.bfloat16 else float("nan"), dtype=run[1], device=run[0])
        rows = rows_of(data, order, starts, cnt)
        cq, c, kr, g = packed(rows[:4], run)
        q = on(P8(rows[4]).reshape(p.rows, -1))
        cs, sn = ops.rope_rows(p.positions, ops.rope_turns(base, rot, run[0]))
        ops.latent_store(None, c, kr, pages, p, H, dim, rank, rot, norm, cs, sn, eps, cq, norm_q, q_rank)
        out = torch.full((p.rows, H * pad8(dv)), 9.0, dtype=run[1], device=run[0])
        ops.latent_attention(q, pages, out, p, w_key, w_value, scale, None, window, g[:, :H], (cs, sn, dim))
        ref, ref_q = (torch.cat([want[s][i][starts[s]:starts[s] + cnt[s]] for s in order]).float() for i in (0, 1))
        near(out.float().cpu().reshape(p.rows, H, -1)[:, :, :dv], ref, run)
        near(cq.float().cpu()[:, None, :q_rank], ref_q[:, None], run)


@pytest.mark.gpu
@pytest.mark.parametrize("window", [1, 33, 512])
def test_decoded_rows_in_a_window(window):
    """One token for each of many sequences, padding rows among them, against the 32-bit kernels on the same numbers."""
    r = random.Random(window)
    rows = 260
    lens = [r.choice([1, 2, 15, 16, 17, 32, 33, 34, window, window + 1, window + 15, window + 17, r.randrange(1, 900)]) for _ in range(rows)]
    need = [-(-n // 16) for n in lens]
    ids, tables = list(range(sum(need))), []
    r.shuffle(ids)
    for n in need:
        tables.append(ids[:n])
        ids = ids[n:]
    slots = [-1 if i % 7 == 3 else i for i in range(rows)]
    p, _, _ = build_portions([n - 1 for n in lens], [1] * rows, tables, slots, False, lambda a: torch.from_numpy(a).to("cuda"))
    live = torch.tensor([i for i in range(rows) if slots[i] >= 0], device="cuda")
    for H, R, C in ((8, 576, 512), (3, 80, 64), (18, 336, 264)):
        q, pages = randn(rows, H * R, seed=1).bfloat16().to("cuda"), randn(sum(need), 16, 1, R, seed=2).bfloat16().to("cuda")
        outs = []
        for dt in (torch.bfloat16, torch.float32):
            out = torch.full((rows, H * C), 9.0, dtype=dt, device="cuda")
            ops.latent_rows(q.to(dt), pages.to(dt), out, p, H, C, 2 * R ** -0.5, None, window)
            outs.append(out.float()[live])
        d = (outs[0] - outs[1]).pow(2).mean(-1).sqrt() / outs[1].std()
        assert torch.isfinite(outs[0]).all() and d.max() < 0.05, float(d.max())


def test_contexts_of_long_portions():
    """Only the pages that the window reaches are laid out, and every key of the window is found through the table."""
    starts, counts = [0, 100, 37, 500], [40, 64, 17, 90]
    tables = [[100 * i + j for j in range(-(-(s + c) // 16))] for i, (s, c) in enumerate(zip(starts, counts))]
    p, order, _ = build_portions(starts, counts, tables, [0, 1, 2, 3], False)
    assert order == [0, 1, 2, 3]
    for window in (0, 1, 16, 50, 10000):
        c = p.context(window)
        assert c is p.context(window)
        for i, (s, n) in enumerate(zip(starts, counts)):
            first = max(0, s - window + 1) if window else 0
            assert c.counts[i] == len(tables[i]) - first // 16
            for j in range(first // 16 * 16, s + n):
                assert int(c.pages[c.tables[i, j // 16]]) == tables[i][j // 16]
        assert int(c.tables.min()) >= 0 and int(c.tables.max()) < len(c.pages)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,N,K,first,rot", [(1, 16, 8, 8, 8), (3, 40, 24, 32, 6), (4, 192, 72, 128, 64), (2, 72, 328, 0, 2)])
def test_product_per_head_turned_and_gated(run, H, N, K, first, rot):
    on = on_run(run)
    for M in (1, 5, 130):
        x, w, g, a = randn(M, H * K, seed=1, run=run), randn(H, K, N, seed=2, run=run), randn(M, H + 8, seed=3, run=run), randn(M, rot // 2, seed=4)
        y = torch.einsum("mhk,hkn->mhn", x.double().reshape(M, H, K), w.double())
        c, s = torch.cos(a), torch.sin(a)
        u, v = y[:, :, first:first + rot:2].clone(), y[:, :, first + 1:first + rot:2].clone()
        y[:, :, first:first + rot:2] = u * c[:, None].double() - v * s[:, None].double()
        y[:, :, first + 1:first + rot:2] = v * c[:, None].double() + u * s[:, None].double()
        out = torch.zeros(M, H * N, dtype=run[1], device=run[0])
        ops.head_linear(on(x), on(w), out, transposed=True, turn=(c.to(run[0]), s.to(run[0]), first))
        assert (out.double().cpu() - y.reshape(M, -1)).abs().max() < (0.02 if run[1] == torch.bfloat16 else 1e-5) * y.abs().max()
        gate = on(g)[:, 8:]
        ops.head_linear(on(x), on(w.transpose(1, 2).contiguous()), out, gate=gate)
        y = torch.einsum("mhk,hkn->mhn", x.double().reshape(M, H, K), w.double()) * O.sigmoid(g[:, 8:].double())[:, :, None]
        assert (out.double().cpu() - y.reshape(M, -1)).abs().max() < (0.02 if run[1] == torch.bfloat16 else 1e-5) * y.abs().max()


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("n", [8, 42, 200, 2560, 9000])
def test_layer_norms_around_the_sum(run, n):
    """Rows with a mean far from zero; gate, scale and the next norm left out one by one."""
    ld, M, eps, on = pad8(n), 5, 1e-5, on_run(run)
    x, y, z = (P8(randn(M, n, seed=i)) for i in range(3))
    y[:, :n] += 30.0
    w, b, gb, s, nw, nb = (P8(randn(n, seed=10 + i)).bfloat16().float() for i in range(6))
    y, z = y.contiguous(), torch.cat([torch.full((M, 8), 50.0), z], 1)
    D = lambda t: t.double()[..., :n]  # noqa: E731
    for gate_dtype in {run[1], torch.float32}:
        zz = z.to(gate_dtype)
        for gate, scale, after in ((True, True, True), (False, True, True), (True, False, True), (True, True, False)):
            t = D(y) * (O.sigmoid(D(zz.float()[:, 8:]) + D(gb)) if gate else 1.0)
            want = D(x) + (D(s) if scale else 1.0) * O.layer_norm(t, D(w), D(b), eps)
            xs = x.clone().to(run[0])
            h = ops.branch_add(xs, y.to(run[0]), (on(w), on(b)), n, eps, zz.to(run[0])[:, 8:] if gate else None, on(gb) if gate else None,
                               on(s) if scale else None, (on(nw), on(nb)) if after else None)
            # the difference from a mean of 30 keeps 2^-24 * 30 of the 32-bit sums
            torch.testing.assert_close(D(xs.cpu()), want, rtol=1e-4, atol=2e-4 if run[1] == torch.float32 else 2e-3)
            assert not xs[:, n:].any()
            if not after:
                assert h is None
                continue
            assert h.dtype == run[1] and not h[:, n:].any()
            torch.testing.assert_close(D(h.cpu()), O.layer_norm(want, D(nw), D(nb), eps), rtol=1e-2 if run[1] == torch.bfloat16 else 1e-4,
                                       atol=2e-2 if run[1] == torch.bfloat16 else 2e-4)
    rows = torch.tensor([3, 0, 0], device=run[0])
    h = ops.layernorm_f32(y.to(run[0]), (on(w), on(b)), n, eps, rows)
    torch.testing.assert_close(D(h.cpu()), O.layer_norm(D(y), D(w), D(b), eps)[[3, 0, 0]], rtol=1e-2 if run[1] == torch.bfloat16 else 1e-4,
                               atol=2e-2 if run[1] == torch.bfloat16 else 2e-4)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,W", [(1, 1, 8), (6, 3, 42), (12, 12, 64), (40, 4, 72), (130, 5, 96), (300, 32, 40)])
def test_softmax_router(run, E, top, W):
    """Weights are the softmax over all experts, not made to add up to one; the order of nearly equal, tiny scores is that of the logits."""
    on, N = on_run(run), pad8(E)
    w = torch.zeros(N, pad8(W))
    w[:E, :W] = randn(E, W, seed=E) * W ** -0.5 * 6
    w = w.bfloat16().float()
    for M in (1, 23, 16384 // top + 5):
        h = P8(randn(M, W, seed=M)).bfloat16().float()
        z = h.double() @ w.double().T
        got = ops.route(ops.linear_fp32(on(h), on(w)), None, top, 1, 1, 1.0, score="softmax", experts=E)
        ids, weights, gap = O.choose(z[:, :E], top)
        off, place = got.offsets.cpu(), got.place.cpu()
        assert off[-1] == M * top and (place.reshape(-1).sort().values == torch.arange(M * top)).all()
        mine = torch.searchsorted(off, place, right=True) - 1
        clear = gap > 1e-4
        assert clear.float().mean() > 0.99 and torch.equal(mine[clear].sort(-1).values, ids[clear].sort(-1).values)
        torch.testing.assert_close(got.weights.double().cpu(), torch.softmax(z[:, :E], -1).gather(1, mine), rtol=1e-4, atol=1e-6)
        assert (got.token.cpu()[place.long()] == torch.arange(M)[:, None]).all()
    assert top == E or float(weights.sum(-1).min()) < 0.999
    same = ops.route(torch.zeros(2, N, device=run[0]), None, top, 1, 1, 1.0, score="softmax", experts=E)     # ties: the lower index
    assert torch.equal((torch.searchsorted(same.offsets.cpu(), same.place.cpu(), right=True) - 1).sort(-1).values, torch.arange(top).expand(2, top))


def test_softmax_scores_with_groups_and_correction():
    """The options of the choice are those of the sigmoid scores."""
    z, corr = randn(9, 8, seed=1), 0.05 * randn(8, seed=2)
    r = ops.route(z, corr, 2, 4, 2, 1.5, score="softmax")
    s = torch.softmax(z, -1)
    c = s + corr
    for t in range(9):
        groups = c[t].reshape(4, 2).sum(-1).topk(2).indices
        allowed = [e for e in range(8) if e // 2 in groups]
        ids = sorted(allowed, key=lambda e: -c[t, e])[:2]
        torch.testing.assert_close(r.weights[t], s[t, ids] * 1.5)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,F,W,limit", [(3, 2, 10, 20, 0.5), (8, 4, 72, 96, 7.0), (40, 6, 136, 64, 1.0), (4, 1, 300, 200, 0.2), (2, 2, 64, 328, 100.0)])
def test_clamped_experts(run, E, top, F, W, limit):
    """Gate and up around the limit on both sides (the gate has no lower one); experts with no rows, with a few and with more than a tile;
    the weighted sum, the gate of the branch, both norms."""
    eps, on = 1e-5, on_run(run)
    Fp, Wp = pad8(F), pad8(W)
    w_in, w_out = torch.zeros(E, 2, Fp, Wp), torch.zeros(E, Wp, Fp)
    w_in[:, :, :F, :W], w_out[:, :W, :F] = randn(E, 2, F, W, seed=1) * W ** -0.5 * min(3 * limit, 8.0), randn(E, W, F, seed=2) * F ** -0.5 * 1.5
    w_in, w_out = w_in.bfloat16().float(), w_out.bfloat16().float()
    w, b, gb, s, nw, nb = (P8(randn(W, seed=10 + i)).bfloat16().float() for i in range(6))
    D = lambda t: t.double()[..., :W]  # noqa: E731
    for M in (1, 5, 150, 700):
        h, z = P8(randn(M, W, seed=M)).bfloat16().float(), randn(M, pad8(E), seed=M + 1)
        z[:, E // 2:] -= 3.0                                  # the second half is hardly ever chosen
        r = ops.route(z.to(run[0]), None, top, 1, 1, 1.0, score="softmax", experts=E)
        rows = ops.expert_down(ops.expert_glu(on(h), on(w_in), r, (1.702, limit)), on(w_out), r)
        gate, x = P8(randn(M, W, seed=M + 3)), P8(randn(M, W, seed=M + 4))
        ids, weights, _ = O.choose(z.double()[:, :E], top)
        y = torch.zeros(M, Wp, dtype=torch.float64)
        for e in range(E):
            f = O.clamped_glu(h.double() @ w_in[e, 0].double().T, h.double() @ w_in[e, 1].double().T, limit)
            y += (f @ w_out[e].double().T) * (weights * (ids == e)).sum(1)[:, None]
        t = O.layer_norm(D(y) * O.sigmoid(D(gate) + D(gb)), D(w), D(b), eps)
        xs = x.clone().to(run[0])
        hn = ops.branch_add(xs, (rows, r), (on(w), on(b)), W, eps, gate.to(run[0]), on(gb), on(s), (on(nw), on(nb)))
        near((xs.cpu() - x)[:, None, :W], (D(s) * t)[:, None].float(), run)
        near(hn.float().cpu()[:, None, :W], O.layer_norm(D(x) + D(s) * t, D(nw), D(nb), eps)[:, None].float(), run)
        assert not xs[:, W:].any() and not hn[:, W:].any()


# ---- the whole model --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_layers_and_logits(run, name):
    cfg, w = case(name)
    seq, seen, margins = toks(45, cfg["vocab"]), [], []
    want = O.forward(cfg, w, seq, seen, margins)
    clear = torch.stack(margins).min(0).values > 0.05 if run[1] == torch.bfloat16 else torch.ones(45, dtype=torch.bool)
    eng = engine(build(cfg, w, run))
    eng.kv.allocate_for_sequence("a", 45)
    ctx, got = eng.runner.prepare_prefill(["a"], [0], [45]), []
    out = eng.runner.forward(torch.tensor(seq, device=run[0]), ctx, all_rows=True,
                             on_layer=lambda i, x: got.append(x[:, :cfg["width"]].double().cpu().clone()))
    assert len(got) == len(seen) == len(O.order_of_runs(cfg)) == eng.model.cfg.num_layers and clear.sum() > 15
    for i, (a, b) in enumerate(zip(got, seen)):
        e = (a - b)[clear].pow(2).mean().sqrt() / b.std()
        assert e < (0.03 if run[1] == torch.bfloat16 else 2e-5), f"run {i}: {float(e)}"
    S.close(out[clear.to(out.device)], want[clear], run)


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
    win = min(cfg["layers"][0]["mixer"]["mask"]["size"], 180)
    cuts = [[T], [2] * (T // 2), [100] + [1] * 110, [17, 64, 65, 63, 1], [win, 1, T - win - 2, 1], [win - 1, 2, T - win - 1], [128, 2, T - 130]]
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
    """A window longer than the sequence: the first token still moves the last logits after hundreds of decoded tokens."""
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
        moved = (wa[0][-1] - wb[0][-1]).norm()
        assert moved > 1e-4 and ((ga[-1] - gb[-1]).double().cpu() - (wa[0][-1] - wb[0][-1])).norm() < 0.1 * moved


@pytest.mark.parametrize("run", RUNS[:2])
@pytest.mark.parametrize("decoded", [False, True])
def test_reach_of_a_window(run, decoded):
    """One layer sees ``window - 1`` tokens back, through its convolution ``taps - 1`` more and through the token pairs one more: the first
    token that is out of reach changes nothing, the last one within it does."""
    window, taps, T = 9, 3, 60
    cfg = config(32, 50, [latent(2, 8, 8, 8, 16, 16, window, moe(4, 2, 8), scale=0.05)], taps=taps)
    w = bf16_exact(O.random_weights(cfg, 5))
    reach = (window - 1) + (taps - 1) + 1
    seq = toks(T, 50, 2)
    eng = engine(build(cfg, w, run))
    cuts = [20] + [1] * (T - 20) if decoded else [T]
    base = feed_cuts(eng, "a", seq, cuts).cpu()
    for j in (0, 7, 16, 30):
        other = list(seq)
        other[j] = (other[j] + 1) % 50
        moved = (feed_cuts(eng, "b", other, cuts).cpu() - base).abs().max(-1).values
        assert not moved[:j].any() and moved[j + reach] > 1e-7 and not moved[j + reach + 1:].any()


@pytest.mark.parametrize("run", RUNS[:2])
def test_looped_layers_are_the_same_layers_written_out(run):
    """Passing a layer again is the same as another layer with its weights; no pass sees another's keys or inputs."""
    layers = [latent(2, 8, 8, 8, 16, 16, 7, moe(4, 2, 8)), latent(3, 8, 4, 8, 8, 24, 12), latent(1, 16, 8, 8, 8, 8, 30, moe(3, 1, 8))]
    seq = toks(50, 40, 3)
    for loop in ((0, 3, 2), (1, 2, 4), (2, 3, 1), (1, 3, 3), (1, 1, 5), (0, 1, 2)):
        cfg = config(32, 40, copy.deepcopy(layers), loop=loop)
        w = bf16_exact(O.random_weights(cfg, 6))
        order = O.order_of_runs(cfg)
        flat = config(32, 40, [copy.deepcopy(layers[i]) for i in order])
        fw = {n: t for n, t in w.items() if not n.startswith("l")}
        for k, i in enumerate(order):
            fw |= {f"l{k}." + n.split(".", 1)[1]: t for n, t in w.items() if n.startswith(f"l{i}.")}
        m = build(cfg, w, run)
        assert m.layer_runs() == order and len(m.kv_layer_shapes()) == len(m.state_layer_shapes()) == len(order)
        got = feed_cuts(engine(m), "a", seq, [21, 1, 28])
        assert torch.equal(got, feed_cuts(engine(build(flat, fw, run)), "a", seq, [21, 1, 28]))
        S.close(got, O.forward(cfg, w, seq), run)


# ---- generation through the scheduler ---------------------------------------------------------------------------------------
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


# ---- loading ----------------------------------------------------------------------------------------------------------------
def test_checkpoint_round_trip_and_registry(tmp_path):
    cfg, w = case("odd")
    m = build(cfg, w, CPU_RUN)
    registry.save_checkpoint(m, str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    assert registry.architecture_at(str(tmp_path)).name == "Lufivik"
    assert {n: tuple(t.shape) for n, t in m.named_checkpoint_tensors()} == {n: tuple(s) for n, s in O.shapes(cfg).items()}
    for n, t in m.named_checkpoint_tensors():
        assert torch.equal(t, w[n]), n
    eng = InferenceEngine(InferenceConfig.from_model_config(registry.read_config(str(tmp_path)), num_blocks=16,
                                                            model_path=str(tmp_path), dtype="float32", max_num_sequences=2,
                                                            inference_mode="kv_cache", temperature=0.0)).initialize()
    if eng.device.type == "cpu":
        seq = toks(30, cfg["vocab"])
        S.close(eng.feed([("a", seq)])["a"], O.forward(cfg, w, seq), CPU_RUN)
        # new weights in place, through the engine's update path
        w2 = bf16_exact(O.random_weights(cfg, 9))
        assert eng.load_weights(w2) == len(w2)
        eng.release("a")
        S.close(eng.feed([("a", seq)])["a"], O.forward(cfg, w2, seq), CPU_RUN)


def test_bad_checkpoints_and_configs():
    cfg, w = case("odd")
    m = build(cfg, w, CPU_RUN)
    before = m.embed_tokens.clone()
    for change in ({"l0.norm1.b": None}, {"l9.norm1": torch.zeros(42)}, {"l1.mix.uq": torch.zeros(3, 3)}, {"l1.norm2": torch.zeros(42)}):
        items = {**w, **change, "embed": torch.zeros_like(w["embed"])}
        with pytest.raises(ValueError, match="nothing was loaded"):
            registry.load_slots(m, [(k, v) for k, v in items.items() if v is not None])
        assert torch.equal(m.embed_tokens, before)
    a = latent(2, 8, 4, 8, 8, 8, 5)

    def changed(**k):
        return {**copy.deepcopy(a), "mixer": {**a["mixer"], **k}}
    bad = [([{"type": "other", "mixer": {}}], "unknown type"), ([{"type": "latent_attention", "mixer": {"heads": 1}}], "missing"),
           ([changed(rot={"base": 10.0, "dims": 2})], "rotated size"), ([changed(mask={"size": 0})], "window"),
           ([{**a, "mlp": {"kind": "dense", "ff": 8}}], "feed-forward kind"), ([{**a, "mlp": {"kind": "moe", "expert": {"ff": 8}}}], "missing"),
           ([{**a, "mlp": {**moe(2, 1, 8), "expert": {"ff": 8}}}], "limit")]
    for layers, why in bad:
        with pytest.raises(ValueError, match=why):
            LufivikConfig.from_dict(config(8, 8, layers))
    for loop in ((0, 2, 2), (1, 0, 2), (0, 1, 0), (-1, 1, 2)):
        with pytest.raises(ValueError, match="loop"):
            LufivikConfig.from_dict(config(8, 8, [a], loop=loop))
    with pytest.raises(ValueError, match="missing"):
        LufivikConfig.from_dict({"vocab": 8})
    for kw, why in ((dict(taps=18), "taps"), (dict(taps=0), "taps")):
        with pytest.raises(ValueError, match=why):
            registry.build_model(LufivikConfig.from_dict(config(8, 8, [a], **kw)), device="cpu")
    with pytest.raises(ValueError, match="cannot choose"):
        registry.build_model(LufivikConfig.from_dict(config(8, 8, [{**a, "mlp": moe(2, 3, 8)}])), device="cpu")
    for kw in (dict(speculative_enabled=True), dict(kv_cache_dtype="fp8")):
        with pytest.raises(ValueError, match="recurrent state"):
            engine(m, **kw)
    for name in ("lufivik-tiny", "lufivik-0.6b"):
        c = registry.PRESETS[name]
        assert 0 < c.num_active_params() and c.num_layers == len(c.layer_runs()) > len(c.layers)
