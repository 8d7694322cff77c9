"""Ruburax through the framework against the plain implementation of ``ruburax_oracle``: every mechanism alone, whole prompts,
portions, mixed batches, reused pages and slots, long decoding, greedy generation.  The same tests run the operators' CPU form
and, on a GPU, the kernels in true 32-bit and in bf16."""
import copy
import json
import math
import random

import pytest
import torch

import ruburax_oracle as O
import test_sotazen as S
from b200fw import _native, ops
from b200fw.infer import InferenceConfig, InferenceEngine
from b200fw.model import registry
from b200fw.model.ruburax import RuburaxConfig
from b200fw.ops.portions import pad8
from test_sotazen import COUNTS, CPU_RUN, P8, RUNS, bf16_exact, engine, feed_cuts, layout, near, packed, randn, rows_of, steps_of, toks


# ---- configurations -------------------------------------------------------------------------------------------------------
def rot(dims, base=700.0, scaling=None):
    return {"base": base, "dims": dims, **({} if scaling is None else {"scaling": dict(zip(("factor", "low", "high", "original"), scaling))})}


def att(heads, kv, dim, vdim, r, scale=0.3, kv_from=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": r, **({} if kv_from is None else {"kv_from": kv_from})}


def attention(*a, ff=None, **k):
    return {"type": "attention", "mixer": att(*a, **k), "mlp": ff}


def parallel(left, heads, dim, vdim, cap, ls, rs, ff=None):
    return {"type": "parallel", "mlp": ff, "mixer": {"left": left, "left_scale": ls, "right_scale": rs, "right": {
        "heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}}


def rglru(width, blocks, conv, ff=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": ff}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, shared=None, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, **({} if shared is None else {"shared": {"ff": shared}}),
            "router": {"experts": experts, "top": top, "scale": scale,
                       **({} if groups is None else {"groups": {"count": groups[0], "keep": groups[1]}})}}


def config(width, vocab, layers, eps=1e-5, mult=0.7, logit=0.6, side=12):
    return {"architecture": "Ruburax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit,
            "layers": layers, **({} if side is None else {"token_side": {"dim": side}})}


STRETCH = (5.0, 1.0, 3.0, 40)
# odd sizes on purpose: nothing a multiple of eight, sizes of q / k and v apart, groups of heads, partial rotation, missing
# feed-forwards, several layers over the keys of one that is not the layer before, one-expert groups, blocks that need padding
ODD = config(42, 67, [
    rglru(27, 3, 5, ff=moe(6, 3, 10, (3, 2), 14)), attention(6, 2, 18, 10, rot(10, 300.0, STRETCH)),
    parallel(att(3, 1, 10, 21, rot(4)), 3, 11, 6, 9.0, 0.8, -1.4, ff=dense(21)), attention(4, 2, 18, 10, rot(10, 300.0, STRETCH), kv_from=1, ff=moe(9, 2, 12)),
    rglru(20, 1, 2, ff=moe(5, 2, 9, (5, 3), 9, 3.0)), attention(2, 2, 18, 10, rot(10, 300.0, STRETCH), kv_from=1, scale=0.5, ff=dense(13))], side=5)
# every head with its own key, unit constants, no token input, one tap, as many experts as are chosen
PLAIN = config(64, 96, [attention(4, 4, 32, 32, rot(32), ff=moe(4, 4, 24)), parallel(att(2, 2, 16, 32, rot(0)), 2, 32, 32, 3.0, 1.0, 1.0, ff=dense(48)),
                        rglru(64, 4, 1, ff=moe(8, 1, 40, (2, 1), 16, 1.0))], eps=1e-3, mult=1.0, logit=1.0, side=None)
# heads as wide as a real model's, more query heads than a tensor-core tile has rows, many experts
WIDE = config(96, 80, [attention(18, 1, 128, 96, rot(64, 5e4, (8.0, 1.0, 4.0, 64)), scale=0.09, ff=dense(200)),
                       parallel(att(4, 2, 128, 128, rot(128)), 2, 128, 64, 15.0, 0.5, 0.9, ff=moe(16, 4, 72, (4, 2), 136)),
                       attention(2, 1, 128, 96, rot(64, 5e4, (8.0, 1.0, 4.0, 64)), scale=0.09, kv_from=0, ff=moe(40, 6, 40, (8, 4))),
                       rglru(256, 2, 4, ff=moe(12, 3, 48, (4, 3), 48))], side=24)
CONFIGS = {"odd": ODD, "plain": PLAIN, "wide": WIDE}
_cache = {}


def case(name, seed=1):
    if (name, seed) not in _cache:
        _cache[name, seed] = (CONFIGS[name], bf16_exact(O.random_weights(CONFIGS[name], seed)))
    return _cache[name, seed]


def expected(name, seq):
    """Logits, and which positions choose their experts by a narrow margin in some layer."""
    key = (name, tuple(seq))
    if key not in _cache:
        margins = []
        out = O.forward(*case(name), seq, margins=margins)
        _cache[key] = out, torch.stack(margins).min(0).values < 0.05
    return _cache[key]


def close(got, want, run, what=""):
    """In bf16 a position whose experts are chosen by a narrow margin may take another one: it is not compared.  A few others may
    still be off, because a neighbour took another expert or because their router saw more rounding than the margin."""
    want, narrow = want
    if run[1] != torch.bfloat16:
        return S.close(got, want, run, what)
    got, want = got.double().cpu()[~narrow], want[~narrow]
    if len(got):
        d = (got - got.mean(-1, keepdim=True)) - (want - want.mean(-1, keepdim=True))
        e = d.pow(2).mean(-1).sqrt() / want.std()
        assert e.median() < 0.03 and int((e > 0.12).sum()) <= max(2, len(e) // 20) and e.max() < 0.6, f"{what}: {e.topk(min(4, len(e)))}"


def build(cfg, weights, run):
    m = registry.build_model(RuburaxConfig.from_dict(cfg), dtype=run[1], device=run[0])
    registry.load_slots(m, weights.items())
    return m


# ---- mechanisms alone -------------------------------------------------------------------------------------------------------
def test_stretched_frequencies():
    for base, dims, s in ((1e4, 32, (8.0, 1.0, 4.0, 512)), (250.0, 10, (3.0, 0.5, 2.0, 64)), (7e5, 64, (32.0, 1.0, 4.0, 8192)), (50.0, 6, None)):
        want = O.frequencies(base, dims, None if s is None else dict(zip(("factor", "low", "high", "original"), s)))
        got = ops.rope_turns(base, dims, "cpu", s) * 2 * math.pi
        torch.testing.assert_close(got, torch.tensor(want, dtype=torch.float64), rtol=1e-12, atol=0)
    kept = ops.rope_turns(1e4, 32, "cpu", (8.0, 1.0, 4.0, 512)) / ops.rope_turns(1e4, 32, "cpu")
    assert kept[0] == 1 and abs(kept[-1] - 1 / 8) < 1e-12 and ((kept > 0.13) & (kept < 0.99)).any()


def halves(t, dims):
    """Channels of the checkpoint's order (pairs i, i + dims / 2) in the stored one (pairs 2 i, 2 i + 1), over the last dimension."""
    order = [j for i in range(dims // 2) for j in (i, i + dims // 2)] + list(range(dims, t.shape[-1]))
    return t[..., order]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,rd,sink,stretch", [
    (6, 2, 12, 20, 8, True, (4.0, 1.0, 3.0, 30)), (5, 1, 9, 7, 6, True, None), (4, 2, 128, 96, 64, False, None), (4, 1, 96, 128, 96, True, None),
    (20, 1, 64, 64, 2, True, (8.0, 1.0, 4.0, 64)), (2, 2, 160, 24, 40, False, None), (3, 3, 128, 128, 128, True, None), (1, 1, 24, 136, 0, True, None),
    (8, 4, 128, 128, 128, True, None), (2, 1, 40, 200, 32, True, None)])
def test_attention_and_shared_keys(run, H, G, dk, dv, rd, sink, stretch):
    """One loud key per query: far away, on page and tile borders, the first tokens, the query's own; and a sink heavy enough to show.
    A second set of queries, with half of the heads, reads the same pages."""
    eps, scale, base = 1e-6, 4.0 / dk ** 0.5 / dk ** 0.5 * 3, 500.0
    T = [sum(c) for c in COUNTS]
    freqs = O.frequencies(base, rd, None if stretch is None else dict(zip(("factor", "low", "high", "original"), stretch)))
    wq, wk = ((1 + 0.3 * randn(dk, seed=i)).bfloat16().float() for i in (5, 6))
    H2 = max(G, H // 2 // G * G)
    bias = [(0.4 * randn(n, d, seed=30 + i)).bfloat16().float() for i, (n, d) in enumerate(((H, dk), (G, dk), (G, dv)))]
    bias2 = (0.4 * randn(H2, dk, seed=33)).bfloat16().float()
    snk = (6.0 + randn(H, seed=7)).bfloat16().float() if sink else None
    data, want = [], []
    for s, t in enumerate(T):
        q, k, v = randn(t, H, dk, seed=40 * s), randn(t, G, dk, seed=40 * s + 1), randn(t, G, dv, seed=40 * s + 2, run=run)
        q2 = randn(t, H2, dk, seed=40 * s + 3)
        if run[1] == torch.bfloat16:
            k = k.bfloat16().float()
        kn = O.rotate_halves(O.rms(k.double() + bias[1].double(), eps) * wk.double(), freqs)
        for qs, b, seed in ((q, bias[0], 7 * s), (q2, bias2, 7 * s + 1)):
            for i, j in S.loud_keys(t, t + 1, seed).items():
                # the query that meets key j head on: the key as the score sees it, turned back by the query's own position
                back = kn[j].clone()
                for c, f in enumerate(freqs):
                    a, n = torch.tensor(i * f, dtype=torch.float64), len(freqs)
                    u, z = back[:, c].clone(), back[:, c + n].clone()
                    back[:, c], back[:, c + n] = u * torch.cos(a) + z * torch.sin(a), z * torch.cos(a) - u * torch.sin(a)
                qs[i] = back.float().repeat_interleave(qs.shape[1] // G, 0) / wq * 2 - b
        if run[1] == torch.bfloat16:
            q, q2 = q.bfloat16().float(), q2.bfloat16().float()
        data.append((q, k, v, q2))
        outs = []
        for qs, b, sk in ((q, bias[0], snk), (q2, bias2, None if snk is None else snk[:H2])):
            qn = O.rotate_halves(O.rms(qs.double() + b.double(), eps) * wq.double(), freqs)
            outs.append(O.causal_attention(qn, kn, v.double() + bias[2].double(), scale, None if sk is None else sk.double()))
        want.append(outs)
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    st = lambda t: P8(halves(t, rd))  # noqa: E731
    turns = ops.rope_turns(base, rd, run[0], stretch) if rd else None
    b = on(torch.cat([st(bias[0]).reshape(-1), st(bias[1]).reshape(-1), P8(bias[2]).reshape(-1)]))
    kc = vc = None
    for starts, cnt in steps_of(COUNTS):
        p, order, pages = layout(starts, cnt, run)
        if kc is None:
            # the tiled kernel may read, masked, what a page holds past its sequence: finite leftovers there
            junk = 3.0 if run[1] == torch.bfloat16 else float("nan")
            kc = torch.full((pages, 16, G, pad8(dk)), junk, dtype=run[1], device=run[0])
            vc = torch.full((pages, 16, G, pad8(dv)), junk, dtype=run[1], device=run[0])
        rows = rows_of(data, order, starts, cnt)
        q, k, v, q2 = packed([halves(rows[0], rd), halves(rows[1], rd), rows[2], halves(rows[3], rd)], run)
        cs, sn = ops.rope_rows(p.positions, turns) if rd else (None, None)
        for i, (qq, heads) in enumerate(((q, H), (q2, H2))):
            kv = (k, v) if i == 0 else (None, None)
            qn = ops.qk_norm_store(qq, *kv, kc, vc, p, heads, dk, True, eps, on(st(wq)), on(st(wk)) if i == 0 else None,
                                   b if i == 0 else on(st(bias2).reshape(-1)), cs, sn)
            out = torch.full((p.rows, heads * pad8(dv)), 9.0, dtype=run[1], device=run[0])
            ops.paged_attention(qn, kc, vc, out, p, heads, scale, sink=None if snk is None else on(snk[:heads]))
            near(out.float().cpu().reshape(p.rows, heads, -1)[:, :, :dv],
                 torch.cat([want[s][i][starts[s]:starts[s] + cnt[s]] for s in order]).float(), run)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dk,dv,cap", [(3, 20, 12, 5.0), (2, 128, 64, 15.0), (1, 8, 136, 2.0), (2, 64, 128, 30.0), (1, 128, 128, 12.0), (1, 200, 24, 9.0),
                                         (2, 24, 248, 9.0), (4, 96, 32, 15.0)])
def test_matrix_memory(run, H, dk, dv, cap):
    """Gates from wide open to shut, so that the running maximum rises, falls below zero and is carried; slots hold leftovers."""
    eps, qs, os = 1e-6, dk ** -0.5, -1.3
    T = [sum(c) for c in COUNTS]
    nw = (1 + 0.3 * randn(H, dv, seed=3)).bfloat16().float()
    bi, bf = (randn(2, H, seed=4) * 2).bfloat16().float()
    bf = bf + 3.0
    data, want = [], []
    for s, t in enumerate(T):
        q, k, v, g = (randn(t, H, d, seed=10 * s + i, run=run) for i, d in enumerate((dk, dk, dv, dv)))
        z = randn(t, 2, H, seed=10 * s + 5) * 6
        z[:, 1] = z[:, 1].abs() + torch.where(torch.rand(t, H, generator=torch.Generator().manual_seed(s)) < 0.05, -12.0, 2.0)
        z[t // 3:t // 2, 0] -= 25.0                     # a stretch of tokens that writes nothing: the maximum decays with f
        data.append((q, k, v, g, z))
        i = cap * torch.tanh((z[:, 0] + bi).double() / cap)
        f = -O.softplus(-cap * torch.tanh((z[:, 1] + bf).double() / cap))
        o = O.memory_core(q.double() * qs, k.double(), v.double(), i, f)
        want.append(O.rms(o, eps) * nw.double() * O.sigmoid(g.double()) * os)
    S_ = torch.full((len(T), H, pad8(dk), pad8(dv)), 7.0, device=run[0])
    n_, m_ = torch.full((len(T), H, pad8(dk)), 7.0, device=run[0]), torch.full((len(T), H), 7.0, device=run[0])
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    for starts, cnt in steps_of(COUNTS):
        p, order, _ = layout(starts, cnt, run)
        rows = rows_of(data, order, starts, cnt)
        q, k, v, g = packed(rows[:4], run)
        z = P8(rows[4]).reshape(p.rows, -1).to(run[0])
        out = torch.full((p.rows, H * pad8(dv)), 9.0, dtype=run[1], device=run[0])
        ops.matrix_memory(q, k, v, g, z[:, :H], z[:, pad8(H):pad8(H) + H], on(bi), on(bf), out, S_, n_, m_, p, on(P8(nw)).reshape(-1), dk, dv,
                          cap, qs, os, eps)
        near(out.float().cpu().reshape(p.rows, H, -1)[:, :, :dv], torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float(), run)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("B,n,K", [(3, 9, 5), (1, 20, 2), (2, 64, 4), (4, 128, 4), (2, 176, 4), (5, 40, 1), (1, 256, 3), (2, 24, 17), (3, 320, 4)])
def test_gated_recurrence(run, B, n, K):
    """Convolution, gates, recurrence and gelu branch; channels that forget at once and channels that keep for thousands of tokens."""
    C, np_ = B * n, pad8(n)
    T = [sum(c) for c in COUNTS]
    w = lambda *s, seed, f=1.0: (randn(*s, seed=seed) * f).bfloat16().float()  # noqa: E731
    xb, yb, cb, taps = w(C, seed=1, f=0.5), w(C, seed=2, f=0.5), w(C, seed=3, f=0.3), w(C, K, seed=4, f=0.6)
    ra, ri = w(B, n, n, seed=5, f=n ** -0.5 * 2), w(B, n, n, seed=6, f=n ** -0.5 * 2)
    rab, rib, lam = w(B, n, seed=7), w(B, n, seed=8), torch.linspace(-11.0, 2.0, C)[torch.randperm(C, generator=torch.Generator().manual_seed(1))].bfloat16().float()
    data = [tuple(randn(t, C, seed=20 * s + i, run=run) for i in range(2)) for s, t in enumerate(T)]
    want = []
    for y, x in data:
        u = O.causal_conv(x.double() + xb.double(), taps.double(), cb.double())
        want.append(O.recurrence_core(u, ra.double(), rab.double(), ri.double(), rib.double(), lam.double()) * O.gelu_tanh(y.double() + yb.double()))
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    vec = lambda t: on(P8(t.reshape(B, n))).reshape(-1)  # noqa: E731
    tp = torch.zeros(B, np_, K)
    tp[:, :n] = taps.reshape(B, n, K)
    wg, gb = torch.zeros(B, 2, np_, np_), torch.zeros(B, 2, np_)
    wg[:, 0, :n, :n], wg[:, 1, :n, :n], gb[:, 0, :n], gb[:, 1, :n] = ra, ri, rab, rib
    state, conv = torch.full((len(T), B * np_), 7.0, device=run[0]), torch.full((len(T), B * np_, K - 1), 7.0, device=run[0])
    for starts, cnt in steps_of(COUNTS):
        p, order, _ = layout(starts, cnt, run)
        y, x = packed([r.reshape(-1, B, n) for r in rows_of(data, order, starts, cnt)], run)
        out = torch.full((p.rows, B * np_), 9.0, dtype=run[1], device=run[0])
        ops.gated_recurrence(y, x, vec(yb), vec(xb), on(tp).reshape(B * np_, K), vec(cb), on(wg), on(gb), vec(lam), out, state, conv, p)
        ref = torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float()
        got = out.float().cpu().reshape(p.rows, B, np_)
        assert not got[:, :, n:].any()
        near(got[:, :, :n].reshape(p.rows, 1, C), ref.reshape(p.rows, 1, C), run)
    # every channel at the end, from its own state
    if run[1] == torch.float32:
        u = [O.causal_conv(x.double() + xb.double(), taps.double(), cb.double()) for _, x in data]
        for s in range(len(T)):
            core = O.recurrence_core(u[s], ra.double(), rab.double(), ri.double(), rib.double(), lam.double())[-1].reshape(B, n)
            slot = int(p.slots[order.index(s)])
            torch.testing.assert_close(state[slot].cpu().reshape(B, np_)[:, :n].double(), core, rtol=1e-4, atol=1e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("B,n", [(2, 160), (3, 24), (1, 256)])
def test_gated_recurrence_over_many_chunks(B, n):
    """More chunks than thread blocks, so that every block walks several of them; blocks of channels that leave lanes without one.
    Against the operators' unfused form on the same numbers."""
    run, C, np_ = ("cuda", torch.bfloat16), B * n, pad8(n)
    T = 64 * 148 * 2 // B * 3 + 40
    on = lambda *s, seed, f=1.0: (randn(*s, seed=seed) * f).bfloat16().to("cuda")  # noqa: E731
    y, x, bias = on(T, C, seed=1), on(T, C, seed=2), [on(C, seed=3 + i, f=0.5) for i in range(3)]
    taps, wg, gb, lam = on(C, 4, seed=7, f=0.5), on(B, 2, np_, np_, seed=8, f=n ** -0.5 * 2), on(B, 2, np_, seed=9), on(C, seed=10, f=2.0) - 4
    p, _, _ = layout([0], [T], run, pages_each=T // 16 + 1)
    outs, states = [], []
    for fused in (True, False):
        out, state, conv = torch.zeros(T, C, dtype=torch.bfloat16, device="cuda"), torch.zeros(1, C, device="cuda"), torch.zeros(1, C, 3, device="cuda")
        if fused:
            ops.gated_recurrence(y, x, bias[0], bias[1], taps, bias[2], wg, gb, lam, out, state, conv, p)
        else:
            u = ops.causal_conv(x, bias[1], taps, bias[2], conv, p)
            ops.linear_recurrence(u, ops.block_gates(u, wg.view(B, 2 * np_, np_)), gb.view(-1), lam, y, bias[0], out, state, p, np_)
        outs.append(out.float())
        states.append(state)
    assert _native.read_status() == 0
    near(outs[0].cpu()[:, None], outs[1].cpu()[:, None], run)
    torch.testing.assert_close(states[0], states[1], rtol=2e-3, atol=2e-3)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,groups,keep", [(6, 3, 3, 2), (5, 2, 5, 3), (8, 1, 2, 1), (9, 9, 1, 1), (64, 6, 8, 3), (256, 8, 8, 4), (40, 6, 8, 4), (33, 4, 11, 2),
                                               (1, 1, 1, 1), (1000, 32, 10, 5)])
def test_routing(run, E, top, groups, keep):
    """Choice scores are negative for most experts (a closed group must not count as zero), and the correction decides the choice but
    not the weight; with and without an expert that every token takes."""
    M = 37
    z, corr = randn(M, pad8(E) + 1, seed=E), (randn(E, seed=E + 1) - 1.5).bfloat16().float()
    zd = z.to(run[0])
    for joint in (False, True) if top < 32 else (False,):
        r = ops.route(zd[:, :-1], corr.to(run[1]).to(run[0]), top, groups, keep, 2.5, zd[:, -1] if joint else None)
        place, token, off, w = r.place.cpu(), r.token.cpu(), r.offsets.cpu(), r.weights.cpu()
        n = M * (top + joint)
        assert off[0] == 0 and off[-1] == n and len(off) == E + joint + 1 and sorted(place.reshape(-1).tolist()) == list(range(n))
        s = O.sigmoid(z.double())
        for t in range(M):
            ids = O.route(s[t, :E], corr.double(), top, None if keep == groups else {"count": groups, "keep": keep})
            got = torch.searchsorted(off, place[t], right=True) - 1
            assert sorted(got.tolist()) == sorted(ids + [E] * joint) and (token[place[t].long()] == t).all()
            want = s[t][got.long()] * 2.5
            if joint:
                assert got[-1] == E
                want[-1] = s[t, -1]
            torch.testing.assert_close(w[t].double(), want, rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,groups,keep,W,shared", [(6, 3, 3, 2, 42, True), (32, 4, 8, 4, 1000, True), (64, 6, 8, 3, 264, False), (80, 2, 4, 2, 128, True),
                                                       (1, 1, 1, 1, 8, True)])
def test_router_product(run, E, top, groups, keep, W, shared):
    """The product and the choice together, with rows that fill no tile, and enough of them for both ways of laying out the pairs."""
    n = pad8(E) + (8 if shared else 0)
    w = torch.zeros(n, pad8(W))
    w[:E, :W] = (randn(E, W, seed=1) * W ** -0.5).bfloat16().float()
    w[pad8(E):, :W] = (randn(n - pad8(E), W, seed=2) * W ** -0.5).bfloat16().float()
    corr = ((torch.arange(E) * 7 % E) * 1.3 / 8).bfloat16().float()
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    for M in (1, 23, 16384 // top + 5):
        h = P8(randn(M, W, seed=M)).bfloat16().float()
        r, gate = ops.router(on(h), on(w), pad8(E) if shared else -1, on(corr), top, groups, keep, 1.5)
        z = h.double() @ w.double().T
        if shared:
            torch.testing.assert_close(gate.double().cpu(), z[:, pad8(E)], rtol=1e-4, atol=1e-4)
            joint, none = ops.router(on(h), on(w), pad8(E), on(corr), top, groups, keep, 1.5, True)
            assert none is None and joint.place.shape[1] == top + 1 and torch.equal(joint.weights[:, :top], r.weights)
            torch.testing.assert_close(joint.weights[:, top].double().cpu(), O.sigmoid(z[:, pad8(E)]), rtol=1e-4, atol=1e-5)
            assert (joint.place[:, top] >= M * top).all() and int(joint.offsets[E]) == M * top
        else:
            assert gate is None
        want = ops.route(z[:, :pad8(E)].float(), corr, top, groups, keep, 1.5)
        same = (r.weights.cpu().sort(-1).values - want.weights.sort(-1).values).abs().max(-1).values < 1e-4
        assert same.float().mean() > 0.999                       # a choice so close that the order of a sum decides it
        off, place = r.offsets.cpu(), r.place.cpu()
        assert off[-1] == M * top and (place.reshape(-1).sort().values == torch.arange(M * top)).all()
        ids = torch.searchsorted(off, place, right=True) - 1
        torch.testing.assert_close(r.weights.double().cpu(), O.sigmoid(z.gather(1, ids)) * 1.5, rtol=1e-4, atol=1e-5)
        assert (r.token.cpu()[place.long()] == torch.arange(M)[:, None]).all()
    z = ops.linear_fp32(on(h), on(w))
    torch.testing.assert_close(z.double().cpu(), h.double() @ w.double().T, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("M,F,W", [(1, 8, 8), (3, 40, 24), (130, 200, 72), (257, 1000, 328), (300, 136, 128)])
def test_gated_product(run, M, F, W):
    h, w = randn(M, W, seed=1).bfloat16().float(), (randn(2 * F, W, seed=2) * W ** -0.5 * 3).bfloat16().float()
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    out = torch.zeros(M, F + 8, dtype=run[1], device=run[0])
    ops.glu_linear(on(h), on(w), out[:, 8:])
    want = O.silu(h.double() @ w[:F].double().T) * (h.double() @ w[F:].double().T)
    tol = dict(rtol=1e-2, atol=1e-2) if run[1] == torch.bfloat16 else dict(rtol=1e-5, atol=1e-4)
    torch.testing.assert_close(out[:, 8:].double().cpu(), want, **tol)
    assert not out[:, :8].any()


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,F,W,shared", [(3, 2, 10, 20, True), (8, 4, 72, 96, True), (40, 6, 136, 64, False), (4, 1, 300, 200, True), (2, 2, 64, 328, True)])
def test_experts(run, E, top, F, W, shared):
    """Experts with no rows, with a few and with more than a tile; the weighted sum, the shared expert, the norm, the residual."""
    eps, coef = 1e-5, 0.6
    Fp, Wp = pad8(F), pad8(W)
    w_in, w_out = torch.zeros(E, 2, Fp, Wp), torch.zeros(E, Wp, Fp)
    w_in[:, :, :F, :W], w_out[:, :W, :F] = randn(E, 2, F, W, seed=1) * W ** -0.5 * 1.5, randn(E, W, F, seed=2) * F ** -0.5 * 1.5
    w_in, w_out = w_in.bfloat16().float(), w_out.bfloat16().float()
    corr = torch.zeros(E)
    corr[E // 2:] -= 1.1                                  # the second half is hardly ever chosen
    norm = P8(1 + 0.2 * randn(W, seed=3)).bfloat16().float()
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    for M in (1, 5, 150, 700):
        h, z = P8(randn(M, W, seed=M)), randn(M, pad8(E), seed=M + 1)
        r = ops.route(z.to(run[0]), on(corr), top, 1, 1, 1.3)
        rows = ops.expert_down(ops.expert_glu(on(h), on(w_in), r), on(w_out), r)
        sh, sg, x = (randn(*s, seed=M + i).to(run[0]) for i, s in ((2, (M, Wp)), (3, (M, 8)), (4, (M, Wp))))
        sh[:, W:] = 0
        x[:, W:] = 0
        x0, y = x.clone(), torch.zeros(M, Wp, dtype=torch.float64)
        ids = torch.searchsorted(r.offsets.cpu(), r.place.cpu(), right=True) - 1
        for e in range(E):
            f = O.silu(h.double() @ w_in[e, 0].double().T) * (h.double() @ w_in[e, 1].double().T)
            y += (f @ w_out[e].double().T) * (r.weights.cpu().double() * (ids == e)).sum(1)[:, None]
        if shared:
            y += O.sigmoid(sg.cpu().double()[:, :1]) * sh.cpu().double()
        out = ops.moe_norm_add(x, rows, r, sh if shared else None, sg[:, 0] if shared else None, on(norm), coef, W, eps)
        want = coef * O.rms(y[:, :W], eps) * norm[:W].double()
        near((x - x0).cpu()[:, None, :W], want[:, None].float(), run)
        assert out.dtype == run[1] and torch.equal(out.float(), x.to(run[1]).float()) and not x[:, W:].any()


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("n", [8, 42, 200, 2560, 9000])
def test_norm_then_sum(run, n):
    ld, M, eps = pad8(n), 5, 1e-5
    x, y, w = (P8(randn(*s, seed=i)) for i, s in enumerate(((M, n), (M, n), (n,))))
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    for coef, f in ((1.0, 1.0), (0.4, -0.01), (2.0, 30.0)):
        want = x.double()[:, :n] + coef * O.rms(f * y.double()[:, :n], eps) * on(w).double().cpu()[:n]
        xs = x.clone().to(run[0])
        h = ops.norm_add(xs, y.to(run[0]), on(w), coef, n, eps, f)
        torch.testing.assert_close(xs[:, :n].double().cpu(), want, rtol=1e-5, atol=1e-5)
        assert h.dtype == run[1] and torch.equal(h.float(), xs.to(run[1]).float()) and not xs[:, n:].any()
    scaled = ops.rmsnorm_f32(xs, on(w), n, eps, None, 0.3).double().cpu()[:, :n]
    torch.testing.assert_close(scaled, 0.3 * O.rms(xs.double().cpu()[:, :n], eps) * on(w).double().cpu()[:n], atol=1e-5,
                               rtol=1e-2 if run[1] == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("run", RUNS)
def test_token_vectors(run):
    V, d, L, M = 11, 16, 3, 7
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    table, gate, ids = on(randn(V, L * d, seed=1)), on(randn(M, 2 * d, seed=2) * 3), torch.tensor([0, 10, 3, 3, 7, 1, 9])
    for layer in range(L):
        got = ops.gelu_times_token(gate[:, d:], table, ids.to(run[0]), layer * d, V).double().cpu()
        want = O.gelu_tanh(gate[:, d:].double().cpu()) * table.double().cpu()[ids, layer * d:(layer + 1) * d]
        torch.testing.assert_close(got, want, rtol=1e-2 if run[1] == torch.bfloat16 else 1e-5, atol=1e-5)
    for M, d, W in ((1, 8, 8), (37, 24, 72), (300, 128, 200), (1100, 80, 64)):
        h, w, table = randn(M, W, seed=1).bfloat16().float(), (randn(d, W, seed=2) * W ** -0.5 * 2).bfloat16().float(), randn(V, 2 * d, seed=3).bfloat16().float()
        ids = torch.randint(0, V, (M,), generator=torch.Generator().manual_seed(M))
        got = ops.token_gate(on(h), on(w), on(table), ids.to(run[0]), d, V).double().cpu()
        want = O.gelu_tanh(h.double() @ w.double().T) * table.double()[ids, d:]
        torch.testing.assert_close(got, want, rtol=2e-2 if run[1] == torch.bfloat16 else 1e-4, atol=2e-2 if run[1] == torch.bfloat16 else 1e-5)


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
    assert len(got) == len(seen) and clear.sum() > 15
    for i, (a, b) in enumerate(zip(got, seen)):
        e = (a - b)[clear].pow(2).mean().sqrt() / b.std()
        assert e < (0.03 if run[1] == torch.bfloat16 else 2e-5), f"layer {i}: {float(e)}"
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
    cuts = [[T], [2] * (T // 2), [100] + [1] * 110, [17, 64, 65, 63, 1], [16, 1, T - 18, 1], [128, 2, T - 130]]
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
    """Open forget gates, slow channels and a cache: the first token still moves the last logits after hundreds of decoded tokens."""
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
        assert moved > 1e-3 and ((ga[-1] - gb[-1]).double().cpu() - (wa[0][-1] - wb[0][-1])).norm() < 0.05 * moved


def test_scales_of_the_two_mixers():
    """Left and right factors, zero and negative ones among them."""
    for ls, rs in ((0.0, 0.7), (0.9, 0.0), (-0.5, 1.5), (2.0, -0.25)):
        cfg = config(40, 50, [parallel(att(2, 1, 16, 8, rot(16)), 2, 8, 16, 5.0, ls, rs, ff=dense(24)), attention(2, 1, 8, 8, rot(8), ff=moe(4, 2, 8))])
        w = bf16_exact(O.random_weights(cfg, 3))
        seq = toks(30, 50, 1)
        S.close(feed_cuts(engine(build(cfg, w, CPU_RUN)), "a", seq, [21, 1, 8]), O.forward(cfg, w, seq), CPU_RUN)


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
    assert registry.architecture_at(str(tmp_path)).name == "Ruburax"
    assert {n: tuple(t.shape) for n, t in m.named_checkpoint_tensors()} == {n: tuple(s) for n, s in O.shapes(cfg).items()}
    eng = InferenceEngine(InferenceConfig.from_model_config(registry.read_config(str(tmp_path)), num_blocks=16,
                                                            model_path=str(tmp_path), dtype="float32", max_num_sequences=2,
                                                            inference_mode="kv_cache", temperature=0.0)).initialize()
    if eng.device.type == "cpu":
        for (n, a), (n2, b) in zip(m.named_checkpoint_tensors(), eng.model.named_checkpoint_tensors()):
            assert n == n2 and torch.equal(a, b) and torch.equal(a, w[n])
        seq = toks(30, cfg["vocab"])
        S.close(eng.feed([("a", seq)])["a"], O.forward(cfg, w, seq), CPU_RUN)
        # new weights in place, through the engine's update path
        w2 = bf16_exact(O.random_weights(cfg, 9))
        assert eng.load_weights(w2) == len(w2)
        eng.release("a")
        S.close(eng.feed([("a", seq)])["a"], O.forward(cfg, w2, seq), CPU_RUN)


def test_pages_of_shared_keys_are_not_stored_twice():
    cfg = RuburaxConfig.from_dict(ODD)
    m = registry.build_model(cfg, device="meta")
    assert m.kv_layer_shapes() == [None, (2, 24, 16), (1, 16, 24), None, None, None] and m.kv_sources() == [None, None, None, 1, None, 1]
    assert cfg.kv_bytes_per_token() == 2 * (2 * 40 + 40)


def test_bad_checkpoints_and_configs():
    cfg, w = case("odd")
    m = build(cfg, w, CPU_RUN)
    before = m.embed_tokens.clone()
    for change in ({"l0.norm1": None}, {"l9.norm1": torch.zeros(42)}, {"l1.mix.q": torch.zeros(3, 3)}, {"l3.mix.k": torch.zeros(36, 42)}):
        items = {**w, **change, "embed": torch.zeros_like(w["embed"])}
        with pytest.raises(ValueError, match="nothing was loaded"):
            registry.load_slots(m, [(k, v) for k, v in items.items() if v is not None])
        assert torch.equal(m.embed_tokens, before)
    a = att(2, 1, 8, 8, rot(8))
    bad = [([{"type": "other", "mixer": {}}], "unknown type"), ([{"type": "rglru", "mixer": {"width": 8}}], "missing"),
           ([rglru(8, 1, 2, ff={"kind": "sparse"})], "feed-forward kind"), ([rglru(8, 1, 2, ff={"kind": "moe", "expert": {"ff": 8}})], "missing"),
           ([parallel({"heads": 1}, 1, 8, 8, 3.0, 1, 1)], "left mixer"), ([attention(2, 1, 8, 8, rot(8), kv_from=0)], "kv_from 0"),
           ([rglru(8, 1, 2), attention(2, 1, 8, 8, rot(8), kv_from=0)], "kv_from 0"),
           ([{"type": "attention", "mixer": a, "mlp": None}, attention(2, 2, 8, 8, rot(8), kv_from=0)], "differ from those of layer 0")]
    for layers, why in bad:
        with pytest.raises(ValueError, match=why):
            RuburaxConfig.from_dict(config(8, 8, layers))
    with pytest.raises(ValueError, match="missing required"):
        RuburaxConfig.from_dict({"vocab": 8})
    for layers, why in (([attention(3, 2, 8, 8, rot(4))], "do not divide"), ([rglru(9, 2, 2)], "equal blocks"),
                        ([rglru(8, 2, 2, ff=moe(6, 2, 8, (4, 2)))], "equal groups"), ([rglru(8, 2, 2, ff=moe(8, 5, 8, (4, 2)))], "cannot choose"),
                        ([attention(2, 1, 8, 8, rot(10))], "rotary dims")):
        with pytest.raises(ValueError, match=why):
            registry.build_model(RuburaxConfig.from_dict(config(8, 8, copy.deepcopy(layers))), device="cpu")
    for kw in (dict(speculative_enabled=True), dict(kv_cache_dtype="fp8")):
        with pytest.raises(ValueError, match="recurrent state"):
            engine(m, **kw)
    for name in ("ruburax-tiny", "ruburax-0.6b"):
        c = registry.PRESETS[name]
        assert 0 < c.num_active_params() < c.num_params()
