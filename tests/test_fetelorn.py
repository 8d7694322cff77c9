"""Fetelorn through the framework against the plain implementation of ``fetelorn_oracle``: every mechanism alone, whole
prompts, portions, mixed batches, reused pages and slots, long decoding, greedy generation.  The same tests run the
operators' CPU form and, on a GPU, the kernels in true 32-bit and in bf16."""
import json
import random

import pytest
import torch

import fetelorn_oracle as O
from b200fw import ops
from b200fw.infer import InferenceConfig, InferenceEngine
from b200fw.infer.hybrid import build_portions
from b200fw.model import registry
from b200fw.model.fetelorn import FetelornConfig
from b200fw.ops.portions import pad8

GPU = pytest.mark.gpu
RUNS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), id="gpu-f32", marks=GPU),
        pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=GPU)]


def retention(heads, dim, vdim, dims, base=700.0, ff=24):
    return {"type": "retention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims},
                      "decay": [1.0 - 2.0 ** -(2 + 7 * h) for h in range(heads)]}}


def parallel(lh, lg, ld, lv, chunk, far, rh, rg, rd, rv, conv, scale=0.4, ff=24):
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff}, "mixer": {
        "left": {"heads": lh, "kv_heads": lg, "dim": ld, "vdim": lv, "scale": scale, "mask": {"size": chunk}, "bias_max": far},
        "right": {"heads": rh, "kv_heads": rg, "dim": rd, "vdim": rv, "conv": conv}}}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Fetelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# odd sizes on purpose: nothing a multiple of eight, q / k and v sizes apart, groups, partial rotation, missing feed-forwards
ODD = config(42, 67, [retention(3, 20, 12, 14), parallel(6, 2, 12, 20, 24, 20, 4, 2, 22, 10, 3, ff=None),
                      retention(1, 10, 28, 10, ff=None), parallel(5, 1, 9, 7, 37, 50, 3, 3, 8, 17, 1)])
# a parallel layer first, one key head for all queries in both halves, long convolution, chunk of one page
PLAIN = config(64, 96, [parallel(4, 1, 32, 16, 16, 40, 4, 1, 32, 16, 6), retention(2, 32, 32, 32)], eps=1e-3)
# heads as wide as a real model's, chunks across several tiles
WIDE = config(96, 80, [retention(2, 128, 64, 64, ff=40), parallel(4, 2, 128, 96, 150, 100, 2, 1, 128, 64, 4, scale=0.06, ff=40),
                       retention(1, 64, 128, 64, ff=40)])
CONFIGS = {"odd": ODD, "plain": PLAIN, "wide": WIDE}


def bf16_exact(weights):
    return {k: v.bfloat16().float() for k, v in weights.items()}


_cache = {}


def case(name, seed=1):
    if (name, seed) not in _cache:
        _cache[name, seed] = (CONFIGS[name], bf16_exact(O.random_weights(CONFIGS[name], seed)))
    return _cache[name, seed]


def build(cfg, weights, run):
    mc = FetelornConfig.from_dict(cfg, {k: tuple(v.shape) for k, v in weights.items()})
    m = registry.build_model(mc, dtype=run[1], device=run[0])
    registry.load_slots(m, weights.items())
    return m


def engine(model, tokens=640, seqs=4, **kw):
    c = InferenceConfig.from_model_config(model.cfg, num_blocks=tokens // 16, max_num_sequences=seqs,
                                          **{"inference_mode": "kv_cache", "temperature": 0.0, **kw})
    return InferenceEngine(c, model).initialize()


def close(got, want, run, what=""):
    """Difference of logits with their mean taken off, relative to the size of the logits."""
    got, want = got.double().cpu(), want.double().cpu()
    d = (got - got.mean(-1, keepdim=True)) - (want - want.mean(-1, keepdim=True))
    e = (d.pow(2).mean(-1).sqrt() / want.std()).max()
    assert e < (0.06 if run[1] == torch.bfloat16 else 2e-4), f"{what}: {float(e):.5f}"


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
    p, order, place = build_portions(starts, counts, tables, slots, run[1] == torch.float32, dev)
    rows = list(range(sum(counts))) if place is None else place.tolist()
    return p, order, rows, n * pages_each


def steps_of(counts_per_seq):
    """[[portions of sequence 0], ...] -> per step (starts, counts) with every sequence present."""
    for k in range(len(counts_per_seq[0])):
        yield [sum(c[:k]) for c in counts_per_seq], [c[k] for c in counts_per_seq]


def packed(parts, run):
    """Side by side in one matrix, every head padded to eight: parts [(tensor [M, H, d])] -> slices."""
    M = parts[0].shape[0]
    flat = [torch.nn.functional.pad(t, (0, pad8(t.shape[-1]) - t.shape[-1])).reshape(M, -1) for t in parts]
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


CUTS = [[[1, 5, 40, 1, 1], [17, 2, 64, 70, 1], [65, 130, 1, 16, 33]]]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dk,dv,rot", [(3, 20, 12, 14), (2, 128, 64, 64), (1, 8, 136, 8), (2, 64, 128, 0)])
def test_retention(run, H, dk, dv, rot):
    eps, decay, counts = 1e-6, [0.5, 0.97, 0.9995][:H], CUTS[0]
    T = [sum(c) for c in counts]
    data = [[randn(t, H, d, seed=10 * s + i, run=run) for i, d in enumerate((dk, dk, dv, dv))] for s, t in enumerate(T)]
    want = []
    for q, k, v, g in data:
        q, k, v, g = (t.double() for t in (q, k, v, g))
        if rot:
            q, k = O.rotate_half(q, 700.0, rot), O.rotate_half(k, 700.0, rot)
        o = O.rms(O.retention_core(q, k * dk ** -0.5, v, decay), eps)
        want.append(o * O.silu(g))
    state = torch.full((len(T), H, pad8(dk), pad8(dv)), 7.0, device=run[0])     # slots hold another request's leftovers
    turns = ops.rope_turns(700.0, rot, run[0]) if rot else None
    for starts, cnt in steps_of(counts):
        p, order, rows, _ = layout(starts, cnt, run)
        cat = [torch.cat([data[s][i][starts[s]:starts[s] + cnt[s]] for s in order]) for i in range(4)]
        q, k, v, g = packed(cat, run)
        out = torch.full((p.rows, H * pad8(dv)), 9.0, dtype=run[1], device=run[0])
        cs, sn = ops.rope_rows(p.positions, turns) if rot else (None, None)
        ops.retention(q, k, v, g, out, state, p, torch.tensor(decay, device=run[0]), dk, dv, cs, sn, dk ** -0.5, eps)
        got = out.float().cpu().reshape(p.rows, H, -1)[:, :, :dv]
        ref = torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float()
        near(got, ref, run)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,K,strength", [(4, 2, 22, 10, 3, 0.3), (2, 1, 128, 64, 4, 1.0), (3, 3, 8, 136, 1, 8.0),
                                                  (2, 2, 64, 128, 6, 40.0)])
def test_gated_delta(run, H, G, dk, dv, K, strength):
    """Inputs with a repeated key (the write must replace what was stored under it), decays from nearly one to vanishing."""
    eps, counts, s0 = 1e-6, CUTS[0], 100
    T, dkp, dvp = [sum(c) for c in counts], pad8(dk), pad8(dv)
    taps = [randn(n * d, K, seed=s0 + i) for i, (n, d) in enumerate(((G, dk), (G, dk), (H, dv)))]
    A_log, dt, nw = randn(H, seed=1) * 0.5, randn(H, dk, seed=2) - 1, 1 + 0.2 * randn(dv, seed=3)
    A_log, nw, dt = A_log.bfloat16().float(), nw.bfloat16().float(), dt.bfloat16().float()
    data = []
    for s, t in enumerate(T):
        x = [randn(t, n, d, seed=20 * s + i, run=run) for i, (n, d) in enumerate(((G, dk), (G, dk), (H, dv)))]
        x[1][t // 2:] = x[1][t // 2:t // 2 + 1]            # the same key again and again
        data.append(x + [randn(t, H, seed=20 * s + 5, run=run) * 2, randn(t, H, dk, seed=20 * s + 6) * strength,
                         randn(t, H, dv, seed=20 * s + 7)])
    want, of = [], torch.arange(H) // (H // G)
    for q, k, v, b, a, g in data:
        def conv(x, w):
            return O.silu(O.short_conv(x.double().reshape(x.shape[0], -1), w.double())).reshape(x.shape)
        q, k, v = O.unit(conv(q, taps[0])) * dk ** -0.5, O.unit(conv(k, taps[1])), conv(v, taps[2])
        dec = torch.exp(-torch.exp(A_log.double())[None, :, None] * O.softplus(a.double() + dt.double()))
        o = O.delta_core(q[:, of], k[:, of], v, dec, O.sigmoid(b.double()))
        want.append(O.rms(o, eps) * nw.double() * O.sigmoid(g.double()))
    P = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))  # noqa: E731
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    tp = torch.cat([torch.nn.functional.pad(w.reshape(n, d, K), (0, 0, 0, pad8(d) - d)).reshape(-1, K)
                    for w, (n, d) in zip(taps, ((G, dk), (G, dk), (H, dv)))])
    state = torch.full((len(T), H, dkp, dvp), float("inf"), device=run[0])
    conv_state = torch.full((len(T), tp.shape[0], K - 1), float("nan"), device=run[0])
    for starts, cnt in steps_of(counts):
        p, order, rows, _ = layout(starts, cnt, run)
        cat = [torch.cat([data[s][i][starts[s]:starts[s] + cnt[s]] for s in order]) for i in range(6)]
        xq, xk, xv, b = packed(cat[:3] + [cat[3][:, None, :]], run)
        w = xq.shape[1] + xk.shape[1] + xv.shape[1]
        x = torch.as_strided(xq, (p.rows, w), xq.stride(), xq.storage_offset())
        z = torch.cat([P(cat[4], dkp).reshape(p.rows, -1), P(cat[5], dvp).reshape(p.rows, -1)], 1).to(run[0])
        q, k, v, g, beta = ops.delta_inputs(x, on(tp), b[:, :H], z[:, :H * dkp], on(A_log), on(P(dt, dkp).reshape(-1)),
                                            conv_state, p, G, dk, dv, dk ** -0.5)
        out = torch.full((p.rows, H * dvp), 9.0, dtype=run[1], device=run[0])
        ops.gated_delta(q, k, v, g, beta, z[:, H * dkp:], on(P(nw, dvp)), out, state, p, G, dk, dv, eps)
        got = out.float().cpu().reshape(p.rows, H, -1)[:, :, :dv]
        ref = torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float()
        near(got, ref, run)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,chunk", [(6, 2, 12, 20, 24), (5, 1, 9, 7, 37), (4, 2, 128, 96, 150), (4, 1, 96, 128, 128),
                                             (8, 1, 64, 64, 17), (2, 2, 160, 24, 40), (7, 1, 128, 128, 1), (2, 1, 128, 128, 1000)])
def test_chunked_attention(run, H, G, dk, dv, chunk):
    """One loud key per query head at a time: on a page border, first and last of a chunk, just outside of it, the query's own
    token.  A key that is wrongly seen, or missed, takes the whole softmax with it."""
    eps, scale, far, rows_rel = 1e-6, 6.0 / dk, max(chunk // 2, 9), 8
    counts = CUTS[0]
    T = [sum(c) for c in counts]
    rel, sink = randn(rows_rel, H, seed=5).bfloat16().float(), (2.0 + randn(H, seed=6)).bfloat16().float()
    data, want = [], []
    for s, t in enumerate(T):
        q, k, v = randn(t, H, dk, seed=30 * s), randn(t, G, dk, seed=30 * s + 1), randn(t, G, dv, seed=30 * s + 2, run=run)
        r = random.Random(s)
        for i in range(0, t, 3):       # query i matches the key at a border near it
            c0 = i // chunk * chunk
            j = r.choice([c0, c0 - 1, i, i - 1, i // 16 * 16, i // 16 * 16 - 1, min(i, c0 + far), (c0 + i) // 2])
            j = min(max(j, 0), t - 1)
            q[i] = k[j].repeat_interleave(H // G, 0)
        q, k = (x.bfloat16().float() for x in (q, k))
        gate = randn(t, H, seed=30 * s + 3, run=run)
        data.append((q, k, v, gate))
        qn, kn = O.rms(q.double(), eps), O.rms(k.double(), eps)
        o = O.chunk_attention_core(qn, kn, v.double(), scale, chunk, rel.double(), far, sink.double())
        want.append(o * O.sigmoid(gate.double())[:, :, None])
    bucket = ops.distance_buckets(rows_rel, far, min(chunk, far + 1), run[0])
    on = lambda t: t.to(run[1]).to(run[0])  # noqa: E731
    kc = vc = None
    for starts, cnt in steps_of(counts):
        p, order, rows, pages = layout(starts, cnt, run)
        if kc is None:
            kc = torch.full((pages, 16, G, pad8(dk)), float("nan"), dtype=run[1], device=run[0])
            vc = torch.full((pages, 16, G, pad8(dv)), float("nan"), dtype=run[1], device=run[0])
            if run[1] == torch.bfloat16:      # the tiled kernel may read, masked, what a page holds past its sequence
                kc.fill_(3.0), vc.fill_(3.0)
        cat = [torch.cat([data[s][i][starts[s]:starts[s] + cnt[s]] for s in order]) for i in range(4)]
        q, k, v, g = packed(cat[:3] + [cat[3][:, None, :]], run)
        qn = ops.qk_norm_store(q, k, v, kc, vc, p, H, dk, True, eps)
        out = torch.full((p.rows, H * pad8(dv)), 9.0, dtype=run[1], device=run[0])
        ops.paged_attention(qn, kc, vc, out, p, H, scale, chunk, on(rel), bucket, on(sink), g[:, :H])
        got = out.float().cpu().reshape(p.rows, H, -1)[:, :, :dv]
        ref = torch.cat([want[s][starts[s]:starts[s] + cnt[s]] for s in order]).float()
        near(got, ref, run)


def test_distance_buckets():
    b = ops.distance_buckets(12, 90, 200).tolist()
    assert b == [min(O.distance_bucket(n, 12, 90), 11) for n in range(200)]
    assert b[:6] == list(range(6)) and b[90] == b[199] == 11
    # a distance exactly on an edge belongs to the upper bucket: 4 * (64 / 4)^(1/2) = 16
    assert ops.distance_buckets(8, 64, 17).tolist()[15:] == [5, 6]


@pytest.mark.parametrize("run", RUNS)
def test_rope_far_positions(run):
    pos = torch.tensor([0, 1, 511, 123456, 10 ** 6 + 7], dtype=torch.int32, device=run[0])
    cs, sn = ops.rope_rows(pos, ops.rope_turns(1e4, 6, run[0]))
    a = pos.cpu().double()[:, None] * torch.tensor([1e4 ** (-2 * i / 6) for i in range(3)], dtype=torch.float64)
    torch.testing.assert_close(cs.cpu().double(), a.cos(), rtol=0, atol=2e-6)
    torch.testing.assert_close(sn.cpu().double(), a.sin(), rtol=0, atol=2e-6)


# ---- the whole model ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_layers_and_logits(run, name):
    cfg, w = case(name)
    seq, seen = toks(45, cfg["vocab"]), []
    want = O.forward(cfg, w, seq, seen)
    m = build(cfg, w, run)
    eng = engine(m)
    eng.kv.allocate_for_sequence("a", 45)
    ctx, got = eng.runner.prepare_prefill(["a"], [0], [45]), []
    out = eng.runner.forward(torch.tensor(seq, device=run[0]), ctx, all_rows=True,
                             on_layer=lambda i, x: got.append(x[:, :cfg["width"]].double().cpu().clone()))
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
    want = O.forward(cfg, w, seq)
    eng = engine(build(cfg, w, run))
    r = random.Random(5)
    chunks = [l["mixer"]["left"]["mask"]["size"] for l in cfg["layers"] if l["type"] == "parallel"]
    cuts = [[T], [2] * (T // 2), [100] + [1] * 110, [17, 64, 65, 63, 1], [chunks[0], 1, T - chunks[0] - 2, 1],
            [chunks[-1] - 1, 2, T - chunks[-1] - 1]]
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
    want = [O.forward(cfg, w, s) for s in seqs]
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
    """A retention head that forgets nothing for hundreds of tokens: the first token still moves the last logits."""
    cfg, w = case("plain")
    T = 400
    a, b = toks(T, cfg["vocab"], 8), toks(T, cfg["vocab"], 8)
    b[0] = (b[0] + 1) % cfg["vocab"]
    eng = engine(build(cfg, w, run))
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    ga = feed_cuts(eng, "a", a, [5] + [1] * (T - 5))
    close(ga, wa, run)
    if run[1] == torch.float32:
        gb = feed_cuts(eng, "b", b, [T])
        moved = (wa[-1] - wb[-1]).norm()
        assert moved > 1e-3 and ((ga[-1] - gb[-1]).double().cpu() - (wa[-1] - wb[-1])).norm() < 0.05 * moved


def test_feed_refuses_what_does_not_fit():
    cfg, w = case("plain")
    eng = engine(build(cfg, w, ("cpu", torch.float32)), tokens=64, seqs=2)
    eng.feed([("a", toks(20, 96))])
    with pytest.raises(RuntimeError, match="exhausted"):
        eng.feed([("a", toks(2, 96)), ("b", toks(40, 96))])
    assert eng.kv.get_seq_token_count("a") == 20 and eng.kv.pool.num_used_blocks == 2 and eng.kv.state.num_free_slots == 1
    eng.feed([("b", [1])])
    with pytest.raises(RuntimeError, match="slot"):
        eng.feed([("c", [1])])
    for bad in ([("a", [])], [("a", [96])], [("a", [-1])], [("a", [1]), ("a", [2])]):
        with pytest.raises(ValueError):
            eng.feed(bad)


# ---- generation through the scheduler -------------------------------------------------------------------------------
def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(O.forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


F32_RUNS = [RUNS[0], RUNS[1]]


@pytest.mark.parametrize("run", F32_RUNS)
def test_greedy_generation(run):
    cfg, w = case("odd")
    prompts = [toks(n, cfg["vocab"], 60 + n) for n in (5, 41, 1, 70, 23, 30)]
    want = [greedy(cfg, w, p, 12) for p in prompts]
    m = build(cfg, w, run)
    # more requests than slots, chunked prompts beside decoding ones, too few pages for all (preemption)
    for kw in (dict(seqs=3, chunk_size=16, max_prefill_tokens=32), dict(seqs=6, tokens=192, chunk_size=24),
               dict(seqs=6, enable_cuda_graph=True), dict(seqs=4, async_decode="force", chunk_size=32)):
        eng = engine(m, **kw)
        assert eng.generate(prompts, max_tokens=12) == want, kw
        assert eng.kv.pool.num_used_blocks == 0 and eng.kv.state.num_free_slots == kw["seqs"], kw
    assert engine(m, inference_mode="eager").generate(prompts[:2], max_tokens=4) == [x[:4] for x in want[:2]]


@pytest.mark.gpu
def test_graph_decoding_matches_plain_bf16():
    cfg, w = case("wide")
    m = build(cfg, w, ("cuda", torch.bfloat16))
    prompts = [toks(n, cfg["vocab"], 80 + n) for n in (40, 3, 130, 64, 77)]
    outs = [engine(m, tokens=1600, seqs=5, enable_cuda_graph=g).generate(prompts, max_tokens=24) for g in (False, True)]
    assert outs[0] == outs[1]


@pytest.mark.gpu
def test_host_running_ahead_of_the_gpu():
    """Chunks of a long prompt read nothing back, so the host queues many steps ahead: the staged row layouts of earlier steps
    must survive until their copies have run."""
    cfg, w = case("wide")
    m = build(cfg, w, ("cuda", torch.bfloat16))
    prompt = toks(3000, cfg["vocab"], 99)
    outs = []
    for sync in (True, False):
        eng = engine(m, tokens=3200, seqs=2, chunk_size=17, max_prefill_tokens=17, adaptive_chunking=False)
        r = eng.add_request("a", prompt, 6)
        if not sync:
            torch.cuda._sleep(int(2e8))          # about 0.1 s of GPU time in front of the first step
        while eng.has_pending():
            eng.step()
            if sync:
                torch.cuda.synchronize()
        outs.append(r.output_tokens)
    assert outs[0] == outs[1]


def test_stop_and_abort():
    cfg, w = case("odd")
    m = build(cfg, w, ("cpu", torch.float32))
    p = toks(20, cfg["vocab"], 1)
    full = greedy(cfg, w, p, 8)
    eng = engine(m, eos_token_id=full[3])
    assert eng.generate([p], max_tokens=8)[0] == full[:full.index(full[3]) + 1]
    r = eng.add_request("x", p, 50)          # two steps: the prompt and one more token, before the stop token
    for _ in range(2):
        eng.step()
    assert eng.abort_request("x") and r.output_tokens == full[:len(r.output_tokens)]
    assert eng.kv.pool.num_used_blocks == 0 and eng.kv.state.num_free_slots == 4


# ---- loading ----------------------------------------------------------------------------------------------------------
def test_checkpoint_round_trip_and_registry(tmp_path):
    cfg, w = case("odd")
    m = build(cfg, w, ("cpu", torch.float32))
    registry.save_checkpoint(m, str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    assert registry.architecture_at(str(tmp_path)).name == "Fetelorn"
    eng = InferenceEngine(InferenceConfig.from_model_config(registry.read_config(str(tmp_path)), num_blocks=16,
                                                            model_path=str(tmp_path), dtype="float32", max_num_sequences=2,
                                                            inference_mode="kv_cache", temperature=0.0)).initialize()
    if eng.device.type == "cpu":
        for (n, a), (n2, b) in zip(m.named_checkpoint_tensors(), eng.model.named_checkpoint_tensors()):
            assert n == n2 and torch.equal(a, b)
        seq = toks(30, cfg["vocab"])
        close(eng.feed([("a", seq)])["a"], O.forward(cfg, w, seq), ("cpu", torch.float32))
        # new weights in place, through the engine's update path
        w2 = bf16_exact(O.random_weights(cfg, 9))
        assert eng.load_weights(w2) == len(w2)
        eng.release("a")
        close(eng.feed([("a", seq)])["a"], O.forward(cfg, w2, seq), ("cpu", torch.float32))


def test_bad_checkpoints_and_configs(tmp_path):
    cfg, w = case("odd")
    m = build(cfg, w, ("cpu", torch.float32))
    before = m.embed_tokens.clone()
    for change in ({"l0.norm1": None}, {"l9.norm1": torch.zeros(42)}, {"l0.mix.q": torch.zeros(3, 3)}):
        items = {**w, **change, "embed": torch.zeros_like(w["embed"])}
        with pytest.raises(ValueError, match="nothing was loaded"):
            registry.load_slots(m, [(k, v) for k, v in items.items() if v is not None])
        assert torch.equal(m.embed_tokens, before)
    with pytest.raises(ValueError, match="unknown type"):
        FetelornConfig.from_dict(config(8, 8, [{"type": "other", "mixer": {}}]))
    with pytest.raises(ValueError, match="missing required"):
        FetelornConfig.from_dict({"vocab": 8})
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.read_config(str(tmp_path))
    with pytest.raises(ValueError, match="recurrent state"):
        engine(m, speculative_enabled=True)
    with pytest.raises(ValueError, match="recurrent state"):
        engine(m, kv_cache_dtype="fp8")
    eng = engine(m, enable_prefix_caching=True)
    assert eng.prefix_cache is None
    for name in ("fetelorn-tiny", "fetelorn-0.6b"):
        assert registry.PRESETS[name].num_params() > 0


# ---- kernels the model leans on -----------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("M,N,K", [(1, 8, 8), (3, 40, 24), (130, 200, 72), (257, 1000, 640)])
def test_gemm_32bit_and_fp32_outputs(M, N, K):
    a, b = torch.randn(M, K, device="cuda"), torch.randn(N, K, device="cuda")
    c = torch.randn(M, N, device="cuda")
    want = a.double() @ b.double().t()
    torch.testing.assert_close(ops.gemm(a, b).double(), want, rtol=1e-5, atol=1e-4)
    torch.testing.assert_close(ops.gemm(a, b, out=c.clone(), accumulate=True).double(), want + c.double(), rtol=1e-5, atol=1e-4)
    ah, bh = a.bfloat16(), b.bfloat16()
    want = ah.double() @ bh.double().t()
    got = ops.gemm(ah, bh, out=torch.empty(M, N, device="cuda"))
    torch.testing.assert_close(got.double(), want, rtol=1e-4, atol=1e-3)
    got = ops.gemm(ah, bh, out=c.clone(), accumulate=True)
    torch.testing.assert_close(got.double(), want + c.double(), rtol=1e-4, atol=1e-3)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("n", [8, 42, 200, 9000])
def test_residual_ops(run, n):
    ld, M, eps = pad8(n), 5, 1e-5
    x, a, b = (torch.nn.functional.pad(randn(M, n, seed=i), (0, ld - n)) for i in (1, 2, 3))
    wa, wb, wn = (torch.nn.functional.pad(1 + 0.1 * randn(n, seed=i), (0, ld - n)).to(run[1]).to(run[0]) for i in (4, 5, 6))
    d = lambda t: t.to(run[0])  # noqa: E731
    rows = torch.tensor([3, 0, 3], device=run[0])
    h = ops.rmsnorm_f32(d(x), wn, n, eps, rows)
    want = O.rms(x[rows.cpu(), :n].double(), eps) * wn[:n].double().cpu()
    t = dict(rtol=1e-2, atol=1e-2) if run[1] == torch.bfloat16 else dict(rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(h[:, :n].double().cpu(), want, **t)
    assert not h[:, n:].any()
    y = d(x).clone()
    h = ops.merge_norm_add(y, d(a), d(b), wa, wb, 0.5, n, eps, wn)
    s = x[:, :n].double() + 0.5 * (O.rms(a[:, :n].double(), eps) * wa[:n].double().cpu() + O.rms(b[:, :n].double(), eps) * wb[:n].double().cpu())
    torch.testing.assert_close(y[:, :n].double().cpu(), s, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(h[:, :n].double().cpu(), O.rms(s, eps) * wn[:n].double().cpu(), **t)
    assert not h[:, n:].any() and ops.merge_norm_add(y, d(a), d(b), wa, wb, 0.5, n, eps) is None
    gu = torch.cat([a, b], 1).to(run[1]).to(run[0])
    out = torch.empty(M, ld, dtype=run[1], device=run[0])
    ops.glu(gu[:, :ld], gu[:, ld:], out)
    g, u = gu[:, :ld].double().cpu(), gu[:, ld:].double().cpu()
    torch.testing.assert_close(out.double().cpu(), O.silu(g) * u, **t)
