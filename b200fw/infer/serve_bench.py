"""Serving throughput of a model preset (prefill and decode through the engine) and the rooflines of its kernels.

Random weights, seeded synthetic prompts.  Phases are timed with CUDA events around engine steps; kernels one by one, with the
L2 cache flushed before every launch."""
from __future__ import annotations

import random
from typing import Callable, Dict, List, Optional, Tuple

import torch

from .. import _native as nv
from .. import ops
from ..model.registry import PRESETS, build_model
from ..obs.profilers import measured_peaks
from ..ops.portions import pad8
from .config import InferenceConfig
from .engine import InferenceEngine
from .hybrid import build_portions

DEV = "cuda"


def _prompts(n: int, length: int, vocab: int, seed: int = 0) -> List[List[int]]:
    r = random.Random(seed)
    return [[r.randrange(3, vocab) for _ in range(length)] for _ in range(n)]


def throughput(preset: str, batch: int = 256, prompt: int = 1024, new_tokens: int = 64, budget: int = 8192) -> Dict:
    """``batch`` requests of ``prompt`` tokens, ``new_tokens`` each: tokens/s of the prompt phase and of the decode phase, and
    the whole call from pinned host ids to host ids."""
    mc = PRESETS[preset]
    model = build_model(mc, dtype=torch.bfloat16, device=torch.device(DEV))
    model.init_weights(0)
    for p in model.parameters():
        p.requires_grad_(False)
    warmup = -(-batch * prompt // budget) + 4       # long enough that the whole batch decodes together
    blocks = batch * (-(-(prompt + max(new_tokens, warmup) + 2) // 16) + 1) + 64
    eng = InferenceEngine(InferenceConfig.from_model_config(
        mc, num_blocks=blocks, inference_mode="kv_cache", max_num_batched_tokens=budget + batch, max_prefill_tokens=budget,
        chunk_size=2048, max_num_sequences=batch, enable_cuda_graph=True, temperature=0.0, eos_token_id=None,
        adaptive_chunking=False), model).initialize()
    eng.generate(_prompts(batch, prompt, mc.vocab_size, 1), warmup)           # allocator, graphs, tensor maps
    eng.generate(_prompts(batch, prompt, mc.vocab_size, 2), warmup)           # capturing the graphs gave the allocator's memory back
    out = {"model": preset, "params": mc.num_params(), "params_per_token": getattr(mc, "num_active_params", mc.num_params)(), "batch": batch, "prompt": prompt, "new_tokens": new_tokens}
    for i, p in enumerate(_prompts(batch, prompt, mc.vocab_size)):
        eng.add_request(f"r{i}", p, new_tokens + 1)
    ev = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
    launches = nv.launch_count
    torch.cuda.synchronize()
    ev[0].record()
    while any(r.num_generated_tokens == 0 for r in eng.requests.values()):
        eng.step()
    ev[1].record()
    before = sum(r.num_generated_tokens for r in eng.requests.values())
    steps = 0
    while eng.has_pending():
        eng.step()
        steps += 1
    ev[2].record()
    torch.cuda.synchronize()
    pre, dec = ev[0].elapsed_time(ev[1]), ev[1].elapsed_time(ev[2])
    made = batch * (new_tokens + 1)
    out.update(prefill_tokens_per_s=batch * prompt / (pre * 1e-3), decode_tokens_per_s=(made - before) / (dec * 1e-3),
               decode_ms_per_step=dec / max(1, steps), end_to_end_tokens_per_s=made / ((pre + dec) * 1e-3),
               gpu_launches=nv.launch_count - launches, device_status=nv.read_status())
    del eng, model
    torch.cuda.empty_cache()
    return out


def prefill_once(preset: str, lengths: List[int], iters: int = 5) -> Dict:
    """One forward pass over whole prompts (no scheduler): tokens/s by CUDA events."""
    mc = PRESETS[preset]
    model = build_model(mc, dtype=torch.bfloat16, device=torch.device(DEV))
    model.init_weights(0)
    for p in model.parameters():
        p.requires_grad_(False)
    eng = InferenceEngine(InferenceConfig.from_model_config(
        mc, num_blocks=sum(-(-n // 16) for n in lengths) + 8, inference_mode="kv_cache", max_num_sequences=len(lengths)),
        model).initialize()
    for i, n in enumerate(lengths):
        eng.kv.allocate_for_sequence(i, n)
    ids = torch.tensor([t for n in lengths for t in _prompts(1, n, mc.vocab_size)[0]], device=DEV)
    ctx = eng.runner.prepare_prefill(list(range(len(lengths))), [0] * len(lengths), lengths)
    for _ in range(3):
        eng.runner.forward(ids, ctx)
    s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    s.record()
    for _ in range(iters):
        eng.runner.forward(ids, ctx)
    e.record()
    torch.cuda.synchronize()
    ms = s.elapsed_time(e) / iters
    return {"model": preset, "lengths": lengths, "ms": ms, "tokens_per_s": sum(lengths) / (ms * 1e-3),
            "device_status": nv.read_status()}


# ---- kernels ---------------------------------------------------------------------------------------------------------
class _Timer:
    def __init__(self, iters: int = 10):
        self.iters, self.flush = iters, torch.empty(256 << 20, dtype=torch.uint8, device=DEV)
        self.peaks = measured_peaks()
        self.rows: Dict[str, Dict] = {}

    def __call__(self, name: str, fn: Callable[[], None], bytes_: float, flops: float = 0.0) -> None:
        for _ in range(3):
            fn()
        ms = []
        for _ in range(self.iters):
            self.flush.zero_()
            s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            s.record()
            fn()
            e.record()
            torch.cuda.synchronize()
            ms.append(s.elapsed_time(e))
        t = sorted(ms)[len(ms) // 2]
        floor = max(bytes_ / (self.peaks["hbm_gbs"] * 1e9), flops / (self.peaks["bf16_tflops"] * 1e12)) * 1e3
        self.rows[name] = {"us": round(t * 1e3, 1), "roofline_us": round(floor * 1e3, 1), "of_measured": round(floor / t, 3)}


def _bf(*shape):
    return torch.randn(*shape, device=DEV).to(torch.bfloat16) * 0.5


def _gemm(t: _Timer, name, M, N, K, out32=False, acc=False, residual=False):
    a, w = _bf(M, K), _bf(N, K)
    o = torch.zeros(M, N, device=DEV, dtype=torch.float32 if out32 else torch.bfloat16)
    r = _bf(M, N) if residual else None
    by = 2 * (M * K + N * K) + M * N * (4 if out32 else 2) * (2 if acc else 1) + (2 * M * N if residual else 0)
    t(name, lambda: ops.gemm(a, w, out=o, accumulate=acc, residual=r), by, 2.0 * M * N * K)


def _layout(lengths: Optional[List[int]], batch: int, ctx: int):
    if lengths is None:
        starts, counts = [ctx - 1] * batch, [1] * batch
    else:
        starts, counts = [0] * len(lengths), list(lengths)
    need = [-(-(s + c) // 16) for s, c in zip(starts, counts)]
    ids, tables = torch.randperm(sum(need)).tolist(), []
    for n in need:
        tables.append(ids[:n])
        ids = ids[n:]
    p, _, _ = build_portions(starts, counts, tables, list(range(len(counts))), False,
                             lambda a: torch.from_numpy(a).to(DEV))
    return p, sum(need), starts, counts


def fetelorn_kernels(preset: str, lengths: Optional[List[int]] = None, batch: int = 256, ctx: int = 1024) -> Dict:
    """Every kernel of a layer at the preset's sizes: whole prompts of ``lengths`` tokens, or one decoded token for each of
    ``batch`` sequences at ``ctx`` tokens."""
    mc, t = PRESETS[preset], _Timer()
    W, V = mc.hidden_size, mc.vocab_size
    ret = next(l for l in mc.layers if l["type"] == "retention")
    par = next(l for l in mc.layers if l["type"] == "parallel")
    p, pages, starts, counts = _layout(lengths, batch, ctx)
    M, n = p.rows, p.nseq
    x, w = torch.randn(M, W, device=DEV), _bf(W)
    t("rmsnorm_f32", lambda: ops.rmsnorm_f32(x, w, W, 1e-6), M * W * 6)
    m, ff = ret["mixer"], ret["mlp"]["ff"]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    nin = H * 2 * (dk + dv) + 2 * ff
    _gemm(t, "gemm in (retention + ff)", M, nin, W)
    _gemm(t, "gemm out (retention + ff), += fp32", M, W, H * dv + ff, True, True)
    y, buf = _bf(M, nin), _bf(M, H * dv + ff)
    o = H * 2 * (dk + dv)
    t("glu", lambda: ops.glu(y[:, o:o + ff], y[:, o + ff:], buf[:, H * dv:]), M * ff * 6)
    turns = ops.rope_turns(1e4, m["rot"]["dims"], DEV)
    t("rope_rows", lambda: ops.rope_rows(p.positions, turns), M * m["rot"]["dims"] * 4)
    cs, sn = ops.rope_rows(p.positions, turns)
    S, dec = torch.zeros(n, H, dk, dv, device=DEV), torch.tensor(m["decay"], device=DEV)
    c = [0, H * dk, 2 * H * dk, 2 * H * dk + H * dv, o]
    flops = M * H * (2.0 * 64 * (dk + dv) / 2 + 4.0 * dk * dv)          # chunked form, 64-token chunks
    state = n * H * dk * dv * 4 * (1 if lengths else 2)
    t("retention", lambda: ops.retention(*(y[:, c[i]:c[i + 1]] for i in range(4)), buf[:, :H * dv], S, p, dec, dk, dv, cs, sn,
                                         dk ** -0.5, 1e-6), M * H * (2 * dk + 3 * dv) * 2 + state, flops if lengths else 0)
    a, b, r = par["mixer"]["left"], par["mixer"]["right"], mc.ranks[mc.layers.index(par)]
    ff = par["mlp"]["ff"]
    lq, lk, lv = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
    rk, rv = b["kv_heads"] * b["dim"], b["heads"] * b["vdim"]
    nin = lq + lk + lv + pad8(a["heads"]) + 2 * rk + rv + pad8(b["heads"]) + r["decay_rank"] + r["gate_rank"] + 2 * ff
    _gemm(t, "gemm in (parallel + ff)", M, nin, W)
    kc, vc = _bf(pages, 16, a["kv_heads"], a["dim"]), _bf(pages, 16, a["kv_heads"], a["vdim"])
    yy, g = _bf(M, lq + lk + lv), _bf(M, a["heads"])
    t("qk_norm_store", lambda: ops.qk_norm_store(yy[:, :lq], yy[:, lq:lq + lk], yy[:, lq + lk:], kc, vc, p, a["heads"], a["dim"],
                                                 True, 1e-6), M * (lq + lk + lv) * 4)
    q = ops.qk_norm_store(yy[:, :lq], yy[:, lq:lq + lk], yy[:, lq + lk:], kc, vc, p, a["heads"], a["dim"], True, 1e-6)
    rel, sink = _bf(r["bias_rows"], a["heads"]), _bf(a["heads"])
    chunk = a["mask"]["size"]
    bucket = ops.distance_buckets(r["bias_rows"], a["bias_max"], min(chunk, a["bias_max"] + 1), DEV)
    att = _bf(M, a["heads"] * a["vdim"])
    seen = 0                                                             # query-key pairs
    for s, k in zip(starts, counts):
        seen += sum((i % chunk) + 1 for i in range(s, s + k))
    by = M * (lq + a["heads"] * a["vdim"]) * 2 + (seen if lengths is None else M) * (lk + lv) * 2
    t("paged_attention", lambda: ops.paged_attention(q, kc, vc, att, p, a["heads"], a["scale"], chunk, rel, bucket, sink, g), by,
      2.0 * seen * a["heads"] * (a["dim"] + a["vdim"]))
    _gemm(t, "gemm left o (fp32)", M, W, a["heads"] * a["vdim"], True)
    low = r["decay_rank"] + r["gate_rank"]
    H, G, dk, dv = b["heads"], b["kv_heads"], b["dim"], b["vdim"]
    _gemm(t, "gemm low-rank second (fp32)", M, H * (dk + dv), low, True)
    C = 2 * G * dk + H * dv
    xx, taps, bb, z = _bf(M, C + 8), _bf(C, b["conv"]), None, torch.randn(M, H * (dk + dv), device=DEV)
    bb = xx[:, C:C + H] if H <= 8 else _bf(M, C + 8)[:, :H]
    A, dt, nw = _bf(H), _bf(H * dk), _bf(dv)
    conv, S = torch.zeros(n, C, b["conv"] - 1, device=DEV), torch.zeros(n, H, dk, dv, device=DEV)
    args = (xx[:, :C], taps, bb, z[:, :H * dk], A, dt, conv, p, G, dk, dv, dk ** -0.5)
    outs = ops.delta_inputs(*args)
    io = sum(t_.numel() * t_.element_size() for t_ in outs)
    t("delta_inputs", lambda: ops.delta_inputs(*args), M * (C * 2 + H * dk * 4 + H * 2) + io)
    out = _bf(M, H * dv)
    flops = M * H * (2.0 * 64 * (2 * dk + 2 * dv) / 2 + 6.0 * dk * dv)
    state = n * H * dk * dv * 4 * (1 if lengths else 2)
    t("gated_delta", lambda: ops.gated_delta(*outs, z[:, H * dk:], nw, out, S, p, G, dk, dv, 1e-6),
      io + M * H * dv * (4 + 2) + state, flops if lengths else 0)
    _gemm(t, "gemm right o (fp32)", M, W, H * dv, True)
    _gemm(t, "gemm down, += fp32", M, W, ff, True, True)
    l32, r32 = torch.randn(M, W, device=DEV), torch.randn(M, W, device=DEV)
    t("merge_norm_add", lambda: ops.merge_norm_add(x, l32, r32, w, w, 0.5, W, 1e-6, w), M * W * (16 + 2))
    if lengths is None:
        _gemm(t, "gemm logits (fp32)", M, V, W, True)
    del t.flush
    return t.rows


def sotazen_kernels(preset: str, lengths: Optional[List[int]] = None, batch: int = 256, ctx: int = 1024) -> Dict:
    """The same for the differential / latent / lightning decoder."""
    mc, t = PRESETS[preset], _Timer()
    W, V, eps = mc.hidden_size, mc.vocab_size, mc.rms_norm_eps
    kinds = {k: next(l for l in mc.layers if l["type"] == k) for k in ("lightning", "attention", "latent_attention")}
    ff = kinds["lightning"]["mlp"]["ff"]
    p, pages, starts, counts = _layout(lengths, batch, ctx)
    M, n = p.rows, p.nseq
    x, y32, w, h = torch.randn(M, W, device=DEV), torch.randn(M, W, device=DEV), _bf(W), _bf(M, W)
    t("post_norm", lambda: ops.post_norm(x, y32, w, 1.5, W, eps), M * W * 14)

    def act(name, N, cols, kind):
        wt = _bf(N, W)
        t(name, lambda: ops.linear_act(h, wt, kind, cols), 2 * (M * W + N * W + M * N), 2.0 * M * N * W)
    act("gemm up, relu^2", ff, ff, "relu2")
    _gemm(t, "gemm down (fp32)", M, W, ff, True)

    m = kinds["lightning"]["mixer"]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    c = [0, H * dk, 2 * H * dk, 2 * H * dk + H * dv, 2 * H * (dk + dv)]
    act("gemm in (lightning), silu", c[4], c[3], "silu")
    y, out = _bf(M, c[4]), _bf(M, H * dv)
    S, dec, ss = torch.zeros(n, H, dk, dv, device=DEV), torch.tensor(m["decay"], device=DEV), torch.empty(M, H, device=DEV)
    nw = _bf(H * dv)
    flops = M * H * (2.0 * 64 * (dk + dv) / 2 + 4.0 * dk * dv)
    state = n * H * dk * dv * 4 * (1 if lengths else 2)
    t("lightning", lambda: ops.retention(*(y[:, c[i]:c[i + 1]] for i in range(4)), out, S, p, dec, dk, dv, None, None, 1.0, eps, nw, ss),
      M * H * (2 * dk + 3 * dv) * 2 + state, flops if lengths else 0)
    _gemm(t, "gemm lightning o (fp32)", M, W, H * dv, True)

    a = kinds["attention"]["mixer"]
    H, G, dk, dv, win = a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["mask"]["size"]
    lq, lk, lv = 2 * H * dk, 2 * G * dk, G * dv
    _gemm(t, "gemm in (differential)", M, lq + lk + lv + H * dv, W)
    kc, vc = _bf(pages, 16, 2 * G, dk), _bf(pages, 16, G, dv)
    yy, wd, bias = _bf(M, lq + lk + lv + H * dv), _bf(dk), _bf(lq + lk + lv)
    cs, sn = ops.rope_rows(p.positions, ops.rope_turns(1e4, a["rot"]["dims"], DEV))

    def store():
        return ops.qk_norm_store(yy[:, :lq], yy[:, lq:lq + lk], yy[:, lq + lk:lq + lk + lv], kc, vc, p, 2 * H, dk, True, eps, wd, wd,
                                 bias, cs, sn)
    t("qk_norm_store (bias, rotation)", store, M * ((lq + lk + lv) * 4 + a["rot"]["dims"] * 4))
    q, lam, gate, out = store(), _bf(4, dk), yy[:, lq + lk + lv:], _bf(M, H * dv)
    seen = sum(min(i + 1, win) for s, k in zip(starts, counts) for i in range(s, s + k))          # query-key pairs
    t("differential_attention", lambda: ops.differential_attention(q, kc, vc, out, p, H, a["scale"], lam, a["diff"], dv, eps, gate, win,
                                                                   a["softcap"]),
      M * (lq + 2 * H * dv) * 2 + (seen if lengths is None else M) * (lk + lv) * 2, 2.0 * seen * 2 * H * (dk + dv))
    _gemm(t, "gemm differential o (fp32)", M, W, H * dv, True)

    b = kinds["latent_attention"]["mixer"]
    H, d, r, dv, C = b["heads"], b["dim"], b["rot_dim"], b["vdim"], b["kv_rank"]
    dq, R = d + r, C + r
    _gemm(t, "gemm in (latent)", M, H * dq + R, W)
    yy, pg = _bf(M, H * dq + R), _bf(pages, 16, 1, R)
    cs, sn = ops.rope_rows(p.positions, ops.rope_turns(1e4, r, DEV))
    wc, w_key, w_value, sink, out = _bf(C), _bf(H, dq, R), _bf(H, dv, C), _bf(H), _bf(M, H * dv)
    q, cc, kr = yy[:, :H * dq], yy[:, H * dq:H * dq + C], yy[:, H * dq + C:]
    t("latent_store", lambda: ops.latent_store(q, cc, kr, pg, p, H, d, C, r, wc, cs, sn, eps), M * (H * r * 4 + R * 4 + r * 4))
    pairs = sum((s + k) * (s + k + 1) / 2 - s * (s + 1) / 2 for s, k in zip(starts, counts))
    if lengths is None:
        ql, ol = _bf(M, H * R), _bf(M, H * C)
        t("head_linear (queries to latent)", lambda: ops.head_linear(q, w_key, ql, True), (M * H * (dq + R) + H * dq * R) * 2)
        t("latent_rows", lambda: ops.latent_rows(ql, pg, ol, p, H, C, b["scale"], sink), (pairs * R + M * H * (R + C)) * 2,
          2.0 * pairs * H * (R + C))
        t("head_linear (latent to values)", lambda: ops.head_linear(ol, w_value, out), (M * H * (dv + C) + H * dv * C) * 2)
    else:
        _gemm(t, "gemm keys from latents", M, H * dq, R)
        _gemm(t, "gemm values from latents", M, H * dv, C)
    t("latent_attention", lambda: ops.latent_attention(q, pg, out, p, w_key, w_value, b["scale"], sink),
      M * H * (dq + dv) * 2 + (pairs if lengths is None else M) * R * 2,
      2.0 * pairs * H * (R + C) if lengths is None else 2.0 * (pairs * H * (dq + dv) + M * H * (dq * R + dv * C)))
    if lengths is not None:
        from ..ops import latent
        k, v = _bf(pages * 16, H * dq), _bf(pages * 16, H * dv)
        t("latent prompt attention alone", lambda: latent.expanded_attention(q, k, v, out, p, H, dq, dv, b["scale"], sink, 0, n, p.context().tables),
          M * H * (dq + dv) * 4, 2.0 * pairs * H * (dq + dv))
        rows = torch.empty(pages * 16, R, device=DEV, dtype=torch.bfloat16)
        t("latent_gather", lambda: latent.gather(pg, p.context().pages, rows), rows.numel() * 4)
    _gemm(t, "gemm latent o (fp32)", M, W, H * dv, True)
    if lengths is None:
        _gemm(t, "gemm logits (fp32)", M, V, W, True)
    del t.flush
    return t.rows


def ruburax_kernels(preset: str, lengths: Optional[List[int]] = None, batch: int = 256, ctx: int = 1024) -> Dict:
    """The same for the attention / parallel / gated-recurrence decoder with experts."""
    mc, t = PRESETS[preset], _Timer()
    W, V, eps = mc.hidden_size, mc.vocab_size, mc.rms_norm_eps
    kinds = {k: next(l["mixer"] for l in mc.layers if l["type"] == k) for k in ("attention", "parallel", "rglru")}
    p, pages, starts, counts = _layout(lengths, batch, ctx)
    M, n = p.rows, p.nseq
    x, y32, w, h = torch.randn(M, W, device=DEV), torch.randn(M, W, device=DEV), _bf(W), _bf(M, W)
    t("norm_add", lambda: ops.norm_add(x, y32, w, 0.5, W, eps), M * W * 14)

    a = kinds["attention"]
    H, G, dk, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
    lq, lk, lv = H * dk, G * dk, G * dv
    _gemm(t, "gemm in (attention)", M, lq + lk + lv, W)
    _gemm(t, "gemm in (attention, shared keys)", M, lq, W)
    kc, vc = _bf(pages, 16, G, dk), _bf(pages, 16, G, dv)
    yy, wd, bias, sink = _bf(M, lq + lk + lv), _bf(dk), _bf(lq + lk + lv), _bf(H)
    s = a["rot"]["scaling"]
    cs, sn = ops.rope_rows(p.positions, ops.rope_turns(a["rot"]["base"], a["rot"]["dims"], DEV, (s["factor"], s["low"], s["high"], s["original"])))

    def store():
        return ops.qk_norm_store(yy[:, :lq], yy[:, lq:lq + lk], yy[:, lq + lk:], kc, vc, p, H, dk, True, eps, wd, wd, bias, cs, sn)
    t("qk_norm_store", store, M * ((lq + lk + lv) * 4 + a["rot"]["dims"] * 4))
    t("qk_norm_store (queries alone)", lambda: ops.qk_norm_store(yy[:, :lq], None, None, kc, vc, p, H, dk, True, eps, wd, None, bias[:lq], cs, sn),
      M * (lq * 4 + a["rot"]["dims"] * 4))
    q, out = store(), _bf(M, H * dv)
    pairs = sum((s + k) * (s + k + 1) / 2 - s * (s + 1) / 2 for s, k in zip(starts, counts))
    t("paged_attention", lambda: ops.paged_attention(q, kc, vc, out, p, H, a["scale"], sink=sink),
      M * (lq + H * dv) * 2 + (pairs if lengths is None else M) * (lk + lv) * 2, 2.0 * pairs * H * (dk + dv))
    _gemm(t, "gemm attention o (fp32)", M, W, H * dv, True)

    b = kinds["parallel"]["right"]
    H2, dk, dv = b["heads"], b["dim"], b["vdim"]
    c = [0, H2 * dk, 2 * H2 * dk, 2 * H2 * dk + H2 * dv, 2 * H2 * (dk + dv)]
    _gemm(t, "gemm in (parallel)", M, lq + lk + lv + c[4], W)
    wz = _bf(2 * pad8(H2), W)
    t("memory gates (fp32 product)", lambda: ops.linear_fp32(h, wz), (M * W + wz.numel()) * 2 + M * wz.shape[0] * 4)
    y, out, nw, bz = _bf(M, c[4]), _bf(M, H2 * dv), _bf(H2 * dv), _bf(2, H2)
    z = torch.randn(M, 2 * pad8(H2), device=DEV)
    z[:, pad8(H2):] += 4
    S, nn, mm = torch.zeros(n, H2, dk, dv, device=DEV), torch.zeros(n, H2, dk, device=DEV), torch.zeros(n, H2, device=DEV)
    flops = M * H2 * (2.0 * 64 * (dk + dv) / 2 + 4.0 * dk * dv)          # chunked form, 64-token chunks
    state = n * H2 * (dk * dv + dk) * 4 * (1 if lengths else 2)
    t("matrix_memory", lambda: ops.matrix_memory(*(y[:, c[i]:c[i + 1]] for i in range(4)), z[:, :H2], z[:, pad8(H2):pad8(H2) + H2], bz[0], bz[1], out,
                                                 S, nn, mm, p, nw, dk, dv, 15.0, dk ** -0.5, 1.0, eps),
      M * H2 * ((2 * dk + 3 * dv) * 2 + 8) + state, flops if lengths else 0)
    _gemm(t, "gemm parallel o (fp32)", M, W, H * a["vdim"] + H2 * dv, True)

    r = kinds["rglru"]
    C, B = r["width"], r["blocks"]
    _gemm(t, "gemm in (recurrence)", M, 2 * C, W)
    y, taps, v, gb = _bf(M, 2 * C), _bf(C, r["conv"]), _bf(C), _bf(B, 2, C // B)
    wg, lam, out = _bf(B, 2, C // B, C // B) * 0.1, torch.full((C,), -5.0, device=DEV, dtype=torch.bfloat16), _bf(M, C)
    S, conv = torch.zeros(n, C, device=DEV), torch.zeros(n, C, r["conv"] - 1, device=DEV)
    t("gated_recurrence", lambda: ops.gated_recurrence(y[:, :C], y[:, C:], v, v, taps, v, wg, gb, lam, out, S, conv, p),
      M * C * 6 + wg.numel() * 2 + n * C * r["conv"] * 4 * 2, 4.0 * M * C * (C // B))
    _gemm(t, "gemm recurrence o (fp32)", M, W, C, True)

    f = next(l["mlp"] for l in mc.layers if l["mlp"]["kind"] == "moe")
    ro, F, sh = f["router"], f["expert"]["ff"], f["shared"]["ff"]
    E, top = ro["experts"], ro["top"]
    wr, corr = _bf(pad8(E) + 8, W) * 0.05, _bf(E) * 0.1

    def route():
        return ops.router(h, wr, pad8(E), corr, top, ro["groups"]["count"], ro["groups"]["keep"], ro["scale"], joint)
    joint = sh == F                      # the shared expert is then one more of the experts
    t("router", route, M * (W * 2 + top * 12) + wr.numel() * 2)
    rt = route()[0]
    E, top = E + int(joint), top + int(joint)
    w_in, w_out = _bf(E, 2, F, W), _bf(E, W, F)
    used = int((rt.offsets[1:] > rt.offsets[:-1]).sum())
    t("expert_glu", lambda: ops.expert_glu(h, w_in, rt), (used * 2 * F * W + M * W + M * top * F) * 2, 4.0 * M * top * F * W)
    act = ops.expert_glu(h, w_in, rt)
    t("expert_down", lambda: ops.expert_down(act, w_out, rt), (used * F * W + M * top * (F + W)) * 2, 2.0 * M * top * F * W)
    rows, sg = ops.expert_down(act, w_out, rt), torch.randn(M, device=DEV)
    sh32, gate = (None, None) if joint else (y32, sg)
    t("moe_norm_add", lambda: ops.moe_norm_add(x, rows, rt, sh32, gate, w, 0.5, W, eps), M * W * (10 + 2 * top + (0 if joint else 4)))
    ff = next(l["mlp"]["ff"] for l in mc.layers if l["mlp"]["kind"] == "dense")
    gu, act = _bf(2 * ff, W), _bf(M, ff)
    t("glu_linear (dense)", lambda: ops.glu_linear(h, gu, act), (M * W + 2 * ff * W + M * ff) * 2, 4.0 * M * ff * W)
    _gemm(t, "gemm dense down (fp32)", M, W, ff, True)
    d = mc.side_dim
    wt, table, ids = _bf(d, W), _bf(V, 4 * d), torch.randint(0, V, (M,), device=DEV)
    t("token_gate", lambda: ops.token_gate(h, wt, table, ids, d, V), (M * W + d * W + 2 * M * d) * 2, 2.0 * M * d * W)
    _gemm(t, "gemm token projection (fp32)", M, W, d, True)
    if lengths is None:
        _gemm(t, "gemm logits (fp32)", M, V, W, True)
    del t.flush
    return t.rows


def lufivik_kernels(preset: str, lengths: Optional[List[int]] = None, batch: int = 256, ctx: int = 1024) -> Dict:
    """The same for the windowed latent-attention decoder with softmax-routed experts."""
    from ..ops import latent
    mc, t = PRESETS[preset], _Timer()
    W, V, eps = mc.hidden_size, mc.vocab_size, mc.norm_eps
    m, f = mc.layers[0]["mixer"], mc.layers[0]["mlp"]
    p, pages, starts, counts = _layout(lengths, batch, ctx)
    M, n = p.rows, p.nseq
    x, y32, w, b, h = torch.randn(M, W, device=DEV), torch.randn(M, W, device=DEV), _bf(W), _bf(W), _bf(M, W)

    table, pairs, last = _bf(V, W), _bf(mc.buckets + 1, W), torch.zeros(n, dtype=torch.int32, device=DEV)
    ids = torch.randint(0, V, (M,), device=DEV)
    t("embedding_pairs", lambda: ops.embedding_pairs(ids, table, pairs, last, p, V, mc.mul_prev, mc.mul_cur, (w, b), W, eps, (w, b)), M * W * 10)
    taps, conv = _bf(W, mc.taps), torch.zeros(n, W, mc.taps - 1, device=DEV)
    t("input convolution", lambda: ops.causal_conv(h, None, taps, None, conv, p, add_input=True),
      M * W * 4 + n * W * (mc.taps - 1) * 4 * (1 if lengths else 2))
    _gemm(t, "gemm residual gate", M, W, W)
    g16 = _bf(M, W)
    t("branch_add", lambda: ops.branch_add(x, y32, (w, b), W, eps, g16, b, w, (w, b)), M * W * 16)

    H, d, r, dv, C, Q, win = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"], m["mask"]["size"]
    dq, R = d + r, C + r
    _gemm(t, "gemm in (latents)", M, Q + R + pad8(H), W)
    yy, pg = _bf(M, Q + R + pad8(H)), _bf(pages, 16, 1, R)
    cs, sn = ops.rope_rows(p.positions, ops.rope_turns(m["rot"]["base"], r, DEV))
    wq, wc, w_key, w_value, out = _bf(Q), _bf(C), _bf(H, dq, R), _bf(H, dv, C), _bf(M, H * dv)
    cq, cc, kr, gate = yy[:, :Q], yy[:, Q:Q + C], yy[:, Q + C:Q + R], yy[:, Q + R:Q + R + H]
    t("latent_store (both latents)", lambda: ops.latent_store(None, cc, kr, pg, p, H, d, C, r, wc, cs, sn, eps, cq, wq, Q),
      M * (Q * 4 + R * 4 + r * 4))
    _gemm(t, "gemm queries", M, H * dq, Q)
    q, turn = _bf(M, H * dq), (cs, sn, d)
    seen = sum(min(i + 1, win) for s, k in zip(starts, counts) for i in range(s, s + k))          # query-key pairs
    if lengths is None:
        ql, ol = _bf(M, H * R), _bf(M, H * C)
        t("head_linear (queries to latent, turned)", lambda: ops.head_linear(q, w_key, ql, True, (cs, sn, C)), (M * H * (dq + R) + H * dq * R) * 2)
        t("latent_rows", lambda: ops.latent_rows(ql, pg, ol, p, H, C, m["scale"], None, win), (seen * R + M * H * (R + C)) * 2,
          2.0 * seen * H * (R + C))
        t("head_linear (latent to values, gated)", lambda: ops.head_linear(ol, w_value, out, gate=gate), (M * H * (dv + C) + H * dv * C) * 2)
        flops = 2.0 * seen * H * (R + C)
    else:
        _gemm(t, "gemm keys from latents", M, H * dq, R)
        _gemm(t, "gemm values from latents", M, H * dv, C)
        t("latent_turn", lambda: ops.latent_turn(q, H, d, cs, sn), M * (H * r * 4 + r * 4))
        k, v, c = _bf(pages * 16, H * dq), _bf(pages * 16, H * dv), p.context(win)
        t("latent prompt attention alone", lambda: latent.expanded_attention(q, k, v, out, p, H, dq, dv, m["scale"], None, 0, n, c.tables, win, gate),
          M * H * (dq + dv) * 4, 2.0 * seen * H * (dq + dv))
        rows = torch.empty(pages * 16, R, device=DEV, dtype=torch.bfloat16)
        t("latent_gather", lambda: latent.gather(pg, c.pages, rows), rows.numel() * 4)
        flops = 2.0 * (seen * H * (dq + dv) + M * H * (dq * R + dv * C))
    t("latent_attention", lambda: ops.latent_attention(q, pg, out, p, w_key, w_value, m["scale"], None, win, gate, turn),
      M * H * (dq + dv) * 2 + (seen if lengths is None else M) * R * 2, flops)
    _gemm(t, "gemm latent o (fp32)", M, W, H * dv, True)

    E, top, F = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
    wr = _bf(pad8(E) + W, W) * 0.05
    t("router and gate product (fp32)", lambda: ops.linear_fp32(h, wr), (M * W + wr.numel()) * 2 + M * wr.shape[0] * 4, 2.0 * M * wr.numel())
    z = ops.linear_fp32(h, wr)
    t("choice and layout", lambda: ops.route(z, None, top, 1, 1, 1.0, score="softmax", experts=E), M * (E * 4 + top * 12))
    rt = ops.route(z, None, top, 1, 1, 1.0, score="softmax", experts=E)
    w_in, w_out, act = _bf(E, 2, F, W), _bf(E, W, F), (1.702, f["expert"]["limit"])
    used = int((rt.offsets[1:] > rt.offsets[:-1]).sum())
    t("expert_glu (clamped)", lambda: ops.expert_glu(h, w_in, rt, act), (used * 2 * F * W + M * W + M * top * F) * 2, 4.0 * M * top * F * W)
    a = ops.expert_glu(h, w_in, rt, act)
    t("expert_down", lambda: ops.expert_down(a, w_out, rt), (used * F * W + M * top * (F + W)) * 2, 2.0 * M * top * F * W)
    rows = ops.expert_down(a, w_out, rt)
    t("branch_add (experts)", lambda: ops.branch_add(x, (rows, rt), (w, b), W, eps, z[:, pad8(E):], b, w, (w, b)), M * W * (14 + 2 * top))
    if lengths is None:
        t("layernorm_f32", lambda: ops.layernorm_f32(x, (w, b), W, eps), M * W * 6)
        _gemm(t, "gemm logits (fp32)", M, V, W, True)
    del t.flush
    return t.rows


def dense_kernels(preset: str, lengths: Optional[List[int]] = None, batch: int = 256, ctx: int = 1024) -> Dict:
    """The same for the dense decoder family."""
    mc, t = PRESETS[preset], _Timer()
    W, V, H, G, D, ff = mc.hidden_size, mc.vocab_size, mc.num_heads, mc.num_kv_heads, mc.head_dim, mc.intermediate_size
    p, pages, starts, counts = _layout(lengths, batch, ctx)
    M = p.rows
    x, w, wd = _bf(M, W), _bf(W), _bf(D)
    t("rmsnorm", lambda: ops.rmsnorm(x, w, 1e-6), M * W * 4)
    nq = (H + 2 * G) * D
    _gemm(t, "gemm qkv", M, nq, W)
    kc, vc = _bf(pages, 16, G, D), _bf(pages, 16, G, D)
    qkv = _bf(M, nq)
    cos, sin = ops.rope_tables(max(ctx, max(counts)) + 1, D, mc.rope_theta, torch.device(DEV))
    pos = p.positions
    blk = p.block_tables[p.row_seq.long(), (pos // 16).long()]
    slots = (blk * 16 + pos % 16).to(torch.int32)

    def store():
        return ops.qknorm_rope_store(qkv, wd, wd, pos, cos, sin, H, G, D, 1e-6, kc, vc, slots)
    t("qknorm_rope_store", store, M * nq * 4)
    q, k, v = store()
    if lengths is None:
        lens = torch.full((batch,), ctx, dtype=torch.int32, device=DEV)
        t("paged_decode_attention", lambda: ops.paged_decode_attention(q, kc, vc, p.block_tables, lens, H),
          batch * ctx * 2 * G * D * 2 + M * 2 * H * D * 2)
    else:
        cu = torch.tensor([0] + list(torch.tensor(lengths).cumsum(0)), dtype=torch.int32, device=DEV)
        pairs = sum(n * (n + 1) / 2 for n in lengths)
        t("paged_prefill_attention", lambda: ops.paged_prefill_attention(q, kc, vc, p.block_tables, cu, cu, max(lengths), H),
          M * (2 * H + 2 * G) * D * 2, 4.0 * pairs * H * D)
    _gemm(t, "gemm o (+ residual)", M, W, H * D, residual=True)
    _gemm(t, "gemm gate_up", M, 2 * ff, W)
    gu = _bf(M, 2 * ff)
    t("swiglu", lambda: ops.swiglu(gu), M * ff * 6)
    _gemm(t, "gemm down (+ residual)", M, W, ff, residual=True)
    if lengths is None:
        _gemm(t, "gemm logits", M, V, W)
    del t.flush
    return t.rows


def kernels(preset: str, lengths: Optional[List[int]] = None, batch: int = 256, ctx: int = 1024) -> Dict:
    by_name = {"Fetelorn": fetelorn_kernels, "Sotazen": sotazen_kernels, "Ruburax": ruburax_kernels, "Lufivik": lufivik_kernels}
    with torch.no_grad():
        return by_name.get(getattr(PRESETS[preset], "architecture", None), dense_kernels)(preset, lengths, batch, ctx)
