"""Runner for models whose layers differ from one another: per-layer pages (or none), recurrent state slots, portions of
prompts and single decoded tokens in one batch, a 32-bit residual stream.

A step is a set of portions, one per sequence.  The rows of short portions (decoded tokens among them) come first and take
the row-by-row kernels, long portions take the tiled ones; every projection runs once over all rows.  The caller's row order
is kept at the interface (:attr:`InferenceContext.row_order`)."""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from .. import ops
from ..ops.portions import Portions
from .context import InferenceContext
from .kv_cache import BlockPool, KVCacheManager, StatePool
from .runner import ModelRunner

TILE = 16          # rows per tile of the row-wise input stages
CHUNKS = (64, 128)     # rows per chunk of the chunked recurrences
SHORT_ROWS = 16    # portions up to this many rows take the row-by-row kernels


class HybridModelRunner(ModelRunner):
    mixed_batches = True      # prompt portions and decoded tokens share one forward pass

    def __init__(self, model, pool: BlockPool, manager: KVCacheManager, partition_size: int = 512,
                 enable_partitioned: bool = False):
        super().__init__(model, pool, manager, partition_size, enable_partitioned)
        self.state: StatePool = manager.state
        self._turns: Dict[tuple, torch.Tensor] = {}
        # the layers in the order they run (one may run several times, each time with pages and state of its own), and whose pages
        # a run reads: its own, or those of an earlier one
        self._runs = list(getattr(model, "layer_runs", lambda: range(len(model.layers)))())
        self._pages = [li if src is None else src for li, src in enumerate(getattr(model, "kv_sources", lambda: [None] * len(self._runs))())]

    # ---- metadata ----------------------------------------------------------------------------------------
    def prepare_prefill(self, seq_ids: Sequence, starts: Sequence[int], counts: Sequence[int]) -> InferenceContext:
        """Sequence ``i`` computes positions ``starts[i] .. starts[i] + counts[i] - 1`` (its pages already cover them)."""
        p, order, place = build_portions(starts, counts, [self.mgr.get_block_table(i) for i in seq_ids],
                                         [self.state.slot(i) for i in seq_ids], self.dtype == torch.float32, self._np)
        n = len(seq_ids)
        cu = np.concatenate([[0], np.cumsum([counts[i] for i in order])])
        last = np.zeros(n, dtype=np.int64)
        last[np.asarray(order, dtype=np.int64)] = cu[1:] - 1       # in the caller's sequence order, as kernel rows
        back = None
        if place is not None:
            back = np.empty_like(place)
            back[place] = np.arange(len(place))
        return InferenceContext(
            is_prefill=True, num_seqs=n, total_q=p.rows, max_seqlen_q=max(counts, default=0), positions=p.positions,
            last_token_rows=self._np(last), portions=p, block_tables=p.block_tables,
            row_order=None if place is None else self._np(back), row_place=None if place is None else self._np(place))

    def prepare_decode(self, seq_ids: Sequence, pad_to: int = 0, max_blocks: int = 0) -> InferenceContext:
        """One decoded token per sequence at position ``len - 1``; rows past the sequences are padding (slot -1)."""
        n = len(seq_ids)
        B = max(n, pad_to)
        tables = [self.mgr.tables[s] for s in seq_ids]
        width = max(max_blocks, max((t.num_blocks for t in tables), default=1), 1)
        bt = np.full((B, width), -1, dtype=np.int32)
        pos = np.zeros(B, dtype=np.int32)
        slots = np.full(B, -1, dtype=np.int32)
        for i, (s, t) in enumerate(zip(seq_ids, tables)):
            ids = t.get_physical_block_ids()
            bt[i, :len(ids)] = ids
            pos[i] = t.num_tokens - 1
            slots[i] = self.state.slot(s)
        bt, pos_d, slots = self._np(bt), self._np(pos), self._np(slots)
        return InferenceContext(is_prefill=False, num_seqs=B, block_tables=bt, positions=pos_d, slot_mapping=slots,
                                max_context_len=int(pos.max()) + 1 if B else 0,
                                portions=self._decode_portions(bt, pos_d, slots, int(pos.max()) + 1 if B else 1))

    def _np(self, a: np.ndarray) -> torch.Tensor:
        return self._stage(torch.from_numpy(np.ascontiguousarray(a)))

    def _decode_portions(self, bt, pos, slots, max_keys: int) -> Portions:
        """One row per sequence.  The arrays that depend on the batch size alone are made once per size."""
        B = pos.shape[0]
        fixed = self.__dict__.setdefault("_decode_fixed", {})
        if B not in fixed:
            ar = torch.arange(B + 1, dtype=torch.int32)
            tiles = torch.stack([ar[:B], ar[:B], torch.ones(B, dtype=torch.int32), torch.zeros(B, dtype=torch.int32)], 1)
            fixed[B] = (ar.to(self.device), tiles.contiguous().to(self.device))
        ar, tiles = fixed[B]
        return Portions(cu=ar, starts=pos, slots=slots, row_seq=ar[:B], positions=pos, tiles=tiles, block_tables=bt, nseq=B,
                        num_short=B, short_rows=B, max_short=1, max_keys=max_keys, ragged=False)

    # ---- CUDA-graph decode ---------------------------------------------------------------------------------
    def graph_inputs(self, n: int, width: int) -> Dict[str, torch.Tensor]:
        d = self.device
        return {"tokens": torch.zeros(n, dtype=torch.long, device=d), "positions": torch.zeros(n, dtype=torch.int32, device=d),
                "block_tables": torch.full((n, width), -1, dtype=torch.int32, device=d),
                "slots": torch.full((n,), -1, dtype=torch.int32, device=d)}

    def graph_values(self, ctx: InferenceContext) -> Dict[str, torch.Tensor]:
        return {"positions": ctx.positions, "block_tables": ctx.block_tables, "slots": ctx.slot_mapping}

    def graph_context(self, inp: Dict[str, torch.Tensor], width: int) -> InferenceContext:
        p = self._decode_portions(inp["block_tables"], inp["positions"], inp["slots"], width * self.block_size)
        return InferenceContext(False, inp["tokens"].shape[0], block_tables=inp["block_tables"], positions=inp["positions"],
                                portions=p)

    # ---- forward -----------------------------------------------------------------------------------------
    @torch.no_grad()
    def forward(self, token_ids: torch.Tensor, ctx: InferenceContext, all_rows: bool = False,
                split_plan: Optional[Tuple[int, int]] = None, rows: Optional[torch.Tensor] = None,
                on_layer=None) -> torch.Tensor:
        """Token ids ``[M]`` (caller's order) -> logits of each sequence's last row, of every row (``all_rows``) or of the
        caller's rows ``rows`` (int64).  ``on_layer(i, x)`` sees the residual rows (kernel order) after every layer run."""
        m, p = self.model, ctx.portions
        self.forward_calls += 1
        ids = token_ids if ctx.row_order is None else token_ids.index_select(0, ctx.row_order)
        p.ids = ids
        x, h = m.embed(ids, p, self.state.sequence)
        tables: Dict[tuple, Tuple[torch.Tensor, torch.Tensor]] = {}

        def rope(base: float, dims: int, stretch: Optional[tuple] = None):
            key = (base, dims, stretch)
            if key not in tables:
                if key not in self._turns:
                    self._turns[key] = ops.rope_turns(base, dims, self.device, stretch)
                tables[key] = ops.rope_rows(p.positions, self._turns[key])
            return tables[key]

        layers = [m.layers[i] for i in self._runs]
        for li, layer in enumerate(layers):
            after = layers[li + 1].norm1 if li + 1 < len(layers) else None
            h = layer(x, h, p, self.pool.layer_kv(self._pages[li]), self.state.layers[li], rope, after)
            if on_layer is not None:
                on_layer(li, x)
        if rows is not None:
            pick = rows if ctx.row_place is None else ctx.row_place.index_select(0, rows)
        elif all_rows:
            pick = ctx.row_place
        else:
            pick = ctx.last_token_rows if ctx.is_prefill else None
        if hasattr(m, "final_norm"):
            return m.logits_from_hidden(m.final_norm(x, pick))
        return m.logits_from_hidden(ops.rmsnorm_f32(x, m.norm, m.cfg.hidden_size, m.cfg.rms_norm_eps, pick,
                                                        getattr(m, "logit_scale", 1.0)))

    def run_batch_decode(self, *a, **k):
        raise NotImplementedError("raw-tensor decode knows no state slots: use prepare_decode + forward")


def build_portions(starts: Sequence[int], counts: Sequence[int], tables: Sequence[Sequence[int]], slots: Sequence[int],
                   serial: bool, dev=torch.from_numpy) -> Tuple[Portions, List[int], Optional[np.ndarray]]:
    """Row layout of one step: sequence ``i`` computes ``counts[i]`` positions from ``starts[i]``.  ``serial``: every portion
    takes the row-by-row kernels (32-bit runs).  Returns the layout, the kernels' order of the sequences, and the kernel row of
    every caller's row (None when the orders agree)."""
    n = len(counts)
    short = [i for i in range(n) if serial or counts[i] <= SHORT_ROWS]
    order = short + [i for i in range(n) if not (serial or counts[i] <= SHORT_ROWS)]
    c = np.asarray([counts[i] for i in order], dtype=np.int32)
    st = np.asarray([starts[i] for i in order], dtype=np.int32)
    cu = np.zeros(n + 1, dtype=np.int32)
    np.cumsum(c, out=cu[1:])
    M = int(cu[-1])
    row_seq = np.repeat(np.arange(n, dtype=np.int32), c)
    pos = (np.arange(M, dtype=np.int32) - cu[row_seq] + st[row_seq]).astype(np.int32)
    bt = np.full((n, max(1, max((len(t) for t in tables), default=1))), -1, dtype=np.int32)
    for r, i in enumerate(order):
        bt[r, :len(tables[i])] = tables[i]
    place = None
    if order != list(range(n)):
        caller = np.zeros(n + 1, dtype=np.int64)
        np.cumsum(np.asarray(counts, dtype=np.int64), out=caller[1:])
        place = np.empty(M, dtype=np.int64)
        place[np.concatenate([np.arange(caller[i], caller[i + 1]) for i in order])] = np.arange(M)
    ns = len(short)
    p = Portions(
        cu=dev(cu), starts=dev(st), slots=dev(np.asarray([slots[i] for i in order], dtype=np.int32)), row_seq=dev(row_seq),
        positions=dev(pos), tiles=dev(_row_tiles(cu, 0, n, TILE)), block_tables=dev(bt), nseq=n, num_short=ns,
        short_rows=int(cu[ns]), max_short=int(c[:ns].max()) if ns else 0, max_keys=int((st + c).max()) if n else 1,
        max_long=int(c[ns:].max()) if ns < n else 0)
    if ns < n:
        for size in CHUNKS:
            first = np.concatenate([[0], np.cumsum((c[ns:] + size - 1) // size)]).astype(np.int32)
            setattr(p, f"chunks{size}", dev(_row_tiles(cu, ns, n, size)))
            setattr(p, f"first{size}", dev(first))
        p.host_long, p.to_device = (st[ns:], c[ns:], bt[ns:]), dev
    return p, order, place


def _row_tiles(cu: np.ndarray, lo: int, hi: int, size: int) -> np.ndarray:
    """``[n, 4]`` = (sequence, first row, rows, offset in the portion) for sequences ``lo .. hi - 1``."""
    cnt = np.diff(cu)[lo:hi]
    per = (cnt + size - 1) // size
    total = int(per.sum())
    seq = np.repeat(np.arange(lo, hi, dtype=np.int32), per)
    off = (np.arange(total, dtype=np.int32) - np.repeat(np.cumsum(per) - per, per).astype(np.int32)) * size
    rows = np.minimum(size, np.diff(cu)[seq] - off) if total else off
    return np.stack([seq, cu[seq] + off, rows, off], 1).astype(np.int32) if total else np.zeros((0, 4), dtype=np.int32)


def make_cache(model, num_blocks: int, block_size: int, num_slots: int, dtype, device) -> Tuple[BlockPool, KVCacheManager]:
    """Pages and state slots for a model with per-layer caches."""
    mc = model.cfg
    pool = BlockPool(num_blocks, block_size, mc.num_layers, mc.num_kv_heads, mc.head_dim, dtype, device,
                     layer_shapes=model.kv_layer_shapes())
    return pool, KVCacheManager(pool, block_size, StatePool(
        num_slots, model.state_layer_shapes(), device, getattr(model, "state_sequence_shapes", dict)()))


@torch.no_grad()
def whole_sequences(model, input_ids: torch.Tensor) -> torch.Tensor:
    """``[B, S]`` ids -> ``[B, S, V]`` logits: one step over whole sequences, with a cache that lives for the call."""
    B, S = input_ids.shape
    dev = model.embed_tokens.device
    pool, mgr = make_cache(model, B * ((S + 15) // 16), 16, B, model.embed_tokens.dtype, dev)
    run = HybridModelRunner(model, pool, mgr)
    for b in range(B):
        mgr.allocate_for_sequence(b, S)
    ctx = run.prepare_prefill(list(range(B)), [0] * B, [S] * B)
    return run.forward(input_ids.reshape(-1).to(dev), ctx, all_rows=True).reshape(B, S, -1)
