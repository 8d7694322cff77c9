"""Row layout of a batch of sequence portions: what every state-carrying or paged op needs to know about a step."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Tuple

import numpy as np
import torch


def pad8(n: int) -> int:
    """Feature counts are stored in multiples of eight (16-byte rows for bf16): padding channels hold zeros."""
    return (n + 7) // 8 * 8


@dataclass
class Portions:
    """Sequence ``s`` owns rows ``cu[s]:cu[s+1]`` of the step's activations; its first row sits at position
    ``starts[s]`` and its recurrent state in slot ``slots[s]`` (-1: padding of a graph batch).  The first
    ``num_short`` sequences (``short_rows`` rows) hold one or a few tokens each and take the row-by-row kernels;
    the others take the tiled ones.  ``block_tables`` rows are padded with -1."""
    cu: torch.Tensor                         # int32 [nseq + 1]
    starts: torch.Tensor                     # int32 [nseq]
    slots: torch.Tensor                      # int32 [nseq]
    row_seq: torch.Tensor                    # int32 [M]
    positions: torch.Tensor                  # int32 [M]
    tiles: torch.Tensor                      # int32 [n, 4] = (sequence, first row, rows, offset in the portion), <= 16 rows
    block_tables: torch.Tensor               # int32 [nseq, max_blocks]
    nseq: int
    num_short: int
    short_rows: int
    max_short: int                           # longest portion among the short ones
    max_keys: int                            # longest context (tokens) of any sequence after this step
    # long portions cut into chunks of 64 and of 128 rows: int32 [n, 4] like tiles, and [nlong + 1] first chunk of each sequence
    chunks64: Optional[torch.Tensor] = None
    first64: Optional[torch.Tensor] = None
    chunks128: Optional[torch.Tensor] = None
    first128: Optional[torch.Tensor] = None
    max_long: int = 0
    # the long portions on the host: int32 [nlong] starts and counts, [nlong, max_blocks] pages; and the copy to the device
    host_long: Optional[Tuple[np.ndarray, np.ndarray, np.ndarray]] = None
    to_device: Optional[Callable[[np.ndarray], torch.Tensor]] = None
    contexts: Dict[int, "Context"] = field(default_factory=dict)
    ids: Optional[torch.Tensor] = None       # int64 [M] token of every row, for layers that look tokens up
    plans: Dict[Tuple[int, int, int], torch.Tensor] = field(default_factory=dict)    # decode_plan: (rows, window, tile) -> tile counts
    ragged: bool = True                      # False: every sequence is one row (decode): row r is sequence r

    @property
    def rows(self) -> int:
        return self.positions.shape[0]

    def context(self, window: int = 0) -> "Context":
        """What the long portions see (``window > 0``: of so many tokens back), laid out page after page."""
        if window not in self.contexts:
            starts, counts, tables = self.host_long
            first = np.maximum(starts - window + 1, 0) // 16 if window > 0 else np.zeros_like(starts)
            end = (starts + counts + 15) // 16
            n = end - first
            base = (np.cumsum(n) - n).astype(np.int32)
            page = np.arange(end.max(), dtype=np.int32)[None, :]
            place = base[:, None] + np.clip(page - first[:, None], 0, n[:, None] - 1)
            self.contexts[window] = Context(
                self.to_device(np.concatenate([tables[i, a:e] for i, (a, e) in enumerate(zip(first, end))])),
                self.to_device(place.astype(np.int32)), n.tolist())
        return self.contexts[window]


@dataclass
class Context:
    pages: torch.Tensor                      # int32 [sum of counts] page of the pool
    tables: torch.Tensor                     # int32 [nlong, max pages] where a sequence's pages are in that layout
    counts: List[int]                        # pages per sequence
