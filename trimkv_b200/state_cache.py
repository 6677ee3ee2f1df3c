"""What the requests of a hybrid decoder keep between steps: recurrent states, convolution inputs, windows of keys and values.

``HybridStateCache`` stands beside ``TrimKVCache`` for models whose layers are not all softmax attention over the whole
past.  A request owns one *slot*, the same in every layer's arrays:

  * ``RecurrentState``: fp32 state ``[slots, heads, n, p]`` and, where the layer has a short convolution, a ring of its last
    ``taps`` inputs ``[slots, taps, channels]`` (input of position p in row p mod taps);
  * ``WindowState``: keys and values of the last ``window`` positions, ``[slots, kv_heads, rows, ...]`` with position p in row
    p mod rows; rows grow with the sequences up to the window and then stay;
  * ``LatentState``: the same for latent attention, one row per position that all heads share, ``[slots, rows, ...]``.

Nothing is cleared when a slot is given back and taken again: every kernel starts a request at position 0 from the empty
state.  Lengths may differ between the requests of a batch; tokens of a step are packed (``StepBatch``), so no kernel sees
padding.  A one-token step (``begin(None)``) needs no host-to-device copy once the batch is fixed, which lets it be
recorded in a CUDA graph.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from . import ops


@dataclass(frozen=True)
class RecurrentState:
    heads: int
    n: int
    p: int
    conv_taps: int = 0
    conv_channels: int = 0
    window = 0

    def arrays(self, rows: int, dtype):
        """name -> (shape of a slot, type, axis of the ring rows or None)"""
        out = {"state": ((self.heads, self.n, self.p), torch.float32, None)}
        if self.conv_taps:
            out["conv"] = ((self.conv_taps, self.conv_channels), dtype, None)
        return out


@dataclass(frozen=True)
class WindowState:
    kv_heads: int
    dp: int          # padded key size of one map
    pp: int          # padded value size
    window: int
    maps: int = 2

    def arrays(self, rows: int, dtype):
        return {"k": ((self.kv_heads, rows, self.maps, self.dp), dtype, 1), "v": ((self.kv_heads, rows, self.pp), dtype, 1)}


@dataclass(frozen=True)
class LatentState:
    row: int         # elements of a position: padded latent and padded rotated key part
    window: int

    def arrays(self, rows: int, dtype):
        return {"latent": ((rows, self.row), dtype, 0)}


@dataclass
class StepBatch:
    """One step's requests.  ``cu`` is None in a one-token step; ``starts`` are the host's copy of ``pos0``."""
    size: int
    tokens: int
    max_tokens: int
    slots: torch.Tensor
    pos0: torch.Tensor
    cu: Optional[torch.Tensor]
    lengths: List[int]
    starts: List[int]
    status: torch.Tensor
    _plans: Dict[int, Tuple[torch.Tensor, int, int]] = field(default_factory=dict)

    def window_plan(self, window: int) -> Tuple[torch.Tensor, int, int]:
        """``(kv_start, rows, longest history)`` of the linear key buffer of a layer with this window: each request's
        tokens behind the positions before the step that the window still reaches."""
        plan = self._plans.get(window)
        if plan is None:
            hist = [min(s, window - 1) for s in self.starts]
            at, starts = 0, []
            for h, n in zip(hist, self.lengths):
                starts.append(at)
                at += h + n
            if max(hist, default=0) == 0:
                plan = (self.cu, at, 0)
            else:
                plan = (torch.tensor(starts, dtype=torch.int32).to(self.slots.device, non_blocking=True), at, max(hist))
            self._plans[window] = plan
        return plan


class HybridStateCache:
    """Slots of a hybrid decoder.  ``open`` adds requests to the batch, ``close`` gives them back, ``begin`` starts a step.

    Rows of the batch are addressed by position (0 .. batch size - 1) in the order they were opened."""

    # HF generate() probes these on any cache object.
    is_compileable = False
    is_sliding = [False]

    def __init__(self, layers: Sequence, device="cuda", dtype=torch.bfloat16, capacity_tokens: int = 0):
        self.layers, self.device, self.dtype = list(layers), torch.device(device), dtype
        self._cap = max(int(capacity_tokens), 64)      # positions per request the windows have rows for
        self._nslots = 0
        self._free: List[int] = []
        self._rows: List[int] = []                     # slot of every row of the batch
        self._len: Dict[int, int] = {}                 # tokens seen, by slot
        self._data: List[dict] = [{} for _ in self.layers]
        self._lens = None
        self._status = None
        self._decode_key = None
        self._generation = 0                           # changes whenever an array moved
        self.static_views = False                      # part of the decoder's cache interface; nothing here depends on it

    # ------------------------------------------------------------------ batch
    def __len__(self):
        return len(self.layers)

    @property
    def _batch(self) -> int:
        return len(self._rows)

    def open(self, count: int) -> List[int]:
        """Adds ``count`` empty requests to the batch; returns their rows."""
        if len(self._free) < count:
            self._resize(max(self._nslots + count - len(self._free), 2 * self._nslots if self._nslots else 0))
        taken = [self._free.pop() for _ in range(count)]
        for s in taken:
            self._len[s] = 0
        first = len(self._rows)
        self._rows += taken
        if taken:
            self._lens[torch.tensor(taken, dtype=torch.int64, device=self.device)] = 0
        self._decode_key = None
        return list(range(first, first + count))

    def close(self, rows: Sequence[int]) -> None:
        """Gives the slots of these rows back; the remaining rows keep their order and move up."""
        gone = set(int(r) for r in rows)
        for r in gone:
            slot = self._rows[r]
            self._free.append(slot)
            del self._len[slot]
        self._rows = [s for r, s in enumerate(self._rows) if r not in gone]
        self._decode_key = None

    def batch_select_indices(self, indices) -> None:
        """Keeps the rows named by ``indices``, in that order (each at most once); the others' slots are given back."""
        keep = [int(i) for i in (indices.tolist() if torch.is_tensor(indices) else indices)]
        if len(set(keep)) != len(keep):
            raise ValueError("a request of this cache cannot be duplicated: its state lives in one slot")
        order = [self._rows[i] for i in keep]
        self.close([r for r in range(len(self._rows)) if r not in set(keep)])
        self._rows = order
        self._decode_key = None

    # ------------------------------------------------------------------ bookkeeping
    def get_seq_length(self, layer_idx: Optional[int] = None) -> int:
        return max((self._len[s] for s in self._rows), default=0)

    def row_lengths(self) -> List[int]:
        return [self._len[s] for s in self._rows]

    def get_cache_length(self, layer_idx: int = 0) -> int:
        """Positions a layer holds something of: its window's rows, or 0 for a layer whose past is a state."""
        st = self.layers[layer_idx]
        return min(self.get_seq_length(), st.window)

    def get_mask_sizes(self, cache_position, layer_idx: int = 0):
        n = cache_position if isinstance(cache_position, int) else cache_position.shape[0]
        return self.get_seq_length() + n, 0

    def advance(self, num_tokens: int = 1) -> None:
        for s in self._rows:
            self._len[s] += num_tokens

    def snapshot_counters(self):
        return dict(self._len)

    def restore_counters(self, snap) -> None:
        self._len = dict(snap)

    def graph_key(self):
        """Changes whenever a recorded one-token step may no longer be replayed."""
        return (self._generation, tuple(self._rows)) if self._lens is not None else None

    def fits(self, num_tokens: int = 1) -> bool:
        """Whether ``num_tokens`` more tokens per request need no array to move."""
        return self._lens is not None and self.get_seq_length() + num_tokens <= self._cap

    def check_status(self) -> None:
        """Synchronises and raises if a kernel reported a device-side problem."""
        if self._status is not None:
            code = ops.read_status(self._status)
            if code:
                raise ops._lib.TrimKVNativeError(f"device status {code}: "
                                                 + {3: "token id outside the vocabulary", 4: "a bounded wait ran out"}.get(code, "unknown"))

    # ------------------------------------------------------------------ a step
    def begin(self, lengths: Optional[Sequence[int]], rows: Optional[Sequence[int]] = None) -> StepBatch:
        """Starts a step in which row ``rows[i]`` (default: the whole batch in order) brings ``lengths[i]`` tokens; None: one
        token each.  Moves every counter on, on the host and on the device."""
        slots = self._rows if rows is None else [self._rows[r] for r in rows]
        if not slots:
            raise ValueError("a step without requests")
        counts = [1] * len(slots) if lengths is None else [int(n) for n in lengths]
        if len(counts) != len(slots) or len(set(slots)) != len(slots) or min(counts) < 1:
            raise ValueError("every request of a step appears once and brings at least one token")
        starts = [self._len[s] for s in slots]
        self.reserve(max(s + n for s, n in zip(starts, counts)))
        if all(n == 1 for n in counts):
            if self._decode_key != tuple(slots):
                if torch.cuda.is_current_stream_capturing():
                    raise RuntimeError("the batch changed while a one-token step was being recorded")
                self._slots_dev = torch.tensor(slots, dtype=torch.int32).to(self.device)
                self._pos0_dev = torch.empty_like(self._slots_dev)
                self._decode_key = tuple(slots)
                self._generation += 1
            dev_slots, pos0, cu = self._slots_dev, self._pos0_dev, None
        else:
            bounds = [0]
            for n in counts:
                bounds.append(bounds[-1] + n)
            packed = torch.tensor(slots + bounds, dtype=torch.int32).to(self.device, non_blocking=True)
            dev_slots, cu = packed[:len(slots)], packed[len(slots):]
            pos0 = torch.empty(len(slots), dtype=torch.int32, device=self.device)
        ops.batch_begin(self._lens, dev_slots, cu, pos0)
        for s, n in zip(slots, counts):
            self._len[s] += n
        return StepBatch(len(slots), sum(counts), max(counts), dev_slots, pos0, cu, counts, starts, self._status)

    def arrays(self, layer_idx: int) -> dict:
        return self._data[layer_idx]

    # ------------------------------------------------------------------ storage
    def reserve(self, tokens: int) -> None:
        """Makes room for sequences of ``tokens`` positions."""
        if tokens <= self._cap:
            return
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("cache capacity exhausted during CUDA graph capture")
        cap = max(tokens, 2 * self._cap)
        before, self._cap = self._cap, cap
        for st, data in zip(self.layers, self._data):
            if data and min(st.window, cap) > min(st.window, before):
                # no sequence has wrapped yet (rows < window), so a position keeps its row
                for name, (shape, dtype, axis) in st.arrays(min(st.window, cap), self.dtype).items():
                    old = data[name]
                    new = torch.empty(self._nslots, *shape, dtype=dtype, device=self.device)
                    new.narrow(axis + 1, 0, old.shape[axis + 1]).copy_(old)
                    data[name] = new
                self._generation += 1

    def _resize(self, nslots: int) -> None:
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("slots exhausted during CUDA graph capture")

        def grown(old, *shape, dtype):
            new = torch.empty(nslots, *shape, dtype=dtype, device=self.device)
            if old is not None:
                new[:self._nslots] = old
            return new
        if self._status is None:
            self._status = ops.new_status(self.device)
        for st, data in zip(self.layers, self._data):
            for name, (shape, dtype, _) in st.arrays(min(st.window, self._cap), self.dtype).items():
                data[name] = grown(data.get(name), *shape, dtype=dtype)
        lens = torch.zeros(nslots, dtype=torch.int32, device=self.device)
        if self._lens is not None:
            lens[:self._nslots] = self._lens
        self._lens = lens
        self._free += list(range(nslots - 1, self._nslots - 1, -1))
        self._nslots = nslots
        self._generation += 1


__all__ = ["HybridStateCache", "LatentState", "RecurrentState", "StepBatch", "WindowState"]
