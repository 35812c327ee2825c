"""What one step hands to the parts: the batch on the device, the residual stream,
and buffers that live as long as the engine."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import numpy as np
import torch


class Workspace:
    """Named device buffers, allocated once for the largest step and reused by every
    step, so that a step allocates nothing and buffer addresses stay fixed."""

    def __init__(self, device, max_tokens: int):
        self.device = torch.device(device)
        self.max_tokens = max_tokens
        self._buffers: dict = {}
        self.generation = 0          # bumped whenever a buffer that `grow` handed out moves
        self._iota = None

    def get(self, name: str, rows: int, tail: tuple, dtype: torch.dtype) -> torch.Tensor:
        """A `[rows, *tail]` view of the buffer `name` (rows <= max_tokens)."""
        if rows > self.max_tokens:
            raise ValueError(f"a step of {rows} tokens exceeds the engine's max_tokens {self.max_tokens}")
        key = (name, tuple(tail), dtype)
        buf = self._buffers.get(key)
        if buf is None:
            buf = torch.zeros((self.max_tokens, *tail), dtype=dtype, device=self.device)
            self._buffers[key] = buf
        return buf[:rows]

    def raw(self, name: str, shape: tuple, dtype: torch.dtype) -> torch.Tensor:
        key = (name, tuple(shape), dtype)
        buf = self._buffers.get(key)
        if buf is None:
            buf = torch.zeros(tuple(shape), dtype=dtype, device=self.device)
            self._buffers[key] = buf
        return buf

    def grow(self, name: str, numel: int, dtype: torch.dtype) -> torch.Tensor:
        """A flat buffer of at least `numel` elements; reallocated (with headroom) when too small.
        Its address may change when it grows, so size it before a CUDA graph is captured."""
        key = (name, "grow", dtype)
        buf = self._buffers.get(key)
        if buf is None or buf.numel() < numel:
            if buf is not None:
                self.generation += 1
            buf = torch.zeros(max(numel, 1) * 3 // 2 + 16, dtype=dtype, device=self.device)
            self._buffers[key] = buf
        return buf

    def iota(self, n: int) -> torch.Tensor:
        """[0, 1, ..., n-1] int32 on the device (a view of one cached tensor)."""
        if self._iota is None or self._iota.numel() < n:
            self._iota = torch.arange(max(n, self.max_tokens), dtype=torch.int32, device=self.device)
        return self._iota[:n]

    def bytes(self) -> int:
        return sum(b.numel() * b.element_size() for b in self._buffers.values())


class ResidualStream:
    """The float32 residual `h` [n, hidden] plus, possibly, partial sums [S, n, hidden] that a
    split-K contraction left behind. The next reader (a norm, or the row gather before the
    head) adds them to `h` in ascending order of S, so the order of the sum is fixed."""

    def __init__(self, h: torch.Tensor):
        self.h = h
        self.pending: Optional[torch.Tensor] = None
        self.streams = None          # several streams side by side, where a model has them (parts/streams.py)

    def take_pending(self) -> Optional[torch.Tensor]:
        p, self.pending = self.pending, None
        return p

    def set_pending(self, partials: torch.Tensor) -> None:
        if self.pending is not None:
            self.fold()
        self.pending = partials

    def fold(self) -> None:
        """Add pending partial sums now (used by parts that want `h` itself)."""
        p = self.take_pending()
        if p is not None:      # h + (p0 + p1 + ...), the order of the kernels that fold partials themselves
            total = p[0]
            for s in range(1, p.shape[0]):
                total = total + p[s]
            self.h.add_(total)

    def add_(self, update: torch.Tensor) -> None:
        """h += update, for parts that compute their output as a separate tensor."""
        self.fold()
        self.h.add_(update.to(self.h.dtype))


@dataclass
class StepContext:
    n: int                                   # tokens in this step
    token_ids: torch.Tensor                  # [n] int32, device
    positions: torch.Tensor                  # [n] int32
    slots: torch.Tensor                      # [n] int32: the request slot of every token
    workspace: Workspace
    compute_dtype: torch.dtype
    # One record per request of the step, rows of a request being contiguous and ascending:
    entry_slots: list = field(default_factory=list)       # host ints
    entry_first_row: list = field(default_factory=list)
    entry_length: list = field(default_factory=list)
    entry_first_pos: list = field(default_factory=list)
    entry_meta: Optional[torch.Tensor] = None              # [4, E] int32 on the device: slot, first row, length, first position
    upload_ints: Optional[object] = None                   # callable(np.ndarray int32) -> device tensor, valid for this step
    sampled: Optional[torch.Tensor] = None                 # [slots] int32: each request's last sampled token (a token id of -1 reads it)
    shared: dict = field(default_factory=dict)             # what parts compute once per step and share between layers
    embedding_output: Optional[torch.Tensor] = None        # [n, hidden] float32: the embedding's rows, kept when a part reads them again
    # Set for a step that is recorded into a CUDA graph: every entry is one decoded token, the batch is
    # padded to a fixed size, and no key lies at or beyond `static_keys`. Parts must then launch the same
    # kernels with the same arguments whatever the positions are, and must not copy from the host.
    static_keys: int = 0

    @property
    def act_dtype(self) -> torch.dtype:
        return self.compute_dtype

    def tile_plan(self, group: int, tile_rows: int = 64):
        """(work list on the device, tiles, items, chunks) of the tensor-core attention kernels for this
        step: entries of at most 16 // group tokens go to the decode kernel (one item each), longer ones are
        cut into tiles of tile_rows // group positions. Made once per step and shared by all layers of this ratio."""
        key = ("attention_tc_plan", group, tile_rows)
        plan = self.shared.get(key)
        if plan is None and self.static_keys:
            E = len(self.entry_length)
            plan = (self.workspace.iota(E), 0, E, (self.static_keys + 255) // 256)
            self.shared[key] = plan
        if plan is None:
            ppt, short = tile_rows // group, 16 // group
            tiled, items, last = [], [], 0
            for e, (L, p0) in enumerate(zip(self.entry_length, self.entry_first_pos)):
                if L <= short:
                    items.append(e)
                    last = max(last, p0 + L - 1)
                else:
                    tiled += [(p0 + min(L, (t + 1) * ppt), e, t) for t in range((L + ppt - 1) // ppt)]
            # the tiles that see the most keys first: CTAs start in this order, and the short ones fill the end
            tiled.sort(key=lambda k: -k[0])
            tiles = [x for _, e, t in tiled for x in (e, t)]
            work = self.upload_ints(np.asarray(tiles + items, dtype=np.int32))
            plan = (work, len(tiles) // 2, len(items), last // 256 + 1 if items else 0)
            self.shared[key] = plan
        return plan

    @property
    def decode_only(self) -> bool:
        return all(l == 1 for l in self.entry_length)


def step_context(entries, workspace: Workspace, compute_dtype: torch.dtype, tokens=None, rows: int = 0) -> StepContext:
    """A `StepContext` for a step given as (slot, length, first position) per entry, its integer inputs in one device buffer in the step
    program's layout (tokens, positions, slots, wanted rows and entry records, each `rows` apart): what measurements and tools that drive
    single parts or operations by hand need."""
    n = sum(e[1] for e in entries)
    R = max(rows, workspace.max_tokens, n, len(entries))
    ints = torch.zeros(9 * R + 64, dtype=torch.int32)
    at = 0
    for k, (slot, length, first) in enumerate(entries):
        ints[R + at:R + at + length] = torch.arange(first, first + length, dtype=torch.int32)
        ints[2 * R + at:2 * R + at + length] = slot
        for j, v in enumerate((slot, at, length, first)):
            ints[4 * R + j * R + k] = v
        at += length
    if tokens is not None:
        ints[:n] = torch.as_tensor(tokens, dtype=torch.int32)
    d = ints.to(workspace.device)
    E = len(entries)
    return StepContext(n=n, token_ids=d[0:n], positions=d[R:R + n], slots=d[2 * R:2 * R + n], workspace=workspace, compute_dtype=compute_dtype,
                       entry_slots=[e[0] for e in entries], entry_first_row=[int(ints[5 * R + k]) for k in range(E)],
                       entry_length=[e[1] for e in entries], entry_first_pos=[e[2] for e in entries], entry_meta=d[4 * R:8 * R].view(4, R)[:, :E],
                       upload_ints=lambda values: torch.from_numpy(np.ascontiguousarray(values, dtype=np.int32)).to(workspace.device))
