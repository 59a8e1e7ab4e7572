"""Grouped-Q8 cache layout math, mirroring ``Kv_cache.Format`` / ``Kv_cache.Layout``
(lib/kv_cache.ml:1-200): the token pool stores, per token, the int8 K and V
segments of every attention layer back to back followed by one fp16 scale per
group; the checkpoint pool stores the recurrent state of every recurrent layer
the same way.  ``group_size`` is 64 in the reference (lib/kv_cache.ml:4);
32 is accepted here for inputs quantised per 32 elements.

``RowLayout`` is the unquantised counterpart (key and value vectors in the model's element type,
value heads may have a size of their own), ``matrix_state_elements`` the size of a recurrent layer's
state, and ``SequenceTable`` the owner of token slots and state rows for the live sequences."""

from __future__ import annotations

from dataclasses import dataclass
from typing import List, Sequence

Q8_GROUP_SIZE = 64


def groups_for_elements(elements: int, group_size: int = Q8_GROUP_SIZE) -> int:
    """Format.groups_for_elements, lib/kv_cache.ml:10-14."""
    if elements < 0:
        raise ValueError("KV element count cannot be negative")
    return elements // group_size + (0 if elements % group_size == 0 else 1)


def bytes_for_elements(elements: int, group_size: int = Q8_GROUP_SIZE) -> int:
    """Format.bytes_for_elements, lib/kv_cache.ml:16-22: one byte per element + 2 per group."""
    return elements + 2 * groups_for_elements(elements, group_size)


@dataclass(frozen=True)
class AttentionLayer:
    kv_heads: int
    head_dim: int

    def __post_init__(self):
        if self.kv_heads <= 0:
            raise ValueError("attention KV layer requires positive kv_heads")
        if self.head_dim <= 0:
            raise ValueError("attention KV layer requires positive head_dim")


@dataclass(frozen=True)
class AttentionRegion:
    geometry: AttentionLayer
    key_offset: int
    value_offset: int
    segment_elements: int


class Layout:
    """Layout.create_heterogeneous, lib/kv_cache.ml:84-180."""

    def __init__(self, attentions: Sequence[AttentionLayer], recurrent_layers: int = 0, recurrent_width: int = 0,
                 recurrent_window: int = 0, group_size: int = Q8_GROUP_SIZE):
        for name, value in (("recurrent_layers", recurrent_layers), ("recurrent_width", recurrent_width),
                            ("recurrent_window", recurrent_window)):
            if value < 0:
                raise ValueError(f"{name} cannot be negative")
        if recurrent_layers > 0 and (recurrent_width == 0 or recurrent_window == 0):
            raise ValueError("recurrent checkpoint layout requires positive width and window")
        self.group_size = group_size
        self.recurrent_layers = recurrent_layers
        self.recurrent_layer_elements = recurrent_width * recurrent_window
        if any(layer.head_dim % group_size for layer in attentions):
            raise ValueError("Q8 KV group_size must divide each attention head dimension")
        if recurrent_layers > 0 and self.recurrent_layer_elements % group_size:
            raise ValueError("Q8 KV group_size must divide each recurrent layer checkpoint")
        regions, offset = [], 0
        for layer in attentions:
            segment = layer.kv_heads * layer.head_dim
            regions.append(AttentionRegion(layer, offset, offset + segment, segment))
            offset += 2 * segment
        self.attentions = tuple(regions)
        self.token_elements = offset
        self.bytes_per_token = bytes_for_elements(offset, group_size)
        self.token_groups = groups_for_elements(offset, group_size)
        self.checkpoint_elements = recurrent_layers * self.recurrent_layer_elements
        self.checkpoint_groups = groups_for_elements(self.checkpoint_elements, group_size)
        self.bytes_per_checkpoint = bytes_for_elements(self.checkpoint_elements, group_size)

    def attention_key_offset(self, layer: int) -> int:
        return self.attentions[layer].key_offset

    def attention_value_offset(self, layer: int) -> int:
        return self.attentions[layer].value_offset


# ---- unquantised rows ------------------------------------------------------------------------------

@dataclass(frozen=True)
class RowRegion:
    """One attention layer's place in a token row, in elements."""

    key_offset: int
    value_offset: int


class RowLayout:
    """A token row: the K then V vectors of every attention layer, (kv_heads, dim, vdim) each; segments and
    rows start at multiples of eight elements (16 bytes of a 2-byte type)."""

    def __init__(self, attentions: Sequence[tuple]):
        align = lambda value: (value + 7) // 8 * 8
        regions, offset = [], 0
        for kv_heads, dim, vdim in attentions:
            key, value = offset, offset + align(kv_heads * dim)
            regions.append(RowRegion(key, value))
            offset = value + align(kv_heads * vdim)
        self.regions = tuple(regions)
        self.token_elements = max(offset, 8)


# value columns one thread block of the state kernels owns
MATRIX_STATE_SLICE = 32


def matrix_state_elements(heads: int, dim: int, vdim: int, *, normalized: bool) -> int:
    """fp32 elements of one sequence's state: the transposed matrices [heads][vdim][dim] and, in the
    normalised form, n [dim] and m per head and slice of value columns; a multiple of four, so that a row
    starts at a 16-byte boundary."""
    slices = (vdim + MATRIX_STATE_SLICE - 1) // MATRIX_STATE_SLICE
    elements = heads * vdim * dim + (heads * slices * (dim + 1) if normalized else 0)
    return (elements + 3) // 4 * 4


class SequenceTable:
    """Owner of what a live sequence holds: a row (of the slot table and of every state pool) and pages of
    ``page`` consecutive token slots.  Rows and pages that are given back are handed out again.  The
    table itself (u32 [rows, stride], one entry per token position) is kept here and mirrored on the
    device by the engine."""

    def __init__(self, rows: int, stride: int, slots: int, page: int = 16):
        import numpy as np

        if rows <= 0 or stride <= 0 or page <= 0 or slots < page:
            raise ValueError("a sequence table needs rows, positions and at least one page of slots")
        self.rows, self.stride, self.page = rows, stride, page
        self.table = np.zeros((rows, stride), np.uint32)
        self.lengths: List[int] = [0] * rows
        self._pages: List[List[int]] = [[] for _ in range(rows)]
        self._live: List[bool] = [False] * rows
        self._free_rows: List[int] = list(range(rows))[::-1]
        self._free_pages: List[int] = list(range(slots // page))[::-1]

    def open(self, row: int = -1) -> int:
        """A free row (or the given one) for a new sequence with nothing behind it."""
        if row < 0:
            if not self._free_rows:
                raise ValueError("no sequence row is free")
            row = self._free_rows.pop()
        else:
            if row >= self.rows or self._live[row]:
                raise ValueError("the sequence row is outside the table or in use")
            self._free_rows.remove(row)
        self._live[row], self.lengths[row] = True, 0
        return row

    def live(self, row: int) -> bool:
        return 0 <= row < self.rows and self._live[row]

    def reserve(self, row: int, tokens: int) -> range:
        """Slots for ``tokens`` more positions of a sequence; returns the table positions that changed.
        Nothing changes when they cannot be had."""
        if not self.live(row):
            raise ValueError("the sequence is not open")
        wanted = self.lengths[row] + tokens
        if wanted > self.stride:
            raise ValueError("the sequence would outgrow the cache capacity")
        have = len(self._pages[row])
        need = (wanted + self.page - 1) // self.page
        if need - have > len(self._free_pages):
            raise ValueError("the cache has no free pages")
        for index in range(have, need):
            page = self._free_pages.pop()
            self._pages[row].append(page)
            first = index * self.page
            for position in range(first, min(first + self.page, self.stride)):
                self.table[row, position] = page * self.page + position - first
        return range(min(have * self.page, self.stride), min(need * self.page, self.stride))

    def advance(self, row: int, tokens: int) -> None:
        self.lengths[row] += tokens

    def close(self, row: int) -> None:
        if not self.live(row):
            raise ValueError("the sequence is not open")
        self._free_pages.extend(reversed(self._pages[row]))
        self._pages[row], self.lengths[row], self._live[row] = [], 0, False
        self._free_rows.append(row)
