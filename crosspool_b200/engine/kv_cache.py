"""Paged KV cache (and recurrent states) of one Instance on one attention device.

Logical layer: fixed-size pages handed out by :class:`PageAllocator`; a sequence owns a list of
pages (its block table row). Physical layer: per-layer K and V buffers ``[pages, page_size,
kv_heads, head_dim]`` that are either ordinary device tensors (fixed capacity) or views over CUDA
VMM address ranges whose physical backing is mapped and unmapped in *bundles*
(:mod:`crosspool_b200.ecs.vmm`), so that co-located Instances can lend each other memory while the
tensors' addresses — and therefore captured CUDA graphs — stay valid. The allocator only hands out
pages whose bundle is mapped, like the reference's ``ElasticPageAllocator``
(src/xpool/integrations/sglang/ecs/allocator.py:61-104).

Layered decoders cache rows per token in the layers that have a cache at all, and keep one recurrent state per live
sequence (:class:`StateSlots`) in those with a recurrence (a layer can have both); they follow the sequence through the same ``ensure`` / ``release``.
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field

import torch

from ..models.config import GroupedMixer, ModelConfig, sub_mixers


class OutOfPages(RuntimeError):
    pass


class PageAllocator:
    """Free-list allocator over page ids; pages become available bundle by bundle."""

    def __init__(self, total_pages: int, pages_per_bundle: int | None = None, mapped_bundles: int | None = None):
        self.total_pages = total_pages
        self.pages_per_bundle = pages_per_bundle or total_pages
        self.num_bundles = (total_pages + self.pages_per_bundle - 1) // self.pages_per_bundle
        self._free: list[list[int]] = [[] for _ in range(self.num_bundles)]
        self._mapped = [False] * self.num_bundles
        self._used_in_bundle = [0] * self.num_bundles
        n = self.num_bundles if mapped_bundles is None else mapped_bundles
        for b in range(n):
            self.publish_bundle(b)

    # -- physical backing events -------------------------------------------------------------
    def bundle_pages(self, b: int) -> range:
        return range(b * self.pages_per_bundle, min((b + 1) * self.pages_per_bundle, self.total_pages))

    def publish_bundle(self, b: int) -> None:
        """The bundle's memory is mapped: its pages may be handed out."""
        assert not self._mapped[b]
        self._mapped[b] = True
        self._free[b] = list(reversed(self.bundle_pages(b)))
        self._used_in_bundle[b] = 0

    def empty_bundles(self) -> list[int]:
        return [b for b in range(self.num_bundles) if self._mapped[b] and self._used_in_bundle[b] == 0]

    def begin_retirement(self, b: int) -> None:
        """Takes an empty bundle out of circulation (it may be unmapped once in-flight work that
        could still read it has finished)."""
        if not self._mapped[b] or self._used_in_bundle[b] != 0:
            raise ValueError(f"bundle {b} is not an empty mapped bundle")
        self._mapped[b] = False
        self._free[b] = []

    def mapped_bundles(self) -> list[int]:
        return [b for b in range(self.num_bundles) if self._mapped[b]]

    def used_in_bundle(self, b: int) -> int:
        return self._used_in_bundle[b]

    def unmapped_bundles(self) -> list[int]:
        return [b for b in range(self.num_bundles) if not self._mapped[b]]

    # -- page hand-out -----------------------------------------------------------------------
    @property
    def free_pages(self) -> int:
        return sum(len(f) for f in self._free)

    @property
    def mapped_pages(self) -> int:
        return sum(len(self.bundle_pages(b)) for b in range(self.num_bundles) if self._mapped[b])

    def alloc(self, n: int) -> list[int]:
        if n > self.free_pages:
            raise OutOfPages(f"need {n} pages, {self.free_pages} free")
        out: list[int] = []
        # fill the fullest bundles first so that lightly used ones drain and can be lent away
        order = sorted((b for b in range(self.num_bundles) if self._free[b]),
                       key=lambda b: (-self._used_in_bundle[b], b))
        for b in order:
            while self._free[b] and len(out) < n:
                out.append(self._free[b].pop())
                self._used_in_bundle[b] += 1
            if len(out) == n:
                break
        return out

    def free(self, pages: list[int]) -> None:
        for p in pages:
            b = p // self.pages_per_bundle
            self._used_in_bundle[b] -= 1
            if self._mapped[b]:
                self._free[b].append(p)


class StateSlots:
    """Hands out the slots of per-sequence recurrent states. A slot is not cleared when it changes hands: the kernels start
    a sequence whose first token sits at position 0 from a zero state."""

    def __init__(self, n: int):
        self.total = n
        self._free = list(range(n - 1, -1, -1))

    @property
    def free_slots(self) -> int:
        return len(self._free)

    def alloc(self) -> int:
        if not self._free:
            raise OutOfPages("no free state slot")
        return self._free.pop()

    def free(self, slot: int) -> None:
        self._free.append(slot)


@dataclass
class KvLayout:
    page_size: int
    num_pages: int
    kv_heads: int
    head_dim: int
    num_layers: int
    elem_bytes: int = 2
    row_widths: tuple[int, ...] = ()   # layered decoders: elements of one token's row per layer (0: the layer caches none)
    pool_elems: int = 0                # block means beside one page, all layers

    @property
    def page_bytes_per_buffer(self) -> int:
        return self.page_size * self.kv_heads * self.head_dim * self.elem_bytes

    @property
    def buffer_bytes(self) -> int:
        return self.num_pages * self.page_bytes_per_buffer

    @property
    def bytes_per_page_all_layers(self) -> int:
        if self.row_widths:
            return (self.page_size * sum(self.row_widths) + self.pool_elems) * self.elem_bytes
        return 2 * self.num_layers * self.page_bytes_per_buffer


@dataclass
class PagedKvCache:
    layout: KvLayout
    k: list[torch.Tensor]
    v: list[torch.Tensor]
    allocator: PageAllocator
    backing: object | None = None  # ecs.vmm.KvVmmBacking when elastic
    tables: dict[int, list[int]] = field(default_factory=dict)
    # recurrent layers: fp32 [slots, *state_shape of the mixer] per layer (None elsewhere), and the slot of every live sequence
    states: list[torch.Tensor | None] = field(default_factory=list)
    # convolution inputs behind every live sequence, [slots, taps, channels] per layer: the input at position p is entry p % taps
    conv: list[torch.Tensor | None] = field(default_factory=list)
    # layers that pool: means of keys and of values of whole token blocks, [pages, rows beside a page, kv heads, head]; the blocks of
    # a sequence fill the rows beside its pages in order
    k_pool: list[torch.Tensor | None] = field(default_factory=list)
    v_pool: list[torch.Tensor | None] = field(default_factory=list)
    slots: StateSlots | None = None
    seq_slots: dict[int, int] = field(default_factory=dict)

    @classmethod
    def fixed(cls, cfg: ModelConfig, num_pages: int, page_size: int = 16, device="cuda",
              dtype: torch.dtype = torch.bfloat16, state_slots: int = 0) -> "PagedKvCache":
        if cfg.layered:
            return cls._layered(cfg, num_pages, page_size, device, dtype, state_slots)
        lay = KvLayout(page_size, num_pages, cfg.num_kv_heads, cfg.head_dim, cfg.num_layers, dtype.itemsize)
        shape = (num_pages, page_size, cfg.num_kv_heads, cfg.head_dim)
        k = [torch.zeros(shape, dtype=dtype, device=device) for _ in range(cfg.num_layers)]
        v = [torch.zeros(shape, dtype=dtype, device=device) for _ in range(cfg.num_layers)]
        return cls(lay, k, v, PageAllocator(num_pages))

    @classmethod
    def _layered(cls, cfg: ModelConfig, num_pages: int, page_size: int, device, dtype: torch.dtype, state_slots: int) -> "PagedKvCache":
        """Pages hold a key row and a value row per token in the layers that cache any (or one latent row that is both); a layer
        may read another one's instead, and layers that pool hold the means of token blocks beside them. Recurrent mixers hold one
        state per slot, and mixers with a convolution its latest inputs."""
        mixers = [s.mixer for s in cfg.layer_specs]
        pools = [m.pool_shapes(page_size) if isinstance(m, GroupedMixer) else () for m in mixers]
        lay = KvLayout(page_size, num_pages, 1, 0, cfg.num_layers, dtype.itemsize, tuple(m.cache_width for m in mixers),
                       sum(math.prod(shape) for p in pools for shape in p))

        def rows(m, i: int) -> torch.Tensor | None:
            if len(m.cache_rows) <= i:
                return None
            return torch.zeros(num_pages, page_size, *m.cache_rows[i], dtype=dtype, device=device)

        states, conv = [None] * len(mixers), [None] * len(mixers)
        for l, m in enumerate(mixers):
            for sub in sub_mixers(m):
                if sub.state_elems:
                    states[l] = torch.zeros(state_slots, *sub.state_shape, dtype=torch.float32, device=device)
                if getattr(sub, "conv", 0):
                    conv[l] = torch.zeros(state_slots, sub.conv, sub.conv_channels, dtype=dtype, device=device)
        k, v = [rows(m, 0) for m in mixers], [rows(m, 1) for m in mixers]
        for l, m in enumerate(mixers):
            if getattr(m, "kv_from", None) is not None:
                k[l], v[l] = k[m.kv_from], v[m.kv_from]
        k_pool, v_pool = ([torch.zeros(num_pages, *p[i], dtype=dtype, device=device) if p else None for p in pools] for i in (0, 1))
        return cls(lay, k, v, PageAllocator(num_pages), states=states, conv=conv, k_pool=k_pool, v_pool=v_pool,
                   slots=StateSlots(state_slots) if cfg.recurrent else None)

    # -- per-sequence page tables --------------------------------------------------------------
    def pages_needed(self, seq_id: int, new_len: int) -> int:
        have = len(self.tables.get(seq_id, ()))
        need = (new_len + self.layout.page_size - 1) // self.layout.page_size
        return max(0, need - have)

    def ensure(self, seq_id: int, new_len: int) -> list[int]:
        """Grows the sequence's table to cover ``new_len`` tokens."""
        n = self.pages_needed(seq_id, new_len)
        if n and n > self.allocator.free_pages:
            raise OutOfPages(f"need {n} pages, {self.allocator.free_pages} free")
        if self.slots is not None and seq_id not in self.seq_slots:
            self.seq_slots[seq_id] = self.slots.alloc()
        t = self.tables.setdefault(seq_id, [])
        if n:
            t.extend(self.allocator.alloc(n))
        return t

    def release(self, seq_id: int) -> None:
        t = self.tables.pop(seq_id, None)
        if t:
            self.allocator.free(t)
        slot = self.seq_slots.pop(seq_id, None)
        if slot is not None:
            self.slots.free(slot)

    def slot(self, seq_id: int, pos: int) -> int:
        t = self.tables[seq_id]
        return t[pos // self.layout.page_size] * self.layout.page_size + pos % self.layout.page_size
