"""From what each cache layer needs to groups, and from groups to device tensors.

A mixer declares what its cache layer needs with a :class:`KVLayerSpec` (paged
keys and values, optionally only a window of them) or a :class:`StateLayerSpec`
(a fixed-size slot per request).  Layers with the same needs form one group; a
paged group has one page pool and one block table per request for all its
layers, so one page id addresses that page in every layer of the group
(as in qwen3_runtime/kv/paged.py:63-72, where the only group is "all layers").

Device layout of a paged key/value group: ``[layers, 2 (K,V), pages + 1, kv_heads,
page_size, head_dim]`` -- per (page, head) a contiguous ``[page_size, head_dim]``
tile, so one key/value tile of a head is a single contiguous read.  The extra
last page is a scratch page that padded rows of a captured decode step write to.
"""

from __future__ import annotations

from dataclasses import dataclass

from .manager import GroupSpec


@dataclass(frozen=True)
class KVLayerSpec:
    """``value_dim``: values have a size of their own (None: the keys' ``head_dim``); keys and values
    are then two device tensors, ``[layers, pages + 1, kv_heads, page_size, head_dim | value_dim]``.
    ``keep_first``: with a window, the sequence's first ``keep_first`` tokens stay readable as well.
    ``chunk``: a token reads only the keys of its own chunk of that many tokens (counted from the sequence's
    first token); pages wholly before the current chunk are given back.  A tuple of chunk sizes: several layers read
    this one's keys, each under chunks of its own; a page is given back when none of them needs it any more."""

    num_kv_heads: int
    head_dim: int
    window: int | None = None
    value_dim: int | None = None
    keep_first: int = 0
    chunk: int | tuple[int, ...] | None = None

    @property
    def split(self) -> bool:
        return self.value_dim is not None and self.value_dim != self.head_dim


def flatten_specs(spec) -> list:
    """A mixer may need several cache layers at once (pages for keys and values beside a state slot,
    two mixers side by side): its spec is then a tuple of specs, possibly nested.  The leaves in
    order."""
    if isinstance(spec, (tuple, list)):
        return [leaf for part in spec for leaf in flatten_specs(part)]
    return [spec]


@dataclass(frozen=True)
class LatentLayerSpec:
    """One row of ``width`` elements per token, shared by all heads (a compressed key/value
    latent, possibly followed by a shared rotated key part), optionally only a window of rows.
    Device layout of such a group: ``[layers, pages + 1, page_size, width]``."""

    width: int
    window: int | None = None


@dataclass(frozen=True)
class StateLayerSpec:
    shape: tuple[int, ...]
    dtype: str = "float32"


def kept_for_readers(cache_id, own, others: list):
    """The spec of cache layer ``cache_id`` that its writer (``own``) and further layers (``others``) read.  They agree
    on heads and sizes; where their masks differ, what any of them may still read is kept."""
    if all(spec == own for spec in others):
        return own
    specs = [own, *others]
    if (not all(isinstance(s, KVLayerSpec) for s in specs)
            or any((s.num_kv_heads, s.head_dim, s.value_dim or s.head_dim)
                   != (own.num_kv_heads, own.head_dim, own.value_dim or own.head_dim) for s in specs)):
        raise ValueError(f"a run entry reads cache layer {cache_id} whose layout differs from its own")
    window = chunk = None
    keep_first = 0
    if all(s.chunk for s in specs):
        chunk = tuple(sorted({c for s in specs for c in (s.chunk if isinstance(s.chunk, tuple) else (s.chunk,))}))
        chunk = chunk[0] if len(chunk) == 1 else chunk
    elif all(s.window for s in specs):
        window, keep_first = max(s.window for s in specs), max(s.keep_first for s in specs)
    return KVLayerSpec(own.num_kv_heads, own.head_dim, window, value_dim=own.value_dim, keep_first=keep_first, chunk=chunk)


@dataclass(frozen=True)
class GroupLayout:
    spec: GroupSpec
    layer_spec: object  # KVLayerSpec | StateLayerSpec
    cache_ids: tuple  # cache layers of this group, in order (ids, or (id, leaf) of a composite spec)


class CacheLayout:
    """Groups for a model: ``layer_specs`` maps cache layer id -> its spec (or None).  A spec that is
    a tuple (see :func:`flatten_specs`) stands for several cache layers: leaf ``k`` of cache layer
    ``c`` is kept under the id ``(c, k)``, and ``composite[c]`` is the tuple itself, so that the
    storage can hand the mixer its views in the same arrangement."""

    def __init__(self, layer_specs: dict[int, object]):
        buckets: dict[object, list] = {}
        self.composite: dict[int, object] = {}
        for cache_id in sorted(layer_specs):
            spec = layer_specs[cache_id]
            if spec is None:
                continue
            if isinstance(spec, (tuple, list)):
                self.composite[cache_id] = spec
                for k, leaf in enumerate(flatten_specs(spec)):
                    if leaf is not None:
                        buckets.setdefault(leaf, []).append((cache_id, k))
                continue
            buckets.setdefault(spec, []).append(cache_id)
        self.groups: list[GroupLayout] = []
        for spec, ids in buckets.items():
            if isinstance(spec, (KVLayerSpec, LatentLayerSpec)):
                if spec.window:
                    gs = GroupSpec("window", spec.window, getattr(spec, "keep_first", 0))
                elif getattr(spec, "chunk", None):
                    gs = GroupSpec("chunk", chunk=spec.chunk)
                else:
                    gs = GroupSpec("full")
            elif isinstance(spec, StateLayerSpec):
                gs = GroupSpec("state")
            else:
                raise TypeError(f"unknown cache layer spec {spec!r}")
            self.groups.append(GroupLayout(gs, spec, tuple(ids)))
        if not any(g.spec.paged for g in self.groups):
            # a model without paged layers still gets block tables of width zero
            pass
        self.where: dict[int, tuple[int, int]] = {}
        for gi, g in enumerate(self.groups):
            for li, cache_id in enumerate(g.cache_ids):
                self.where[cache_id] = (gi, li)
        self.paged_groups = [gi for gi, g in enumerate(self.groups) if g.spec.paged]

    @property
    def group_specs(self) -> list[GroupSpec]:
        return [g.spec for g in self.groups]

    def page_bytes(self, page_size: int, dtype_bytes: int) -> list[int]:
        """Bytes of one page (all layers, K and V) for each paged group."""
        out = []
        for gi in self.paged_groups:
            g = self.groups[gi]
            s = g.layer_spec
            if isinstance(s, LatentLayerSpec):
                out.append(len(g.cache_ids) * s.width * page_size * dtype_bytes)
            else:
                per_token = s.num_kv_heads * (s.head_dim + (s.value_dim or s.head_dim))
                out.append(len(g.cache_ids) * per_token * page_size * dtype_bytes)
        return out

    def token_bytes(self, dtype_bytes: int) -> int:
        """Bytes of keys and values one token adds over all paged groups
        (qwen3_runtime/engine/memory.py:8-10)."""
        return sum(self.page_bytes(1, dtype_bytes))

    def pages_for_budget(self, budget_bytes: int, page_size: int, dtype_bytes: int, *,
                         max_num_seqs: int | None = None, max_step_tokens: int | None = None) -> list[int]:
        """Pages for each paged group that together fit in ``budget_bytes``
        (qwen3_runtime/engine/memory.py:17-27 for the single group of the reference).

        A group that keeps every key needs pages in proportion to the tokens held, so such
        groups all get the same count.  A window group never holds more, per request, than
        its window plus the portion being computed; with ``max_num_seqs`` and
        ``max_step_tokens`` given it gets no more pages than that, and what it leaves goes to
        the groups that keep everything."""
        per = self.page_bytes(page_size, dtype_bytes)
        if not per or sum(per) <= 0:
            return [0 for _ in per]
        equal = int(budget_bytes // sum(per))
        counts = [equal] * len(per)
        if max_num_seqs is None or max_step_tokens is None:
            return counts
        spent, open_bytes = 0, 0
        for i, gi in enumerate(self.paged_groups):
            window = self.groups[gi].spec.reach  # the most keys a request holds
            if window:
                kept = -(-self.groups[gi].spec.keep_first // page_size)
                cap = max_num_seqs * (-(-(window + max_step_tokens) // page_size) + 2 + kept)
                counts[i] = min(equal, cap)
                spent += counts[i] * per[i]
            else:
                open_bytes += per[i]
        if open_bytes:
            full = int((budget_bytes - spent) // open_bytes)
            counts = [c if self.groups[gi].spec.reach else full
                      for c, gi in zip(counts, self.paged_groups)]
        return counts
