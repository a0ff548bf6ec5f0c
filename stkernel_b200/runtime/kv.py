"""Hybrid paged KV manager.

Several cache *groups* share one page-id space per group kind:

* ``swa``   — every layer's sliding-window latent cache (64-token pages).  Only the
  pages that still intersect a request's window are kept; older ones are released
  as the request advances, so SWA memory is O(window), not O(context).
* ``c4``    — compressed latent cache + indexer-K cache of every ratio-4 layer
  (one row per 4 tokens).
* ``c128``  — compressed latent cache of every ratio-128 layer.
* compressor *state* rows (raw value/gate rows of the open window) live in a
  dense per-request-row tensor owned by each layer.

Each group has a free list and a per-request block table row
(``[max_requests, max_pages]`` int32, -1 = no page) that lives on the device at a
fixed address, so captured CUDA graphs keep working while tables change.
This is the engine-side counterpart of the KV specs and slot mappings the
reference builds on (overlay/attention.py:743-759,836-849,
overlay/sparse_swa_dsv4.py:87-111).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Tuple

import torch

from ..config import FULL_CONTEXT, HybridConfig, ModelConfig, attention_part, recurrent_part
from ..ops.cache import PAGE, PagedCache
from ..ops.grouped import grouped_row
from ..ops.latent import latent_row
from ..ops.shifted import shift_state
from ..ops.talking import talking_row
from .planning import dcp_owner


class OutOfPages(RuntimeError):
    pass


@dataclass
class GroupTable:
    """Free list + device block table of one cache group."""
    name: str
    num_pages: int
    max_requests: int
    max_pages_per_req: int
    device: torch.device
    rows_per_token: float            # 1 for swa, 1/ratio for compressed groups
    # Decode context parallel: logical page lp of every request is stored by rank lp % dcp_size only.  The other
    # ranks map it to one shared scratch page past the pool (`trash`), so kernels that write a compressed row through
    # the table need no owner test, and nothing ever reads that page.
    dcp_rank: int = 0
    dcp_size: int = 1
    table_host: torch.Tensor = field(init=False)
    table_dev: torch.Tensor = field(init=False)
    free: List[int] = field(init=False)
    dirty: bool = field(default=True, init=False)
    on_pressure: Optional[Callable[[], bool]] = field(default=None, init=False)

    def __post_init__(self) -> None:
        self.table_host = torch.full((self.max_requests, self.max_pages_per_req), -1, dtype=torch.int32)
        if self.device.type == "cuda":
            self.table_host = self.table_host.pin_memory()
        self.table_np = self.table_host.numpy()          # host truth; never read by an async copy
        # upload snapshots: the DMA of step k may run while the host already edits the table for step
        # k+1, so rows are copied into one of two pinned snapshots and uploaded from there
        self.snap = [torch.full_like(self.table_host, -1) for _ in range(2)]
        if self.device.type == "cuda":
            self.snap = [t.pin_memory() for t in self.snap]
        self.snap_np = [t.numpy() for t in self.snap]
        self.table_dev = torch.full((self.max_requests, self.max_pages_per_req), -1, dtype=torch.int32,
                                    device=self.device)
        self.free = list(range(self.num_pages - 1, -1, -1))
        # owners per physical page: a request row, and any number of prefix-cache entries sharing it
        self.ref = [0] * self.num_pages
        # resident logical pages of each row form one interval [lo, hi)
        self.lo = [0] * self.max_requests
        self.hi = [0] * self.max_requests
        self.dirty_rows = set()
        self.trash = self.num_pages if self.dcp_size > 1 else -2          # physical id of the scratch page

    def owns(self, logical: int) -> bool:
        return self.dcp_size == 1 or dcp_owner(logical * PAGE, self.dcp_size, PAGE) == self.dcp_rank

    def local_table(self) -> torch.Tensor:
        """[max_requests, ceil(max_pages / dcp)] block table over this rank's own pages only: column l is logical
        page l * dcp_size + dcp_rank.  Row r of that local numbering is global row
        ((r // PAGE) * dcp_size + dcp_rank) * PAGE + r % PAGE."""
        return self.table_dev[:, self.dcp_rank::self.dcp_size].contiguous()

    def ensure(self, row: int, first_logical: int, last_logical: int) -> None:
        """Make logical pages [first, last] of request `row` resident (the resident set stays an interval)."""
        if last_logical >= self.max_pages_per_req:
            raise OutOfPages(f"{self.name}: request needs logical page {last_logical} >= {self.max_pages_per_req}")
        first_logical = max(first_logical, 0)
        if self.hi[row] == self.lo[row]:
            self.lo[row] = self.hi[row] = first_logical
        t = self.table_np[row]
        start = max(self.hi[row], first_logical)
        if first_logical < self.lo[row]:
            raise OutOfPages(f"{self.name}: page {first_logical} of row {row} was already released")
        for lp in range(start, last_logical + 1):
            if self.owns(lp):
                while not self.free and self.on_pressure is not None and self.on_pressure():
                    pass                                   # cached prefixes give pages back, oldest first
                if not self.free:
                    # the pages taken so far stay with the row (the interval below covers them): nothing leaks
                    raise OutOfPages(f"{self.name}: pool of {self.num_pages} pages exhausted")
                t[lp] = self.free.pop()
                self.ref[int(t[lp])] = 1
            else:
                t[lp] = self.trash
            self.hi[row] = lp + 1
            self.dirty = True
            self.dirty_rows.add(row)

    def release_before(self, row: int, logical: int) -> None:
        t = self.table_np[row]
        end = min(max(logical, 0), self.hi[row])
        for lp in range(self.lo[row], end):
            self.unref(int(t[lp]))
            t[lp] = -1
        if end > self.lo[row]:
            self.lo[row] = end
            self.dirty = True
            self.dirty_rows.add(row)

    def unref(self, page: int) -> None:
        if page == self.trash:
            return
        self.ref[page] -= 1
        if self.ref[page] == 0:
            self.free.append(page)

    def share(self, row: int, first_logical: int, last_logical: int) -> List[int]:
        """Physical pages of logical pages [first, last] of `row`, each with one more owner."""
        t = self.table_np[row]
        pages = [int(t[lp]) for lp in range(first_logical, last_logical + 1)]
        if any(pg < 0 for pg in pages):
            raise OutOfPages(f"{self.name}: cannot share a page that is not resident")
        for pg in pages:
            if pg != self.trash:
                self.ref[pg] += 1
        return pages

    def adopt(self, row: int, first_logical: int, pages: List[int]) -> None:
        """Map shared physical pages as logical pages [first, first + len) of an empty row."""
        assert self.hi[row] == self.lo[row], "adopt needs a row without resident pages"
        t = self.table_np[row]
        for i, pg in enumerate(pages):
            t[first_logical + i] = pg
            if pg != self.trash:
                self.ref[pg] += 1
        self.lo[row], self.hi[row] = first_logical, first_logical + len(pages)
        self.dirty = True
        self.dirty_rows.add(row)

    def release_all(self, row: int) -> None:
        self.release_before(row, self.max_pages_per_req)
        self.lo[row] = self.hi[row] = 0

    def sync(self, parity: int = 0) -> None:
        """Upload the rows that changed since the last step (through pinned snapshot `parity`, which
        the caller guarantees is no longer being read by an earlier upload)."""
        if self.dirty:
            snap, snap_np = self.snap[parity], self.snap_np[parity]
            if len(self.dirty_rows) * 4 >= self.max_requests:
                snap_np[:] = self.table_np
                self.table_dev.copy_(snap, non_blocking=True)
            else:
                for r in self.dirty_rows:
                    snap_np[r] = self.table_np[r]
                    self.table_dev[r].copy_(snap[r], non_blocking=True)
            self.dirty_rows.clear()
            self.dirty = False

    @property
    def pages_in_use(self) -> int:
        return self.num_pages - len(self.free)

    def held(self, row: int) -> int:
        """Pool pages behind the resident logical pages of `row` (with context parallelism: this rank's only)."""
        n, r = self.dcp_size, self.dcp_rank
        below = lambda x: (x - r + n - 1) // n if x > r else 0         # logical pages < x that this rank stores
        return below(self.hi[row]) - below(self.lo[row])


class CacheManager:
    """What the scheduler and the engine ask of any model family's caches: request rows, page groups, admission."""

    def __init__(self, device, max_requests: int):
        self.device = torch.device(device)
        self.max_requests = max_requests
        self.free_rows = list(range(max_requests - 1, -1, -1))
        # context tokens promised to admitted requests, in whatever unit the family's admission counts (pages)
        self.reserved: Dict[int, int] = {}

    def groups(self) -> List[GroupTable]:
        raise NotImplementedError

    def alloc_row(self) -> int:
        if not self.free_rows:
            raise OutOfPages("no free request row")
        return self.free_rows.pop()

    def free_row(self, row: int) -> None:
        for g in self.groups():
            g.release_all(row)
        self.reserved.pop(row, None)
        self.free_rows.append(row)

    def sync(self, parity: int = 0) -> None:
        for g in self.groups():
            g.sync(parity)

    def reserve(self, row: int, context: int) -> None:
        """Promise request `row` room for a context of `context` tokens."""

    def prepare(self, row: int, start_pos: int, n_tokens: int, lookback: Optional[int] = None) -> None:
        """Make resident what a step that appends positions [start, start+n) to request `row` touches."""
        raise NotImplementedError

    def fits(self, context: int) -> bool:
        """Whether a request of this context could ever be admitted."""
        return True

    def can_admit(self, n_tokens: int, context: int) -> bool:
        raise NotImplementedError

    def usage(self) -> float:
        """Share of the pages in use (the gauge of the serving metrics)."""
        raise NotImplementedError


class KVManager(CacheManager):
    """Owns the group tables, the per-layer cache tensors and the request-row allocator."""

    def __init__(self, cfg: ModelConfig, device, max_requests: int, max_model_len: int, swa_pages: int,
                 c4_pages: int, c128_pages: int = 0, max_chunk: int = 4096, layers: Optional[List[int]] = None,
                 extra_swa_layers: int = 0, spec_tokens: int = 0, dcp_rank: int = 0, dcp_size: int = 1):
        """dcp_size > 1: the ratio-4 caches (compressed latent rows and indexer keys, the part of the KV that grows
        with the context) are dealt page by page over the ranks; `c4_pages` is then this rank's pool.  The
        sliding-window and ratio-128 caches stay replicated (a window, and 1/32 of the ratio-4 rows)."""
        super().__init__(device, max_requests)
        self.cfg = cfg
        self.dcp_rank, self.dcp_size = dcp_rank, dcp_size
        fp8 = cfg.kv_cache_dtype == "fp8_ds_mla"
        D, Rd = cfg.head_dim, cfg.qk_rope_head_dim
        # the block table spans the whole context; SWA residency is bounded by window + chunk
        pages_ctx = (max_model_len + PAGE - 1) // PAGE + 1
        self.swa = GroupTable("swa", swa_pages, max_requests, pages_ctx, self.device, 1.0)
        self.c4 = GroupTable("c4", max(c4_pages, 1), max_requests, (max_model_len // 4) // PAGE + 2, self.device, 0.25,
                             dcp_rank, dcp_size)
        self.c128 = GroupTable("c128", max(c128_pages, 1), max_requests, (max_model_len // 128) // PAGE + 2,
                               self.device, 1 / 128)
        self.layers = layers if layers is not None else list(range(cfg.num_hidden_layers))
        self.model_has_c4 = any(cfg.layer_kind(l) == "c4a" for l in range(cfg.num_hidden_layers))
        self.model_has_c128 = any(cfg.layer_kind(l) == "c128a" for l in range(cfg.num_hidden_layers))
        self.swa_cache: Dict[int, PagedCache] = {}
        self.comp_cache: Dict[int, PagedCache] = {}
        self.idx_cache: Dict[int, PagedCache] = {}
        self.comp_state: Dict[int, torch.Tensor] = {}
        self.idx_state: Dict[int, torch.Tensor] = {}
        n_total = cfg.num_hidden_layers + extra_swa_layers
        # Speculative verification writes up to `spec_tokens` raw compressor rows past the accepted
        # prefix; the rings are widened so that those writes never land on a row that a window
        # closing after the rollback still needs.
        ring4 = 8 if spec_tokens == 0 else 32
        ring128 = 128 if spec_tokens == 0 else 160
        for li in list(self.layers) + list(range(cfg.num_hidden_layers, n_total)):
            self.swa_cache[li] = PagedCache.allocate(swa_pages, D, Rd, fp8, "latent", self.device)
            kind = cfg.layer_kind(li) if li < cfg.num_hidden_layers else "swa"
            if kind == "c4a":
                n4 = self.c4.num_pages + (1 if dcp_size > 1 else 0)          # + the scratch page
                self.comp_cache[li] = PagedCache.allocate(n4, D, Rd, fp8, "latent", self.device)
                self.idx_cache[li] = PagedCache.allocate(n4, cfg.index_head_dim, Rd, fp8, "indexer", self.device,
                                                         fp4=cfg.indexer_dtype == "mxfp4")
                self.comp_state[li] = torch.zeros(max_requests, ring4, 2 * 2 * D, dtype=torch.float32, device=self.device)
                self.idx_state[li] = torch.zeros(max_requests, ring4, 2 * 2 * cfg.index_head_dim, dtype=torch.float32,
                                                 device=self.device)
            elif kind == "c128a":
                self.comp_cache[li] = PagedCache.allocate(self.c128.num_pages, D, Rd, fp8, "latent", self.device)
                self.comp_state[li] = torch.zeros(max_requests, ring128, 2 * D, dtype=torch.float32, device=self.device)
        self.spec_tokens = spec_tokens
        # `reserved` holds the ratio-4 pages promised to admitted requests for their whole context (allocated page by
        # page as they grow): admission counts the part not yet allocated as taken, so a pool smaller than
        # max_requests x max_model_len makes requests wait instead of running out of pages in the middle of a step

    # ---- request rows -------------------------------------------------------
    def groups(self) -> List[GroupTable]:
        return [self.swa, self.c4, self.c128]

    def reserve(self, row: int, context: int) -> None:
        """Promise request `row` the ratio-4 pages of a context of `context` tokens."""
        self.reserved[row] = self.admit_needs(0, context)[1]

    def promised(self) -> int:
        """Ratio-4 pages promised to running requests and not allocated yet."""
        return sum(max(0, need - self.c4.held(row)) for row, need in self.reserved.items())

    # ---- per-step residency ---------------------------------------------------
    def prepare(self, row: int, start_pos: int, n_tokens: int, lookback: Optional[int] = None) -> None:
        """Make resident what a step that appends positions [start, start+n) to request `row` touches,
        and release SWA pages that have left the window."""
        cfg = self.cfg
        W = cfg.sliding_window if lookback is None else lookback
        end = start_pos + n_tokens                 # exclusive
        lo = max(0, start_pos - W + 1)
        self.swa.release_before(row, lo // PAGE)
        self.swa.ensure(row, lo // PAGE, (end - 1) // PAGE)
        # by the kinds of the whole model, not of this pipeline stage's layers: every stage keeps the same tables, so
        # their schedulers and prefix caches decide alike
        if self.model_has_c4:
            n_rows = end // 4
            if n_rows > 0:
                self.c4.ensure(row, 0, (n_rows - 1) // PAGE)
        if self.model_has_c128:
            n_rows = end // 128
            if n_rows > 0:
                self.c128.ensure(row, 0, (n_rows - 1) // PAGE)

    def admit_needs(self, n_tokens: int, context: int) -> Tuple[int, int]:
        """(sliding-window pages, ratio-4 pages) a new request of this size must find free."""
        c4 = ((context + (2 * self.spec_tokens + 1 if self.spec_tokens else 0)) // 4) // PAGE + 1
        return (min(n_tokens, context) + self.cfg.sliding_window) // PAGE + 2, -(-c4 // self.dcp_size)

    def fits(self, context: int) -> bool:
        """Whether a request of this context could ever be admitted (its ratio-4 pages fit the whole pool)."""
        return self.admit_needs(0, context)[1] <= self.c4.num_pages

    def can_admit(self, n_tokens: int, context: int) -> bool:
        need_swa, need_c4 = self.admit_needs(n_tokens, context)
        return (bool(self.free_rows) and len(self.swa.free) >= need_swa
                and len(self.c4.free) - self.promised() >= need_c4)

    def usage(self) -> float:
        return self.c4.pages_in_use / max(1, self.c4.num_pages)

    def bytes_allocated(self) -> int:
        n = 0
        for d in (self.swa_cache, self.comp_cache, self.idx_cache):
            n += sum(c.buf.numel() for c in d.values())
        for d in (self.comp_state, self.idx_state):
            n += sum(t.numel() * 4 for t in d.values())
        return n


class HybridKVManager(CacheManager):
    """Caches of a decoder described layer by layer (`HybridConfig`).

    * attention layers: paged rows, one page group per distinct window (layers of the same window share the block table).
      A page holds `[kv_heads, PAGE, row]`; a row is the projected key followed by the rotated copy of its first
      `rot_dims` dimensions, padded to 16 bytes.  The projected key is the value, and with its rotated head replaced it is
      the key, so nothing is stored twice.  Pages are released as they leave the window.
    * latent-attention layers: paged rows of one latent and one rotated key part (`ops/latent.py`), in the page group of the
      full context, whose pages stay until the request ends.  A layer that attends over another layer's latents has none.
    * grouped-attention layers: paged rows `[kv_heads, PAGE, row]` of value and key (`ops/grouped.py`), in the full-context group.
    * mLSTM layers: per request row the matrix memory `[heads, dim, vdim]`, the normaliser `[heads, dim]` and the running
      maximum `[heads]`, fp32.  Nothing is cleared when a row changes hands: a span that starts at position 0 reads zeros.
    * talking-heads attention: paged rows `[PAGE, row]` of all heads' values and keys (`ops/talking.py`).  Chunks of n positions use the
      page group of a window of n, which holds whatever a chunk can see.
    * time-mixing layers: the matrix state as for retention.  "shifted" blocks: per request row the last token, and per layer the last
      norm output and shifted row (`ops/shifted.py`).
    * retention and Mamba-2 layers: per request row the matrix state `[heads, dim, vdim]` in fp32, and for Mamba-2 the last inputs
      of the convolution `[taps - 1, channels]` as projected (position p at p mod taps - 1); not cleared either.

    A parallel mixer's two sides have their cache and state under the same layer.

    pool_tokens caps the full-context group at this many tokens over all requests together; admission then promises every
    request the pages of its whole context and makes others wait.
    """

    def __init__(self, cfg: HybridConfig, device, max_requests: int, max_model_len: int, max_chunk: int,
                 extra_pages: int = 0, pool_tokens: Optional[int] = None):
        super().__init__(device, max_requests)
        self.cfg = cfg
        dt = torch.float32 if cfg.dtype == "float32" else torch.bfloat16
        self.max_model_len = max_model_len
        pages_ctx = (max_model_len + PAGE - 1) // PAGE + 1
        self.by_window: Dict[int, GroupTable] = {}
        for w in cfg.windows():
            pages = hybrid_pool_pages(w, max_requests, max_model_len, max_chunk) + extra_pages
            name = f"window{w}"
            if w >= FULL_CONTEXT:
                name = "full"
                if pool_tokens is not None:
                    pages = min(pages, max(-(-pool_tokens // PAGE), pages_ctx))
            self.by_window[w] = GroupTable(name, pages, max_requests, pages_ctx, self.device, 1.0)
        self.full = self.by_window.get(FULL_CONTEXT)
        self.kv_cache: Dict[int, torch.Tensor] = {}
        self.state: Dict[int, Tuple[torch.Tensor, ...]] = {}
        for li, l in enumerate(cfg.layers):
            m, r = attention_part(l.mixer), recurrent_part(l.mixer)
            if m is not None and m.kind == "attention":
                g = self.by_window[m.window]
                self.kv_cache[li] = torch.zeros(g.num_pages, m.kv_heads, PAGE, kv_row_width(m.dim, m.rot_dims), dtype=dt,
                                                device=self.device)
            elif m is not None and m.kind == "grouped_attention":
                self.kv_cache[li] = torch.zeros(self.full.num_pages, m.kv_heads, PAGE, grouped_row(m.dim, m.vdim)[0], dtype=dt,
                                                device=self.device)
            elif m is not None and m.kind == "talking_attention":
                g = self.by_window[m.window]
                self.kv_cache[li] = torch.zeros(g.num_pages, PAGE, talking_row(m.kv_heads, m.dim, m.vdim)[0], dtype=dt, device=self.device)
            elif m is not None and m.kv_from is None:
                self.kv_cache[li] = torch.zeros(self.full.num_pages, PAGE, latent_row(m.kv_rank, m.rot_dim)[0], dtype=dt,
                                                device=self.device)
            if r is None:
                continue
            z = lambda *s: torch.zeros(max_requests, r.heads, *s, dtype=torch.float32, device=self.device)
            if r.kind == "mlstm":
                self.state[li] = (z(r.dim, r.vdim), z(r.dim), z())
            elif r.kind in ("retention", "time_mix"):
                self.state[li] = (z(r.dim, r.vdim),)
            else:
                self.state[li] = (z(r.state, r.vdim), torch.zeros(max_requests, r.conv - 1, r.conv_dim, dtype=dt, device=self.device))

        self.shift = shift_state(len(cfg.layers), max_requests, cfg.hidden_size, self.device) if cfg.block == "shifted" else None

    def groups(self) -> List[GroupTable]:
        return list(self.by_window.values())

    def group_of(self, layer: int) -> GroupTable:
        return self.by_window[attention_part(self.cfg.layers[layer].mixer).window]

    def prepare(self, row: int, start_pos: int, n_tokens: int, lookback: Optional[int] = None) -> None:
        end = start_pos + n_tokens
        for w, g in self.by_window.items():
            lo = max(0, start_pos - w + 1)
            g.release_before(row, lo // PAGE)
            g.ensure(row, lo // PAGE, (end - 1) // PAGE)

    # ---- admission: the full-context group promises whole contexts --------------------------------
    @staticmethod
    def full_pages(context: int) -> int:
        return context // PAGE + 1

    def reserve(self, row: int, context: int) -> None:
        if self.full is not None:
            self.reserved[row] = self.full_pages(context)

    def promised(self) -> int:
        """Full-context pages promised to running requests and not allocated yet."""
        return sum(max(0, need - self.full.held(row)) for row, need in self.reserved.items())

    def fits(self, context: int) -> bool:
        return self.full is None or self.full_pages(context) <= self.full.num_pages

    def can_admit(self, n_tokens: int, context: int) -> bool:
        n = min(n_tokens, context)
        if not self.free_rows or any(len(g.free) < n // PAGE + 2 for w, g in self.by_window.items() if w < FULL_CONTEXT):
            return False
        return self.full is None or len(self.full.free) - self.promised() >= self.full_pages(context)

    def usage(self) -> float:
        total = sum(g.num_pages for g in self.by_window.values())
        if total == 0:
            return (self.max_requests - len(self.free_rows)) / self.max_requests
        return sum(g.pages_in_use for g in self.by_window.values()) / total

    def bytes_allocated(self) -> int:
        n = sum(t.numel() * t.element_size() for t in self.kv_cache.values())
        if self.shift is not None:
            n += sum(t.numel() * t.element_size() for t in (self.shift.token, self.shift.now, self.shift.then))
        return n + sum(t.numel() * t.element_size() for st in self.state.values() for t in st)


def hybrid_bytes_per_context_token(cfg: HybridConfig) -> int:
    """Bytes of full-context cache that one token of context costs (windows and recurrent states are bounded)."""
    es = 4 if cfg.dtype == "float32" else 2
    n = 0
    for l in cfg.layers:
        m = attention_part(l.mixer)
        if m is not None and m.kind == "latent_attention" and m.kv_from is None:
            n += latent_row(m.kv_rank, m.rot_dim)[0] * es
        elif m is not None and m.kind == "grouped_attention":
            n += m.kv_heads * grouped_row(m.dim, m.vdim)[0] * es
        elif m is not None and m.kind == "talking_attention" and m.chunk is None:
            n += talking_row(m.kv_heads, m.dim, m.vdim)[0] * es
    return n


def kv_row_width(dim: int, rot_dims: int) -> int:
    """Elements of a cached row (key as projected, rotated head), a multiple of 8 so that rows stay 16-byte aligned."""
    return (dim + rot_dims + 7) // 8 * 8


def hybrid_pool_pages(window: int, max_requests: int, max_context: int, max_chunk: int) -> int:
    """Pages of one window group so that `max_requests` requests never run out: the window (or the whole context, if that
    is shorter) of each, and one step's new tokens."""
    span = min(window, max_context)
    return max_requests * ((span + PAGE - 1) // PAGE + 2) + (max_chunk + PAGE - 1) // PAGE + 2


def size_pools(cfg: ModelConfig, max_requests: int, max_context: int, max_chunk: int, dcp_size: int = 1,
               pool_tokens: Optional[int] = None) -> Dict[str, int]:
    """Pages needed so that `max_requests` sequences of `max_context` tokens fit (no prefix sharing); with decode
    context parallelism `c4_pages` is one rank's share (every dcp_size-th page of each request, rounded up).
    pool_tokens: cap the compressed pools at this many context tokens over all requests together (plus the partial
    pages every request may leave open); admission then makes requests wait for room."""
    swa = max_requests * ((cfg.sliding_window + PAGE - 1) // PAGE + 2) + (max_chunk + PAGE - 1) // PAGE + 2
    c4 = max_requests * -(-((max_context // 4 + PAGE - 1) // PAGE + 1) // dcp_size)
    c128 = max_requests * ((max_context // 128 + PAGE - 1) // PAGE + 1)
    if pool_tokens is not None:
        c4 = min(c4, -(-(pool_tokens // 4) // (PAGE * dcp_size)) + max_requests)
        c128 = min(c128, -(-(pool_tokens // 128) // PAGE) + 2 * max_requests + 1)
    return {"swa_pages": swa, "c4_pages": c4, "c128_pages": c128}


def kv_bytes_per_context_token(cfg: ModelConfig, layers: Optional[List[int]] = None, dcp_size: int = 1) -> float:
    """Bytes of compressed KV (latent + indexer-K rows of the ratio-4 layers, latent rows of the ratio-128 layers) that
    one token of context costs a rank: the quantity that turns a memory budget into `pool_tokens`."""
    fp8 = cfg.kv_cache_dtype == "fp8_ds_mla"
    D, Rd, di = cfg.head_dim, cfg.qk_rope_head_dim, cfg.index_head_dim
    latent = PagedCache.page_bytes(D, Rd, fp8, "latent") / PAGE
    index = PagedCache.page_bytes(di, Rd, fp8, "indexer", fp4=cfg.indexer_dtype == "mxfp4") / PAGE
    total = 0.0
    for li in (layers if layers is not None else range(cfg.num_hidden_layers)):
        kind = cfg.layer_kind(li)
        if kind == "c4a":
            total += (latent + index) / 4 / dcp_size
        elif kind == "c128a":
            total += latent / 128
    return total


def memory_pool_tokens(cfg: ModelConfig, utilization: float, free_bytes: int, total_bytes: int, min_tokens: int,
                       layers: Optional[List[int]] = None, dcp_size: int = 1) -> int:
    """Context tokens the compressed pools may hold when this process may use `utilization` of the device's memory:
    that share minus what is taken already (the weights; other tenants of a shared GPU count too), divided by the
    bytes one token costs, but never less than one request of `min_tokens` (launchers/start-hy4-tp4.sh:16-30 GPU_MEM)."""
    budget = utilization * total_bytes - (total_bytes - free_bytes)
    per_token = kv_bytes_per_context_token(cfg, layers, dcp_size)
    return max(min_tokens, int(budget / max(per_token, 1e-9)))
