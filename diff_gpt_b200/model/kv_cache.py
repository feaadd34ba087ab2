"""KV storage for the decode path.

`KVCache` keeps the reference's public surface (constructor, `insert_kv`,
`prefill`, `get_pos`, `reset`, attributes `kv_shape`, `kv_cache`, `pos`;
reference: src/diff_gpt/model/kv_cache.py:4-116) so code written against the
reference — including its Engine — keeps working; the CUDA kernels read and
write its dense (L, 2, B, H, T, D) tensor in place through `layer_layout`.

`PagedKVCache` is the layout the Monte-Carlo engine uses instead of replicating
the prompt (the reference's `prefill` broadcast, kv_cache.py:79): K/V live in
fixed-size pages, every trajectory of a series points at the SAME prompt pages,
and each trajectory owns a contiguous run of pages for the tokens it generates.

`RowCache` (requests fed step by step) and `PagedRowCache` (the engine) serve the models that are built from a
configuration: one row of numbers per token and layer run, bounded by the windows, and the per-sequence state
(`SeqState`) that such models carry beside it.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops


class KVCache:
    """Dense cache, one tensor (n_layer, 2, batch, n_head, seq_len, head_dim).

    `.pos` advances when the last layer has inserted (kv_cache.py:113-115).
    """

    __slots__ = ("kv_shape", "kv_cache", "pos")

    def __init__(self, batch_size: int, num_heads: int, seq_len: int, head_dim: int, num_layers: int) -> None:
        self.kv_shape = (num_layers, 2, batch_size, num_heads, seq_len, head_dim)
        self.kv_cache = torch.zeros(0)
        self.pos = 0

    # -- reference API ---------------------------------------------------------
    def reset(self) -> None:
        self.pos = 0

    def get_pos(self) -> int:
        return self.pos

    def prefill(self, other: "KVCache") -> None:
        """Take over `other`'s first `other.pos` tokens, broadcasting a batch of 1 to this batch."""
        assert self.kv_cache.size(0) == 0, "Cannot prefill a non-empty KV cache"
        assert other.kv_cache.size(0) != 0, "Cannot prefill with a None KV cache"
        mine, theirs = self.kv_shape, other.kv_shape
        names = ("Layer count", "K/V dimension", None, "Head count", None, "Head dim")
        for axis, label in enumerate(names):
            if label is not None:
                assert mine[axis] == theirs[axis], f"{label} mismatch: {mine[axis]} != {theirs[axis]}"
        assert mine[2] == theirs[2] or theirs[2] == 1, (
            f"Batch size mismatch: {mine[2]} vs {theirs[2]} (other must be 1 or equal)"
        )
        assert mine[4] >= theirs[4], f"Sequence length mismatch: {mine[4]} < {theirs[4]}"
        src = other.kv_cache
        self.kv_cache = torch.empty(self.kv_shape, dtype=src.dtype, device=src.device)
        n = other.pos
        self.kv_cache[:, :, :, :, :n].copy_(src[:, :, :, :, :n])
        self.pos = n

    def insert_kv(self, layer_idx: int, k: torch.Tensor, v: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
        """Write k, v (B, H, T_add, D) at the cursor; return views of everything cached so far."""
        t_add = k.size(2)
        t_end = self.pos + t_add
        self.ensure(t_end, k.dtype, k.device)
        store = self.kv_cache
        store[layer_idx, 0, :, :, self.pos : t_end].copy_(k)
        store[layer_idx, 1, :, :, self.pos : t_end].copy_(v)
        keys = store[layer_idx, 0, :, :, :t_end]
        values = store[layer_idx, 1, :, :, :t_end]
        if layer_idx == store.size(0) - 1:
            self.pos = t_end
        return keys, values

    # -- what the kernels need ---------------------------------------------------
    def ensure(self, t_end: int, dtype: torch.dtype, device: torch.device) -> None:
        """Allocate lazily; grow to (t_end + 1024) rounded up to 1024 when full (kv_cache.py:87-106)."""
        if self.kv_cache.size(0) == 0:
            self.kv_cache = torch.empty(self.kv_shape, dtype=dtype, device=device)
        have = self.kv_cache.size(4)
        if t_end > have:
            want = (t_end + 1024 + 1023) & ~1023
            grown = torch.empty(
                (*self.kv_cache.shape[:4], want, self.kv_cache.shape[5]), dtype=dtype, device=device
            )
            grown[:, :, :, :, :have].copy_(self.kv_cache)
            self.kv_cache = grown
            self.kv_shape = self.kv_cache.shape

    def layer_layout(self, layer: int) -> ops.KvLayout:
        _, _, _, H, T, D = self.kv_cache.shape
        c = self.kv_cache
        return ops.kv_layout(c[layer, 0], c[layer, 1], page_stride=H * T * D, head_stride=T * D, page_tokens=T)


class PagedKVCache:
    """Paged K/V with one shared prompt per series and private pages per trajectory.

    pool            (n_layer, n_pages, 2, n_head, page_tokens, head_dim)
    prefix_table    (n_series, prefix_pages)            int32  -> prompt pages of a series
    row_table       (n_rows, prefix_pages + own_pages)  int32  -> same prompt pages, then the row's own run
    Rows are series-major: row = series * rows_per_series + trajectory.
    A row's generated token g sits at logical slot prefix_pages * page_tokens + g.
    """

    def __init__(
        self,
        n_layer: int,
        n_head: int,
        head_dim: int,
        n_series: int,
        rows_per_series: int,
        prefix_len: int,
        max_new: int,
        dtype: torch.dtype,
        device: torch.device | str,
        page_tokens: int = 64,
        pool: torch.Tensor | None = None,
    ) -> None:
        pt = page_tokens
        self.page_tokens = pt
        self.n_layer, self.n_head, self.head_dim = n_layer, n_head, head_dim
        self.n_series, self.rows_per_series = n_series, rows_per_series
        self.n_rows = n_series * rows_per_series
        self.prefix_len = prefix_len
        self.prefix_pages = max(1, -(-prefix_len // pt))
        self.own_pages = max(1, -(-max_new // pt))
        self.max_new = max_new
        n_pages = n_series * self.prefix_pages + self.n_rows * self.own_pages
        shape = (n_layer, n_pages, 2, n_head, pt, head_dim)
        if pool is not None:  # storage handed in by the caller (e.g. kept across calls); contents need not be cleared
            assert tuple(pool.shape) == shape and pool.dtype == dtype and pool.is_contiguous(), "pool does not fit this cache"
            self.pool = pool
        else:
            self.pool = torch.empty(shape, dtype=dtype, device=device)
        pre = torch.arange(n_series * self.prefix_pages, dtype=torch.int32).view(n_series, self.prefix_pages)
        own = n_series * self.prefix_pages + torch.arange(self.n_rows * self.own_pages, dtype=torch.int32).view(
            self.n_rows, self.own_pages
        )
        row = torch.cat([pre.repeat_interleave(rows_per_series, dim=0), own], dim=1)
        self.prefix_table = pre.contiguous().to(device)
        self.row_table = row.contiguous().to(device)
        self.suffix_slot0 = self.prefix_pages * pt

    @property
    def bytes(self) -> int:
        return self.pool.numel() * self.pool.element_size()

    prompts_exchangeable = True  # the prompt pages of a block of series are one run of the pool

    def begin_prompts(self) -> None:
        """Called before a new set of prompts is prefilled."""

    def prompts_ready(self) -> None:
        """Called when every prompt is in place, and again to undo a decode forward that was only a warm-up."""

    def _layout(self, layer: int, table: torch.Tensor) -> ops.KvLayout:
        H, pt, D = self.n_head, self.page_tokens, self.head_dim
        p = self.pool[layer]
        return ops.kv_layout(
            p[0, 0], p[0, 1], page_stride=2 * H * pt * D, head_stride=pt * D, page_tokens=pt, page_table=table,
            n_pages=p.shape[0],
        )

    def prefix_layout(self, layer: int) -> ops.KvLayout:
        """Sequence index = series (prompt prefill and the shared-prefix attention phase)."""
        return self._layout(layer, self.prefix_table)

    def row_layout(self, layer: int) -> ops.KvLayout:
        """Sequence index = row (append and per-trajectory attention)."""
        return self._layout(layer, self.row_table)


@dataclass(frozen=True)
class StateSpec:
    """A tensor of per-sequence state: shape [lead, n_seq, *shape], `fill` before the first token."""

    lead: int
    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32
    fill: float = 0

    def make(self, n_seq: int, device) -> torch.Tensor:
        return torch.full((self.lead, n_seq, *self.shape), self.fill, dtype=self.dtype, device=device)


class SeqState:
    """What a model carries from token to token besides cached rows: convolution inputs, recurrent states, the last token.

    A forward over several tokens reads one buffer and writes the other (`source` / `target`, then `flip`), so that no
    thread overwrites what another still reads; one token at a time is updated in place.
    """

    def __init__(self, specs: dict[str, StateSpec], n_seq: int, device) -> None:
        self.specs = specs
        self.buffers = [{k: s.make(n_seq, device) for k, s in specs.items()} for _ in range(2)]
        self.current = 0

    @property
    def source(self) -> dict[str, torch.Tensor]:
        return self.buffers[self.current]

    @property
    def target(self) -> dict[str, torch.Tensor]:
        return self.buffers[1 - self.current]

    def flip(self) -> None:
        self.current = 1 - self.current

    def clear(self) -> None:
        for buf in self.buffers:
            for k, t in buf.items():
                t.fill_(self.specs[k].fill)
        self.current = 0


class RowCache:
    """Cache for requests fed step by step: one row of numbers per token and storage key (a latent, or the keys and values
    of all heads), and the model's per-sequence state.

    widths      {key: columns of a row}, one entry per layer (or layer run) that caches rows
    keep        tokens before a new one that some layer's window can still reach (the largest window less one), or None
                when a layer sees everything
    keep_first  first tokens that stay visible from every distance
    Rows live in one dense run of slots per sequence.  Only the first `keep_first` and the last `keep` tokens are ever
    needed: when the run is full the latter move to its front, behind the former, and `base` (how many tokens have been
    dropped) moves with them.  Rows carry their positions in themselves where they have any, so slots are all that the
    attention kernels need: a window counts slots back from the newest, and what was dropped lay behind every window.
    """

    def __init__(self, batch_size: int, widths: dict[int, int], keep: int | None, states: dict[str, StateSpec], dtype: torch.dtype,
                 device, keep_first: int = 0) -> None:
        self.batch_size, self.widths, self.keep, self.keep_first = batch_size, widths, keep, keep_first
        self.dtype, self.device = dtype, device
        self.store: dict[int, torch.Tensor] = {}
        self.capacity = 0
        self.state = SeqState(states, batch_size, device)
        self.pos = 0
        self.base = 0

    def reset(self) -> None:
        self.pos = self.base = 0
        self.state.clear()

    def get_pos(self) -> int:
        return self.pos

    @property
    def slot(self) -> int:
        """The slot the next token goes to."""
        return self.pos - self.base

    def ensure(self, T: int) -> None:
        """Make room for T more tokens behind the ones that can still be seen."""
        if self.slot + T <= self.capacity:
            return
        fixed = min(self.slot, self.keep_first)
        live = self.slot - fixed if self.keep is None else min(self.slot - fixed, self.keep)
        first = self.slot - live
        if fixed + live + T <= self.capacity:
            for t in self.store.values():
                t[:, fixed : fixed + live] = t[:, first : first + live].clone()
        else:
            # room to slide in: as many slots again as stay live (at least 1024), so a move is paid for by many tokens
            want = (fixed + live + T + max(live, 1024) + 63) // 64 * 64
            for key, r in self.widths.items():
                grown = torch.empty((self.batch_size, want, r), dtype=self.dtype, device=self.device)
                if fixed + live:
                    grown[:, :fixed] = self.store[key][:, :fixed]
                    grown[:, fixed : fixed + live] = self.store[key][:, first : first + live]
                self.store[key] = grown
            self.capacity = want
        self.base += first - fixed

    def layout(self, key: int) -> ops.KvLayout:
        c = self.store[key]
        return ops.kv_layout(c, c, page_stride=c.stride(0), head_stride=0, page_tokens=self.capacity)

    def kv_layout(self, key: int, D: int, v_col: int) -> ops.KvLayout:
        """The same rows as separate keys and values of heads D wide, the values from column `v_col` on."""
        c = self.store[key]
        return ops.kv_layout(c, c[:, :, v_col:], page_stride=c.stride(0), head_stride=D, page_tokens=self.capacity)

    def span(self, key: int, first: int, end: int) -> torch.Tensor:
        """Rows of slots [first, end) of all sequences as [batch * (end - first), r] (a copy if there are several)."""
        c = self.store[key][:, first:end]
        return c.reshape(-1, c.shape[-1])


class PagedRowCache:
    """`PagedKVCache` for cached rows: per storage key one pool of pages (n_pages, page_tokens, r).

    The prompt's pages are shared by a series' rows.  A row's own pages are a ring when every layer has a window: the
    table of a row maps each page of generated tokens to physical page (index mod ring length), and the ring is long
    enough that the page being written is out of every window.  Pages that may hold first tokens which stay visible (a
    prompt can be shorter than `keep_first`) lie in front of the ring and are never written again.  The per-sequence state
    is kept per series at the prompt's end (`prompts`) and per row (`states`).
    """

    prompts_exchangeable = False

    def __init__(self, widths: dict[int, int], keep: int | None, states: dict[str, StateSpec], n_series: int, rows_per_series: int,
                 prefix_len: int, max_new: int, dtype: torch.dtype, device, page_tokens: int = 64, keep_first: int = 0) -> None:
        pt = self.page_tokens = page_tokens
        self.n_series, self.rows_per_series = n_series, rows_per_series
        self.n_rows = n_series * rows_per_series
        self.prefix_len, self.max_new = prefix_len, max_new
        self.prefix_pages = max(1, -(-prefix_len // pt))
        self.own_pages = max(1, -(-max_new // pt))
        fixed = -(-max(0, keep_first - 1) // pt)  # a prompt has at least one token
        self.ring_pages = self.own_pages if keep is None else min(self.own_pages, fixed + -(-keep // pt) + 1)
        n_pages = n_series * self.prefix_pages + self.n_rows * self.ring_pages
        self.pools = {key: torch.zeros((n_pages, pt, r), dtype=dtype, device=device) for key, r in widths.items()}
        pre = torch.arange(n_series * self.prefix_pages, dtype=torch.int32).view(n_series, self.prefix_pages)
        ring = torch.arange(self.n_rows * self.ring_pages, dtype=torch.int32).view(self.n_rows, self.ring_pages)
        page = torch.arange(self.own_pages)
        if self.ring_pages < self.own_pages:
            page = torch.where(page < fixed, page, fixed + (page - fixed) % (self.ring_pages - fixed))
        own = n_series * self.prefix_pages + ring[:, page]
        row = torch.cat([pre.repeat_interleave(rows_per_series, dim=0), own], dim=1)
        self.prefix_table = pre.contiguous().to(device)
        self.row_table = row.contiguous().to(device)
        self.suffix_slot0 = self.prefix_pages * pt
        self.specs = states
        self.states = {k: s.make(self.n_rows, device) for k, s in states.items()}
        self.prompts: list[tuple[torch.Tensor, dict[str, torch.Tensor]]] = []  # (series indices, states at the prompt's end)

    @property
    def bytes(self) -> int:
        return sum(p.numel() * p.element_size() for p in self.pools.values())

    def prompt_states(self, members: list[int]) -> dict[str, torch.Tensor]:
        """Where the prompts of these series leave their state, [lead, len(members), ...] each."""
        dev = self.prefix_table.device
        states = {k: s.make(len(members), dev) for k, s in self.specs.items()}
        self.prompts.append((torch.tensor(members, device=dev), states))
        return states

    def begin_prompts(self) -> None:
        for _, states in self.prompts:
            for k, t in states.items():
                t.fill_(self.specs[k].fill)

    def prompts_ready(self) -> None:
        """Every row starts from the state its series' prompt has left."""
        for members, states in self.prompts:
            for k, t in states.items():
                rows = self.states[k].view(t.shape[0], self.n_series, self.rows_per_series, *t.shape[2:])
                rows[:, members] = t.unsqueeze(2).expand(-1, -1, self.rows_per_series, *t.shape[2:])

    def layout(self, key: int, table: torch.Tensor) -> ops.KvLayout:
        p = self.pools[key]
        return ops.kv_layout(p, p, page_stride=p.stride(0), head_stride=0, page_tokens=self.page_tokens, page_table=table,
                             n_pages=p.shape[0])

    def kv_layout(self, key: int, table: torch.Tensor, D: int, v_col: int) -> ops.KvLayout:
        """The same rows as separate keys and values of heads D wide, the values from column `v_col` on."""
        p = self.pools[key]
        return ops.kv_layout(p, p[:, :, v_col:], page_stride=p.stride(0), head_stride=D, page_tokens=self.page_tokens, page_table=table,
                             n_pages=p.shape[0])


# ---- the same for latents beside the inputs of causal convolutions ----------------------------------
def conv_state(n_layer: int, taps: int, width: int) -> dict[str, StateSpec]:
    """The last taps - 1 inputs of every layer's causal convolution, fp32 [n_layer, n_seq, taps - 1, width]."""
    return {"conv": StateSpec(n_layer, (taps - 1, width))}


class LatentCache(RowCache):
    """ranks: {layer: columns of a cached latent} for the layers that own one; other layers read an owner's."""

    def __init__(self, batch_size: int, ranks: dict[int, int], keep: int | None, n_layer: int, taps: int, width: int,
                 dtype: torch.dtype, device) -> None:
        super().__init__(batch_size, ranks, keep, conv_state(n_layer, taps, width), dtype, device)

    @property
    def ranks(self) -> dict[int, int]:
        return self.widths

    @property
    def latents(self) -> dict[int, torch.Tensor]:
        return self.store


class PagedLatentCache(PagedRowCache):
    def __init__(self, ranks: dict[int, int], keep: int | None, n_layer: int, taps: int, width: int, n_series: int,
                 rows_per_series: int, prefix_len: int, max_new: int, dtype: torch.dtype, device, page_tokens: int = 64) -> None:
        super().__init__(ranks, keep, conv_state(n_layer, taps, width), n_series, rows_per_series, prefix_len, max_new, dtype, device,
                         page_tokens)

    @property
    def rows(self) -> torch.Tensor:
        return self.states["conv"]

    def prompt_states(self, members: list[int]) -> torch.Tensor:
        return super().prompt_states(members)["conv"]
