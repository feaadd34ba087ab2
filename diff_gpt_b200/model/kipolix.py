"""Kipolix: a decoder whose layers mix tokens by retention (linear attention with a fixed decay per head) or by
grouped-query attention over a sliding window with kept first tokens, around several fp32 residual streams; a stretch of
layers may run several times with the same weights.

With e the embedding of a token plus that of its bigram, S streams x_s = e and, for every sublayer (mixer, feed-forward),

    u    = sum_s in[s] x_s                        h = rms_norm(u) * (1 + norm)
    x_t <- sum_s mix[s, t] x_s + out[t] f(h)      all streams at once

    retention     q, k rotated (halves paired), k / sqrt(dim):   S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
                  f = W_o [ rms_norm(o) per head * silu(W_g h) ]
    attention     q, k normalised over the whole projection, rotated (neighbours paired);  i sees j <= i with
                  i - j < mask.size or j < mask.keep_first;  f = W_o [ softmax(q . k * scale) v ]
    feed-forward  f = W_down (silu(W_gate h) * W_up h)

and the head reads rms_norm(sum_s x_s) * (1 + norm).

`KipolixPlan.run` enqueues

    embedding + bigram + norm -> [q | k | v (| gate) GEMM -> (norm + rotation + append -> attention) or retention ->
    out-proj GEMM -> streams + norm -> gate | up GEMM with SiLU gate -> down GEMM -> streams + norm] x layer runs ->
    streams + final norm -> head GEMM

on cuBLAS for plain products and this library's kernels for the rest.  Streams, norms, angles, scores, probabilities,
recurrent states and what enters them are fp32.  Attention has two forms: few query tokens per sequence read the cached
rows once per group of heads (`ops.grouped_attn`), many use the prefill kernels (`ops.fmha_grouped`).  Every run of a
layer has its own cache rows or state.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable

import torch
import torch.nn.functional as F

from .. import ops
from .._lib import region
from .configured import FUSED_FF_MIN_ROWS, ConfiguredModel, fp32_reductions, pick_latent_splits, round_up
from .kv_cache import PagedRowCache, RowCache, StateSpec
from .rope import rotation_table

PREFILL_MIN_TOKENS = 32  # query tokens per sequence from which the prefill attention kernels are used
PREFILL_HEAD_DIMS = (32, 64, 128)  # their head sizes; smaller heads are padded with zeros


# ---- configuration --------------------------------------------------------------------
@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float


@dataclass(frozen=True)
class Retention:
    heads: int
    dim: int
    vdim: int
    rot: Rotation
    decay: tuple[float, ...]


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot: Rotation
    scale: float
    window: int
    keep_first: int

    @property
    def head(self) -> int:
        """Head size the kernels work with: query, key and value heads are padded with zeros to one common size."""
        need = max(self.dim, self.vdim)
        return next((d for d in PREFILL_HEAD_DIMS if d >= need), round_up(need, 8))


@dataclass(frozen=True)
class Layer:
    mixer: Retention | Attention
    ff: int | None  # None: no feed-forward


def _mixer(kind: str, entry: dict) -> Retention | Attention:
    m = dict(entry)
    rot = dict(m.pop("rot"))
    rotation = Rotation(dims=int(rot.pop("dims")), base=float(rot.pop("base")))
    sizes = dict(heads=int(m.pop("heads")), dim=int(m.pop("dim")), vdim=int(m.pop("vdim")), rot=rotation)
    mask: dict = {}
    if kind == "retention":
        out = Retention(**sizes, decay=tuple(float(d) for d in m.pop("decay")))
        if len(out.decay) != out.heads or not all(0.0 <= d <= 1.0 for d in out.decay):
            raise ValueError("one decay in [0, 1] per head is needed")
    elif kind == "attention":
        mask = dict(m.pop("mask"))
        out = Attention(**sizes, kv_heads=int(m.pop("kv_heads")), scale=float(m.pop("scale")), window=int(mask.pop("size")),
                        keep_first=int(mask.pop("keep_first")))
        if out.kv_heads < 1 or out.heads % out.kv_heads:
            raise ValueError("the query heads must be a multiple of the key/value heads")
        if out.window < 1 or out.keep_first < 0:
            raise ValueError("a window holds at least the token itself")
    else:
        raise ValueError(f"unknown mixer type {kind!r}")
    if m or mask or rot:  # a key that is not understood would change what the layer computes
        raise ValueError(f"unknown keys {sorted(m) + sorted(mask) + sorted(rot)} in a mixer")
    if rotation.dims % 2 or not 2 <= rotation.dims <= out.dim:
        raise ValueError("the rotated dimensions come in pairs and lie inside a head")
    return out


@dataclass(frozen=True)
class KipolixConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    buckets: int
    mul_prev: int
    mul_cur: int
    loop: tuple[int, int, int]  # layers [start, stop) run `times` times in a row
    layers: tuple[Layer, ...] = field(default_factory=tuple)

    @staticmethod
    def from_dict(c: dict) -> "KipolixConfig":
        layers = []
        for i, entry in enumerate(c["layers"]):
            try:
                mixer = _mixer(entry["type"], entry["mixer"])
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
            mlp = entry.get("mlp")
            if mlp is not None and (mlp["kind"] != "dense" or set(mlp) != {"kind", "ff"}):
                raise ValueError(f"layer {i}: unknown feed-forward {mlp}")
            layers.append(Layer(mixer=mixer, ff=None if mlp is None else int(mlp["ff"])))
        if not layers:
            raise ValueError("a model has at least one layer")
        loop = c.get("loop") or {"start": 0, "stop": 0, "times": 1}
        start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
        if not 0 <= start <= stop <= len(layers) or times < 1:
            raise ValueError(f"loop {loop} does not name a stretch of the layers")
        big = c["embedding"]["bigram"]
        out = KipolixConfig(
            vocab=int(c["vocab"]), width=int(c["width"]), eps=float(c["norm"]["eps"]), streams=int(c["streams"]),
            buckets=int(big["buckets"]), mul_prev=int(big["mul_prev"]), mul_cur=int(big["mul_cur"]), loop=(start, stop, times),
            layers=tuple(layers),
        )
        if set(c["embedding"]) != {"bigram"} or set(big) != {"buckets", "mul_prev", "mul_cur"}:
            raise ValueError(f"unknown keys in the embedding: {c['embedding']}")
        if out.streams < 1 or out.buckets < 1:
            raise ValueError("at least one stream and one bucket are needed")
        return out

    @property
    def runs(self) -> tuple[int, ...]:
        """The layers in the order in which they run; a looped stretch is there as often as it runs."""
        a, b, times = self.loop
        n = len(self.layers)
        return (*range(a), *(tuple(range(a, b)) * times), *range(b, n))

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Checkpoint names and shapes."""
        C, S = self.width, self.streams
        out: dict[str, tuple[int, ...]] = {
            "embed": (self.vocab, C), "bigram": (self.buckets + 1, C), "final.norm": (C,), "head": (self.vocab, C),
        }
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer.mixer
            out[p + "norm1"] = (C,)
            out[p + "mix.q"] = (m.heads * m.dim, C)
            G = m.heads if isinstance(m, Retention) else m.kv_heads
            out[p + "mix.k"] = (G * m.dim, C)
            out[p + "mix.v"] = (G * m.vdim, C)
            if isinstance(m, Retention):
                out[p + "mix.g"] = (m.heads * m.vdim, C)
            else:
                out[p + "mix.q.norm"] = (m.heads * m.dim,)
                out[p + "mix.k.norm"] = (G * m.dim,)
            out[p + "mix.o"] = (C, m.heads * m.vdim)
            if layer.ff is not None:
                out[p + "norm2"] = (C,)
                out[p + "mlp.gate"] = (layer.ff, C)
                out[p + "mlp.up"] = (layer.ff, C)
                out[p + "mlp.down"] = (C, layer.ff)
            for q in (1,) if layer.ff is None else (1, 2):
                out[f"{p}hc{q}.in"] = out[f"{p}hc{q}.out"] = (S,)
                out[f"{p}hc{q}.mix"] = (S, S)
        return out


# ---- weights as the kernels want them ----------------------------------------------------
@dataclass
class _Sublayer:
    """One sublayer's entry from and exit to the streams, fp32."""

    inp: torch.Tensor  # [S]
    mix: torch.Tensor  # [S, S], from x to
    out: torch.Tensor  # [S]
    norm: torch.Tensor  # [C], 1 + w


@dataclass
class _PackedLayer:
    m: Retention | Attention
    w_in_t: torch.Tensor  # [C, projection columns]
    cols: tuple[int, ...]  # where q, k, v (and the gate) start
    q_norm: torch.Tensor | None
    k_norm: torch.Tensor | None
    decay: torch.Tensor | None
    w_o_t: torch.Tensor
    sub1: _Sublayer
    sub2: _Sublayer | None
    w_gu: torch.Tensor | None  # [2 ff, C], gate and up rows interleaved
    w_down_t: torch.Tensor | None


@dataclass
class _Packed:
    emb: torch.Tensor
    bigram: torch.Tensor
    head: torch.Tensor
    final_norm: torch.Tensor
    layers: list
    stamp: tuple


# ---- how one forward call is bound to cached rows and states ---------------------------------
@dataclass
class RowBinding:
    """Where the new rows and states go, and which cached keys each query sees.

    Queries see the logical keys 0 .. len0 + len1 + step + t - 1 (see `dgpt_grouped_attn`) that their window or the kept
    first keys allow; `keys` is a host-side bound on their number.
    context     cached keys in front of the call's own when they and the new ones are logical keys 0, 1, ... of one run
                (prompts and portions), for the prefill kernels; None otherwise
    kv_layout   (layer run, head size, value column) -> the rows as separate keys and values
    tables      {(base, dims): rotation table}
    """

    layout: Callable[[int], object]
    slot0: torch.Tensor
    pos0: torch.Tensor
    start1: torch.Tensor
    len1: torch.Tensor
    keys: int
    tables: dict
    state_out: dict[str, torch.Tensor]
    state_in: dict[str, torch.Tensor] | None = None
    len0: torch.Tensor | None = None
    step: torch.Tensor | None = None
    context: int | None = None
    kv_layout: Callable[[int, int, int], object] | None = None
    fmha_impl: int = 0


class KipolixPlan:
    """Buffers for one (n_seq, T) forward and the launch sequence that fills them (see `ForwardPlan`)."""

    def __init__(self, model: "Kipolix", n_seq: int, T: int, last_only: bool = False, want_logits: bool = True,
                 rows: int | None = None) -> None:
        """`rows`: the number of rows whose logits are asked for by index at each run (overrides last_only)."""
        cfg, emb = model.config, model.embedding
        self.model, self.n_seq, self.T, self.n = model, n_seq, T, n_seq * T
        self.dev, self.dt = emb.device, emb.dtype
        n, C, V = self.n, cfg.width, cfg.vocab
        self._bufs: dict = {}
        self.e = torch.empty((n, C), dtype=torch.float32, device=self.dev)
        self.x = torch.empty((cfg.streams, n, C), dtype=torch.float32, device=self.dev)
        self.h, self.y = (torch.empty((n, C), dtype=self.dt, device=self.dev) for _ in range(2))
        n_out = rows if rows is not None else (n_seq if last_only else n)
        self.rows = None
        if rows is None and last_only and T > 1:
            self.rows = torch.arange(T - 1, n, T, dtype=torch.int32, device=self.dev)
        self.xn = torch.empty((n_out, C), dtype=self.dt, device=self.dev)
        self.logits = torch.empty((n_out, V), dtype=self.dt, device=self.dev) if want_logits else None
        self.own_head = self.dt == torch.bfloat16 and C % 8 == 0 and V % 16 == 0
        self.fused_ff = self.dt == torch.bfloat16 and C % 8 == 0 and n >= FUSED_FF_MIN_ROWS
        self.status = torch.zeros(1, dtype=torch.int32, device=self.dev)

    def _buf(self, name: str, *shape: int, dtype=None) -> torch.Tensor:
        key = (name, shape)
        t = self._bufs.get(key)
        if t is None:
            t = self._bufs[key] = torch.empty(shape, dtype=dtype or self.dt, device=self.dev)
        return t

    def _retention(self, run: int, lw: _PackedLayer, proj: torch.Tensor, b: RowBinding) -> torch.Tensor:
        m, n_seq, T = lw.m, self.n_seq, self.T
        y = self._buf("o", self.n, m.heads * m.vdim)
        ws = self._buf("ret_ws", max(4, ops.retention_workspace_bytes(n_seq, T, m.heads, m.dim, m.vdim) // 4), dtype=torch.float32)
        name = f"ret{run}"
        ops.retention(
            proj, lw.cols, b.tables[m.rot.base, m.rot.dims], b.pos0, b.step, lw.decay, min(m.decay), m.dim**-0.5,
            None if b.state_in is None else b.state_in[name], b.state_out[name], self.model.config.eps, y, ws, n_seq=n_seq, T=T,
            dim=m.dim, vdim=m.vdim, status=self.status,
        )
        return y

    def _attention(self, run: int, lw: _PackedLayer, proj: torch.Tensor, b: RowBinding) -> torch.Tensor:
        m, n_seq, T, n = lw.m, self.n_seq, self.T, self.n
        H, G, D = m.heads, m.kv_heads, m.head
        width, v_col = 2 * G * D, G * D
        q, o = self._buf("q", n, H * D), self._buf("o", n, H * D)
        ops.proj_norm_rope_append(
            proj, lw.q_norm, lw.k_norm, H * m.dim, G * m.dim, self.model.config.eps, b.tables[m.rot.base, m.rot.dims], q, b.layout(run),
            width, b.pos0, b.slot0, b.step, n_seq=n_seq, T=T, H=H, G=G, D=D, Dv=D, status=self.status,
        )
        if b.context is not None and T >= PREFILL_MIN_TOKENS and D in PREFILL_HEAD_DIMS:
            ops.fmha_grouped(
                q, b.kv_layout(run, D, v_col), o, token_stride=width, n_keys=b.context + T, B=n_seq, H=H, G=G, D=D, q_offset=b.context,
                window=m.window, keep_first=m.keep_first, scale=m.scale, impl=b.fmha_impl, status=self.status,
            )
            return o
        splits = pick_latent_splits(n, G, min(b.keys, m.window + m.keep_first))
        ws = None
        if splits > 1:
            ws = self._buf("ws", ops.latent_attn_workspace_bytes(n, H, D, splits) // 4, dtype=torch.float32)
        ops.grouped_attn(
            q, b.layout(run), b.len0, b.start1, b.len1, b.step, o, row_width=width, v_col=v_col, n_seq=n_seq, T=T, H=H, G=G, dk=D, dv=D,
            window=m.window, keep_first=m.keep_first, scale=m.scale, workspace=ws, n_splits=splits, status=self.status,
        )
        return o

    def _feed_forward(self, lw: _PackedLayer) -> None:
        """self.y = W_down (silu(W_gate h) * W_up h)"""
        two_ff = lw.w_gu.shape[0]
        act = self._buf("act", self.n, two_ff // 2)
        if self.fused_ff and two_ff % 16 == 0:
            ops.linear(self.h, lw.w_gu, act, silu_gate=True, status=self.status)
        else:
            gu = self._buf("gu", self.n, two_ff)
            with region("gemm_up"):
                torch.mm(self.h, lw.w_gu.t(), out=gu)
            ops.silu_mul(gu, act)
        with region("gemm_down"):
            torch.mm(act, lw.w_down_t, out=self.y)

    def run(self, ids32: torch.Tensor, b: RowBinding, rows: torch.Tensor | None = None,
            tap: Callable[[int, torch.Tensor], None] | None = None) -> torch.Tensor | None:
        """`rows`: int32 places (among the n tokens) whose logits are wanted; `tap(k, x)` sees the sum of the streams after
        the k-th layer run."""
        with fp32_reductions():
            return self._run(ids32, b, rows, tap)

    def _run(self, ids32, b, rows, tap):
        m = self.model
        cfg, W = m.config, m.packed_weights()
        eps, runs = cfg.eps, cfg.runs
        first = W.layers[runs[0]].sub1
        ops.embed_streams(
            ids32, None if b.state_in is None else b.state_in["prev"], b.state_out["prev"], W.emb, W.bigram, cfg.mul_prev, cfg.mul_cur,
            first.inp, first.norm, eps, self.e, self.h, n_seq=self.n_seq, T=self.T,
        )
        x = self.e  # all streams are still equal
        for k, i in enumerate(runs):
            lw = W.layers[i]
            proj = self._buf("proj", self.n, lw.w_in_t.shape[1])
            with region("gemm_in"):
                torch.mm(self.h, lw.w_in_t, out=proj)
            o = (self._retention if isinstance(lw.m, Retention) else self._attention)(k, lw, proj, b)
            with region("gemm_proj"):
                torch.mm(o, lw.w_o_t, out=self.y)
            sub = lw.sub1
            if lw.sub2 is not None:
                nxt = lw.sub2
                ops.streams_step(x, self.y, sub.mix, sub.out, self.x, nxt.inp, nxt.norm, eps, self.h)
                x, sub = self.x, nxt
                self._feed_forward(lw)
            if k + 1 < len(runs):
                nxt = W.layers[runs[k + 1]].sub1
                ops.streams_step(x, self.y, sub.mix, sub.out, self.x, nxt.inp, nxt.norm, eps, self.h)
                x = self.x
                if tap is not None:
                    tap(k, x.sum(0))
            elif tap is not None:
                after = torch.empty_like(self.x)
                ops.streams_step(x, self.y, sub.mix, sub.out, after)
                tap(k, after.sum(0))
        if self.xn.shape[0] == 0:
            return self.logits
        ops.streams_final(x, self.y, sub.mix, sub.out, W.final_norm, eps, self.xn, rows=self.rows if rows is None else rows)
        if self.logits is None:
            return None
        if self.own_head:
            ops.linear(self.xn, W.head, self.logits, status=self.status)
        else:
            with region("gemm_logits"):
                torch.mm(self.xn, W.head.t(), out=self.logits)
        return self.logits


class Kipolix(ConfiguredModel):
    def __init__(self, config: KipolixConfig | dict, block_size: int = 32768) -> None:
        """`block_size` only bounds how far the Engine generates (positions have no end of their own)."""
        cfg = config if isinstance(config, KipolixConfig) else KipolixConfig.from_dict(config)
        super().__init__(cfg, cfg.tensor_shapes(), block_size, cfg.vocab, cfg.width, cfg.layers[0].mixer.heads, len(cfg.layers))
        mixers = [cfg.layers[i].mixer for i in cfg.runs]
        attn = {k: m for k, m in enumerate(mixers) if isinstance(m, Attention)}
        self.row_widths = {k: 2 * m.kv_heads * m.head for k, m in attn.items()}
        self.keep = max((m.window for m in attn.values()), default=1) - 1
        self.keep_first = max((m.keep_first for m in attn.values()), default=0)
        self.state_specs = {"prev": StateSpec(1, (), torch.int32, -1)}
        for k, m in enumerate(mixers):
            if isinstance(m, Retention):
                self.state_specs[f"ret{k}"] = StateSpec(1, (m.heads, m.dim, m.vdim))
        self._tables: dict = {}

    # ---- weights -------------------------------------------------------------------------
    def pack(self, stamp) -> _Packed:
        cfg = self.config
        return _Packed(
            emb=self.embedding.detach(), bigram=self.tensor("bigram").detach(), head=self.tensor("head").detach(),
            final_norm=(1 + self.tensor("final.norm").detach().float()).contiguous(),
            layers=[self._pack_layer(i) for i in range(len(cfg.layers))], stamp=stamp,
        )

    def _pack_layer(self, i: int) -> _PackedLayer:
        C, layer = self.config.width, self.config.layers[i]
        m, ff = layer.mixer, layer.ff

        def w(name):
            return self.tensor(f"l{i}.{name}").detach()

        def heads(t, size, to):  # [heads * size, ...] -> [heads * to, ...], zero rows at the end of each head
            t = t.view(-1, size, *t.shape[1:])
            return F.pad(t, (0, 0) * (t.dim() - 2) + (0, to - size)).reshape(-1, *t.shape[2:])

        def sub(q):
            f = [w(f"hc{q}.{name}").float().contiguous() for name in ("in", "mix", "out")]
            return _Sublayer(*f, norm=(1 + w(f"norm{q}").float()).contiguous())

        q_norm = k_norm = decay = None
        if isinstance(m, Retention):
            parts = [w("mix.q"), w("mix.k"), w("mix.v"), w("mix.g")]
            parts = [F.pad(t, (0, 0, 0, round_up(t.shape[0], 8) - t.shape[0])) for t in parts]  # sections start aligned
            w_o = w("mix.o")
            decay = torch.tensor(m.decay, dtype=torch.float32, device=w_o.device)
        else:
            D = m.head
            parts = [heads(w("mix.q"), m.dim, D), heads(w("mix.k"), m.dim, D), heads(w("mix.v"), m.vdim, D)]
            q_norm, k_norm = (heads(w(f"mix.{n}.norm").float()[:, None], m.dim, D)[:, 0].contiguous() for n in ("q", "k"))
            w_o = F.pad(w("mix.o").view(C, m.heads, m.vdim), (0, D - m.vdim)).reshape(C, m.heads * D).contiguous()
        starts = [0]
        for t in parts:
            starts.append(starts[-1] + t.shape[0])
        return _PackedLayer(
            m=m, w_in_t=torch.cat(parts).contiguous().t(), cols=tuple(starts[:-1]), q_norm=q_norm, k_norm=k_norm, decay=decay,
            w_o_t=w_o.t(), sub1=sub(1), sub2=None if ff is None else sub(2),
            w_gu=None if ff is None else torch.stack([w("mlp.gate"), w("mlp.up")], dim=1).reshape(2 * ff, C).contiguous(),
            w_down_t=None if ff is None else w("mlp.down").t(),
        )

    def tables(self, positions: int) -> dict:
        """Rotation tables that cover this many positions (grown by doubling; a binding keeps the ones it was given)."""
        dev = self.embedding.device
        for layer in self.config.layers:
            key = (layer.mixer.rot.base, layer.mixer.rot.dims)
            have = self._tables.get(key)
            if have is None or have.shape[0] < positions or have.device != dev:
                n = max(1024, 1 << (positions - 1).bit_length())
                self._tables[key] = rotation_table(key[0], key[1], n, dev)
        return dict(self._tables)

    # ---- what the Engine needs -------------------------------------------------------------
    def new_cache(self, batch_size: int = 1, seq_len: int = 0) -> RowCache:
        emb = self.embedding
        cache = RowCache(batch_size, self.row_widths, self.keep, self.state_specs, emb.dtype, emb.device, self.keep_first)
        if seq_len > 0:
            cache.ensure(seq_len)
        return cache

    def paged_cache(self, n_series, rows_per_series, prefix_len, max_new, page_tokens, pool=None) -> PagedRowCache:
        assert pool is None, "this model's cache allocates its own pools"
        emb = self.embedding
        return PagedRowCache(self.row_widths, self.keep, self.state_specs, n_series, rows_per_series, prefix_len, max_new, emb.dtype,
                             emb.device, page_tokens=page_tokens, keep_first=self.keep_first)

    def prefill_plan(self, cache, members, P, fmha_impl):
        dev = cache.prefix_table.device
        n = len(members)
        table = cache.prefix_table[torch.tensor(members, device=dev)].contiguous()
        zero = torch.zeros(n, dtype=torch.int32, device=dev)
        layouts = {k: cache.layout(k, table) for k in self.row_widths}
        states = cache.prompt_states(members)
        bind = RowBinding(
            layout=layouts.__getitem__, slot0=zero, pos0=zero, start1=zero, len1=torch.ones(n, dtype=torch.int32, device=dev), keys=P,
            tables=self.tables(P), state_in=states if P == 1 else None, state_out=states, context=0,
            kv_layout=lambda k, D, v_col: cache.kv_layout(k, table, D, v_col), fmha_impl=fmha_impl if fmha_impl <= 3 else 0,
        )
        return bind, KipolixPlan(self, n, P, last_only=True)

    def decode_plan(self, cache, prompt_lens, max_keys, step, shared, fmha_impl, overlap_prefix, want_logits):
        R, dev = cache.n_rows, prompt_lens.device
        slot0 = torch.full((R,), cache.suffix_slot0, dtype=torch.int32, device=dev)
        row_len = prompt_lens.repeat_interleave(cache.rows_per_series).contiguous()
        layouts = {k: cache.layout(k, cache.row_table) for k in self.row_widths}
        bind = RowBinding(
            layout=layouts.__getitem__, slot0=slot0, pos0=row_len, start1=slot0, len0=row_len,
            len1=torch.ones(R, dtype=torch.int32, device=dev), step=step, keys=max_keys, tables=self.tables(max_keys),
            state_in=cache.states, state_out=cache.states,
        )
        return bind, KipolixPlan(self, R, 1, want_logits=want_logits)

    def new_plan(self, n_seq, T, **kw) -> KipolixPlan:
        return KipolixPlan(self, n_seq, T, **kw)

    def step_binding(self, cache: RowCache, B: int, T: int) -> RowBinding:
        dev = self.embedding.device
        slot, state = cache.slot, cache.state
        start = torch.full((B,), slot, dtype=torch.int32, device=dev)
        return RowBinding(
            layout=cache.layout, slot0=start, pos0=torch.full((B,), cache.pos, dtype=torch.int32, device=dev),
            start1=torch.zeros_like(start), len1=start + 1, keys=slot + T, tables=self.tables(cache.pos + T), state_in=state.source,
            state_out=state.source if T == 1 else state.target, context=slot, kv_layout=cache.kv_layout,
        )
