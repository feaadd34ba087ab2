"""Delunex: a decoder with sliding-window latent attention, an fp32 residual stream averaged over depth, and a causal
convolution in front of every mixer.

Per layer i, with X_0 the scaled embedding and x what the layer before hands on:

    h   = x + conv_i(x)                                  causal, per channel
    c   = rms_norm(W_dkv h) * w                          the cached latent (or another layer's: `kv_from`)
    y   = W_o [ sigmoid(W_g h)_n * attn(W_q,n h; W_uk,n c, W_uv,n c) ]_n    last `mask.size` tokens, no positions
    x'  = x + rms_norm(y) * norm1
    X_i+1 = x' + rms_norm(W_down xielu(W_up x')) * norm2  (x' itself in a layer without feed-forward)
    x   = sum_j dwa_i[j] X_j                             handed on to layer i + 1, or to the head

`DelunexPlan.run` enqueues

    embed -> [conv -> q | latent | gate GEMM -> latent norm + append -> attention -> out-proj GEMM -> norm + add ->
    up GEMM + xIELU -> down GEMM -> norm + add -> depth average] x L -> norm -> tied-table GEMM

on cuBLAS for plain products and this library's kernels for the rest.  X_j, x and x' stay fp32.  Attention has two
forms: few query tokens (decoding, short portions) work on the cached latents directly, with the key and value
expansions absorbed into the query and the output (`ops.latent_attn`: the cache is read once for all heads); many
query tokens expand keys and values with one GEMM and use the tensor-core attention kernels with a window
(`ops.fmha_window`).
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Callable

import torch
import torch.nn.functional as F

from .. import ops
from .._lib import region
from .configured import FUSED_FF_MIN_ROWS, ConfiguredModel, fp32_reductions, pick_latent_splits, round_up
from .kv_cache import LatentCache, PagedLatentCache

EXPAND_MIN_TOKENS = 32  # query tokens per sequence from which keys and values are expanded
EXPAND_HEAD_DIMS = (32, 64, 128)  # head sizes of the tensor-core attention kernels; smaller heads are padded with zeros


# ---- configuration --------------------------------------------------------------------
@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int
    kv_from: int | None = None


@dataclass(frozen=True)
class Layer:
    mixer: LatentAttention
    ff: int | None  # None: no feed-forward


@dataclass(frozen=True)
class DelunexConfig:
    vocab: int
    width: int
    eps: float
    taps: int
    embedding_scale: float
    logit_scale: float
    layers: tuple[Layer, ...] = field(default_factory=tuple)

    @staticmethod
    def from_dict(c: dict) -> "DelunexConfig":
        layers = []
        for i, entry in enumerate(c["layers"]):
            if entry["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
            m = dict(entry["mixer"])
            mask = dict(m.pop("mask"))
            window = int(mask.pop("size"))
            mixer = LatentAttention(
                heads=int(m.pop("heads")), dim=int(m.pop("dim")), vdim=int(m.pop("vdim")), kv_rank=int(m.pop("kv_rank")),
                scale=float(m.pop("scale")), window=window, kv_from=m.pop("kv_from", None),
            )
            if m or mask:  # a key that is not understood would change what the layer computes
                raise ValueError(f"layer {i}: unknown keys {sorted(m) + sorted(mask)} in its mixer")
            if window < 1:
                raise ValueError(f"layer {i}: a window holds at least the token itself")
            if mixer.kv_from is not None:
                j = mixer.kv_from
                if not 0 <= j < i or layers[j].mixer.kv_from is not None or layers[j].mixer.kv_rank != mixer.kv_rank:
                    raise ValueError(f"layer {i}: kv_from must name an earlier layer with a latent of its own and equal kv_rank")
            mlp = entry.get("mlp")
            if mlp is not None and (mlp["kind"] != "dense" or set(mlp) != {"kind", "ff"}):
                raise ValueError(f"layer {i}: unknown feed-forward {mlp}")
            layers.append(Layer(mixer=mixer, ff=None if mlp is None else int(mlp["ff"])))
        if not layers:
            raise ValueError("a model has at least one layer")
        return DelunexConfig(
            vocab=int(c["vocab"]), width=int(c["width"]), eps=float(c["norm"]["eps"]), taps=int(c["canon"]["taps"]),
            embedding_scale=float(c["embedding"]["scale"]), logit_scale=float(c["logit_scale"]), layers=tuple(layers),
        )

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Checkpoint names and shapes."""
        C = self.width
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab, C), "final.norm": (C,)}
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer.mixer
            out[p + "norm1"] = (C,)
            out[p + "mix.q"] = (m.heads * m.dim, C)
            if m.kv_from is None:
                out[p + "mix.dkv"] = (m.kv_rank, C)
                out[p + "mix.dkv.norm"] = (m.kv_rank,)
            out[p + "mix.uk"] = (m.heads * m.dim, m.kv_rank)
            out[p + "mix.uv"] = (m.heads * m.vdim, m.kv_rank)
            out[p + "mix.g"] = (m.heads, C)
            out[p + "mix.o"] = (C, m.heads * m.vdim)
            if layer.ff is not None:
                out[p + "norm2"] = (C,)
                out[p + "mlp.up"] = (layer.ff, C)
                out[p + "mlp.down"] = (C, layer.ff)
                out[p + "mlp.act"] = (2,)
            out[p + "canon1"] = (C, self.taps)
            out[p + "dwa"] = (i + 2,)
        return out


def padded_head(m: LatentAttention) -> int:
    """Head size the kernels work with: query, key and value heads are padded with zeros to one common size."""
    need = max(m.dim, m.vdim)
    return next((d for d in EXPAND_HEAD_DIMS if d >= need), round_up(need, 8))


# ---- weights as the kernels want them ----------------------------------------------------
@dataclass
class _PackedLayer:
    H: int
    D: int  # padded head size
    r: int  # columns of a cached latent (kv_rank padded to a multiple of 8)
    rank: int
    owner: int  # layer whose latent is read
    window: int
    scale: float
    w_in_t: torch.Tensor  # [C, H * D + own r + gate columns]
    gate_col: int
    dkv_norm: torch.Tensor | None
    w_kv_t: torch.Tensor  # [r, 2 * H * D]
    w_uk: torch.Tensor  # [H, D, r]
    w_uv_t: torch.Tensor  # [H, r, D]
    w_o_t: torch.Tensor  # [H * D, C]
    norm1: torch.Tensor
    norm2: torch.Tensor | None
    w_up: torch.Tensor | None
    w_down_t: torch.Tensor | None
    act: tuple[float, float] | None
    conv: torch.Tensor  # fp32 [taps, C]
    dwa: torch.Tensor  # fp32 [i + 2]


@dataclass
class _Packed:
    emb: torch.Tensor
    one: torch.Tensor
    final_norm: torch.Tensor  # times logit_scale
    layers: list
    stamp: tuple

    @property
    def head(self) -> torch.Tensor:
        return self.emb


# ---- how one forward call is bound to cached state ------------------------------------------
@dataclass
class LatentBinding:
    """Where the new latents go, which cached ones each query sees, and the convolutions' states.

    Queries see the last `window` of the logical keys 0 .. len0 + len1 + step + t - 1 (see `dgpt_latent_attn`).
    keys        host-side bound on the logical keys of any query
    expand      keys and values may be expanded: `latents(layer, n)` gives the latents of the n tokens before the call
                and of its own tokens, per sequence, as [n_seq * (n + T), r]; `context` tokens lie before the call
    """

    layout: Callable[[int], object]
    slot0: torch.Tensor
    len1: torch.Tensor
    keys: int
    start1: torch.Tensor
    len0: torch.Tensor | None = None
    step: torch.Tensor | None = None
    expand: bool = False
    context: int = 0
    latents: Callable[[int, int], torch.Tensor] | None = None
    conv_in: torch.Tensor | None = None  # [n_layer, n_seq, taps - 1, C]
    conv_out: torch.Tensor | None = None
    fmha_impl: int = 0


class DelunexPlan:
    """Buffers for one (n_seq, T) forward and the launch sequence that fills them (see `ForwardPlan`)."""

    def __init__(self, model: "Delunex", n_seq: int, T: int, last_only: bool = False, want_logits: bool = True,
                 rows: int | None = None) -> None:
        """`rows`: the number of rows whose logits are asked for by index at each run (overrides last_only)."""
        cfg, emb = model.config, model.embedding
        self.model, self.n_seq, self.T, self.n = model, n_seq, T, n_seq * T
        self.dev, self.dt = emb.device, emb.dtype
        n, C, V = self.n, cfg.width, cfg.vocab
        self._bufs: dict = {}
        f32 = torch.float32
        self.slab = torch.empty((len(cfg.layers) + 1, n, C), dtype=f32, device=self.dev)
        self.x = [torch.empty((n, C), dtype=f32, device=self.dev) for _ in range(2)]
        self.x1 = torch.empty((n, C), dtype=f32, device=self.dev)
        self.h, self.u, self.y = (torch.empty((n, C), dtype=self.dt, device=self.dev) for _ in range(3))
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

    def expands(self, lw: _PackedLayer, b: LatentBinding) -> bool:
        return b.expand and self.T >= EXPAND_MIN_TOKENS and lw.D in EXPAND_HEAD_DIMS

    def flat(self, layer: int, r: int) -> torch.Tensor:
        """Contiguous copy of the latents this call appends for `layer`."""
        return self._buf(f"flat{layer}", self.n, r)

    def _mixer(self, i: int, lw: _PackedLayer, b: LatentBinding, readers_expand: bool) -> None:
        """self.y = mixer(self.h)"""
        n, n_seq, T, H, D, r = self.n, self.n_seq, self.T, lw.H, lw.D, lw.r
        proj = self._buf("proj", n, lw.w_in_t.shape[1])
        with region("gemm_in"):
            torch.mm(self.h, lw.w_in_t, out=proj)
        q, gate = proj[:, : H * D], proj[:, lw.gate_col : lw.gate_col + H]
        if lw.owner == i:
            ops.latent_append(
                proj[:, H * D : H * D + lw.rank], lw.dkv_norm, self.model.config.eps, b.layout(i), b.slot0, b.step, n_seq=n_seq,
                T=T, r=r, flat=self.flat(i, r) if (readers_expand and b.latents is None) else None, status=self.status,
            )
        o = self._buf("o", n, H * D)
        if self.expands(lw, b):
            context = min(b.context, lw.window - 1)
            lat = self.flat(lw.owner, r) if b.latents is None else b.latents(lw.owner, context)
            kv = self._buf("kv", lat.shape[0], 2 * H * D)
            with region("gemm_kv"):
                torch.mm(lat, lw.w_kv_t, out=kv)
            ops.fmha_window(
                q, kv[:, : H * D], kv[:, H * D :], o, B=n_seq, H=H, D=D, n_keys=context + T, q_offset=context, window=lw.window,
                scale=lw.scale, gate=gate, impl=b.fmha_impl, status=self.status,
            )
        else:
            qa, oa = self._buf("qa", n, H * r), self._buf("oa", n, H * r)
            with region("gemm_absorb"):
                torch.bmm(q.view(n, H, D).transpose(0, 1), lw.w_uk, out=qa.view(n, H, r).transpose(0, 1))
            splits = pick_latent_splits(n, -(-H // 64), min(b.keys, lw.window))
            ws = None
            if splits > 1:
                ws = self._buf("ws", ops.latent_attn_workspace_bytes(n, H, r, splits) // 4, dtype=torch.float32)
            ops.latent_attn(
                qa, b.layout(lw.owner), b.len0, b.start1, b.len1, b.step, oa, n_seq=n_seq, T=T, H=H, r=r, window=lw.window,
                scale=lw.scale, gate=gate, workspace=ws, n_splits=splits, status=self.status,
            )
            with region("gemm_absorb"):
                torch.bmm(oa.view(n, H, r).transpose(0, 1), lw.w_uv_t, out=o.view(n, H, D).transpose(0, 1))
        with region("gemm_proj"):
            torch.mm(o, lw.w_o_t, out=self.y)

    def _feed_forward(self, lw: _PackedLayer) -> None:
        """self.y = W_down xielu(W_up self.u)"""
        ff = lw.w_up.shape[0]
        act = self._buf("act", self.n, ff)
        if self.fused_ff and ff % 16 == 0:
            ops.linear(self.u, lw.w_up, act, xielu=lw.act, status=self.status)
        else:
            up = self._buf("up", self.n, ff)
            with region("gemm_up"):
                torch.mm(self.u, lw.w_up.t(), out=up)
            ops.xielu(up, act, *lw.act)
        with region("gemm_down"):
            torch.mm(act, lw.w_down_t, out=self.y)

    def run(self, ids32: torch.Tensor, b: LatentBinding, rows: torch.Tensor | None = None,
            tap: Callable[[int, torch.Tensor], None] | None = None) -> torch.Tensor | None:
        """`rows`: int32 places (among the n tokens) whose logits are wanted; `tap(i, x)` sees what leaves layer i."""
        with fp32_reductions():
            return self._run(ids32, b, rows, tap)

    def _run(self, ids32, b, rows, tap):
        m = self.model
        cfg, W = m.config, m.packed_weights()
        L, eps, n_seq, T = len(cfg.layers), cfg.eps, self.n_seq, self.T
        expand = {lw.owner for lw in W.layers if self.expands(lw, b)}

        def states(i):
            src = None if b.conv_in is None else b.conv_in[i]
            return src, (None if b.conv_out is None else b.conv_out[i])

        ops.embed_scale(ids32, W.emb, self.slab[0], cfg.embedding_scale)
        s_in, s_out = states(0)
        ops.depth_avg_conv(self.slab, 1, W.one, W.layers[0].conv, self.h, n_seq=n_seq, T=T, state_in=s_in, state_out=s_out)
        x = self.slab[0]
        for i, lw in enumerate(W.layers):
            self._mixer(i, lw, b, i in expand)
            norm = lw.norm1
            if lw.w_up is not None:
                ops.norm_add(self.y, lw.norm1, eps, x, self.x1, rounded=self.u)
                x, norm = self.x1, lw.norm2
                self._feed_forward(lw)
            last = i + 1 == L
            x_next = self.x[i & 1]
            if not last and T == 1:
                ops.layer_tail(self.y, norm, eps, x, self.slab, i + 2, lw.dwa, W.layers[i + 1].conv, b.conv_out[i + 1], x_next, self.h)
            else:
                ops.norm_add(self.y, norm, eps, x, self.slab[i + 1])
                if not last:
                    s_in, s_out = states(i + 1)
                    ops.depth_avg_conv(self.slab, i + 2, lw.dwa, W.layers[i + 1].conv, self.h, n_seq=n_seq, T=T, x=x_next,
                                       state_in=s_in, state_out=s_out)
            if tap is not None:
                tap(i, torch.einsum("j,jnc->nc", lw.dwa, self.slab[: i + 2]) if last else x_next)
            x = x_next
        if self.xn.shape[0] == 0:
            return self.logits
        ops.depth_avg_norm(self.slab, L + 1, W.layers[-1].dwa, W.final_norm, eps, self.xn, rows=self.rows if rows is None else rows)
        if self.logits is None:
            return None
        if self.own_head:
            ops.linear(self.xn, W.emb, self.logits, status=self.status)
        else:
            with region("gemm_logits"):
                torch.mm(self.xn, W.emb.t(), out=self.logits)
        return self.logits


class Delunex(ConfiguredModel):
    def __init__(self, config: DelunexConfig | dict, block_size: int = 32768) -> None:
        """`block_size` only bounds how far the Engine generates (the design has no positions)."""
        cfg = config if isinstance(config, DelunexConfig) else DelunexConfig.from_dict(config)
        super().__init__(cfg, cfg.tensor_shapes(), block_size, cfg.vocab, cfg.width, cfg.layers[0].mixer.heads, len(cfg.layers))
        self.ranks = {i: round_up(l.mixer.kv_rank, 8) for i, l in enumerate(cfg.layers) if l.mixer.kv_from is None}
        self.keep = max(l.mixer.window for l in cfg.layers) - 1

    # ---- weights -------------------------------------------------------------------------
    def pack(self, stamp) -> _Packed:
        cfg = self.config
        emb = self.embedding.detach()
        return _Packed(
            emb=emb, one=torch.ones(1, device=emb.device), final_norm=self.tensor("final.norm").float() * cfg.logit_scale,
            layers=[self._pack_layer(i) for i in range(len(cfg.layers))], stamp=stamp,
        )

    def _pack_layer(self, i: int) -> _PackedLayer:
        cfg = self.config
        m, ff = cfg.layers[i].mixer, cfg.layers[i].ff
        C, H, D, r = cfg.width, m.heads, padded_head(m), round_up(m.kv_rank, 8)

        def w(name):
            return self.tensor(f"l{i}.{name}").detach()

        def heads(t, size, cols):  # [H * size, k] -> [H * D, cols], zero-padded per head and at the end of the rows
            return F.pad(t.view(H, size, -1), (0, cols - t.shape[1], 0, D - size)).reshape(H * D, cols)

        own = m.kv_from is None
        parts = [heads(w("mix.q"), m.dim, C)]
        if own:
            parts.append(F.pad(w("mix.dkv"), (0, 0, 0, r - m.kv_rank)))
        parts.append(F.pad(w("mix.g"), (0, 0, 0, round_up(H, 8) - H)))
        w_kv = torch.cat([heads(w("mix.uk"), m.dim, r), heads(w("mix.uv"), m.vdim, r)]).contiguous()
        w_o = F.pad(w("mix.o").view(C, H, m.vdim), (0, D - m.vdim)).reshape(C, H * D).contiguous()
        act = None
        if ff is not None:
            p, q = w("mlp.act").double().tolist()
            act = (_softplus(p), 0.5 + _softplus(q))
        return _PackedLayer(
            H=H, D=D, r=r, rank=m.kv_rank, owner=i if own else m.kv_from, window=m.window, scale=m.scale,
            w_in_t=torch.cat(parts).contiguous().t(),
            gate_col=H * D + (r if own else 0),
            dkv_norm=w("mix.dkv.norm").float().contiguous() if own else None,
            w_kv_t=w_kv.t(),
            w_uk=w_kv[: H * D].view(H, D, r),
            w_uv_t=w_kv[H * D :].view(H, D, r).transpose(1, 2),
            w_o_t=w_o.t(),
            norm1=w("norm1").float().contiguous(),
            norm2=None if ff is None else w("norm2").float().contiguous(),
            w_up=None if ff is None else w("mlp.up"),
            w_down_t=None if ff is None else w("mlp.down").t(),
            act=act,
            conv=w("canon1").float().t().contiguous(),
            dwa=w("dwa").float().contiguous(),
        )

    # ---- what the Engine needs -------------------------------------------------------------
    def new_cache(self, batch_size: int = 1, seq_len: int = 0) -> LatentCache:
        emb = self.embedding
        cache = LatentCache(batch_size, self.ranks, self.keep, self.n_layer, self.config.taps, self.n_embd, emb.dtype, emb.device)
        if seq_len > 0:
            cache.ensure(seq_len)
        return cache

    def paged_cache(self, n_series, rows_per_series, prefix_len, max_new, page_tokens, pool=None) -> PagedLatentCache:
        assert pool is None, "this model's cache allocates its own pools"
        emb = self.embedding
        return PagedLatentCache(self.ranks, self.keep, self.n_layer, self.config.taps, self.n_embd, n_series, rows_per_series,
                                prefix_len, max_new, emb.dtype, emb.device, page_tokens=page_tokens)

    def prefill_plan(self, cache, members, P, fmha_impl):
        dev = cache.prefix_table.device
        n = len(members)
        table = cache.prefix_table[torch.tensor(members, device=dev)].contiguous()
        zero = torch.zeros(n, dtype=torch.int32, device=dev)
        layouts = {layer: cache.layout(layer, table) for layer in self.ranks}
        states = cache.prompt_states(members)
        bind = LatentBinding(
            layout=layouts.__getitem__, slot0=zero, start1=zero, len1=torch.ones(n, dtype=torch.int32, device=dev), keys=P,
            expand=True, conv_in=states if P == 1 else None, conv_out=states, fmha_impl=fmha_impl if fmha_impl <= 3 else 0,
        )
        return bind, DelunexPlan(self, n, P, last_only=True)

    def decode_plan(self, cache, prompt_lens, max_keys, step, shared, fmha_impl, overlap_prefix, want_logits):
        R, dev = cache.n_rows, prompt_lens.device
        slot0 = torch.full((R,), cache.suffix_slot0, dtype=torch.int32, device=dev)
        layouts = {layer: cache.layout(layer, cache.row_table) for layer in self.ranks}
        bind = LatentBinding(
            layout=layouts.__getitem__, slot0=slot0, start1=slot0, len0=prompt_lens.repeat_interleave(cache.rows_per_series).contiguous(),
            len1=torch.ones(R, dtype=torch.int32, device=dev), step=step, keys=max_keys, conv_in=cache.rows, conv_out=cache.rows,
        )
        return bind, DelunexPlan(self, R, 1, want_logits=want_logits)

    def new_plan(self, n_seq, T, **kw) -> DelunexPlan:
        return DelunexPlan(self, n_seq, T, **kw)

    def step_binding(self, cache: LatentCache, B: int, T: int) -> LatentBinding:
        dev = self.embedding.device
        slot = cache.slot
        start = torch.full((B,), slot, dtype=torch.int32, device=dev)
        state = cache.state
        return LatentBinding(
            layout=cache.layout, slot0=start, start1=torch.zeros_like(start), len1=start + 1, keys=slot + T, expand=True,
            context=slot, latents=lambda layer, n: cache.span(layer, slot - n, slot + T), conv_in=state.source["conv"],
            conv_out=(state.source if T == 1 else state.target)["conv"],
        )


def _softplus(v: float) -> float:
    return math.log1p(math.exp(-abs(v))) + max(v, 0.0)
