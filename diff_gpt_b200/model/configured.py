"""What models built from a configuration share: parameters under their checkpoint names, loading, and the forward calls
behind a cache of rows (whole prompts, portions, single tokens)."""

from __future__ import annotations

import contextlib
from abc import abstractmethod
from typing import Callable

import torch
import torch.nn as nn
import torch.nn.functional as F

from .gpt import DeviceModel, _sm_count
from .kv_cache import RowCache

FUSED_FF_MIN_ROWS = 256  # rows from which the up projection runs on the library's GEMM with the activation fused


@contextlib.contextmanager
def fp32_reductions():
    """bf16 products accumulate and reduce in fp32 (split-K partial sums included)."""
    m = torch.backends.cuda.matmul
    was = m.allow_bf16_reduced_precision_reduction
    m.allow_bf16_reduced_precision_reduction = False
    try:
        yield
    finally:
        m.allow_bf16_reduced_precision_reduction = was


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


def pick_latent_splits(rows: int, head_groups: int, keys: int) -> int:
    """Attention over cached rows: CTAs per row along the keys: enough that every multiprocessor has one, each with a 128-key tile at least."""
    ctas = max(1, rows * head_groups)
    if ctas >= _sm_count() or keys <= 128:
        return 1
    return max(1, min(_sm_count() // ctas, -(-keys // 128), 64))


class ConfiguredModel(DeviceModel):
    """Parameters are held under their checkpoint names with dots replaced (`l0.mix.q` -> `l0__mix__q`).

    A subclass gives the launch sequence of a forward (`new_plan`) and how a step is bound to a cache (`step_binding`).
    """

    def __init__(self, config, shapes: dict[str, tuple[int, ...]], block_size: int, vocab: int, width: int, heads: int, layers: int) -> None:
        super().__init__(block_size=block_size, vocab_size=vocab, n_embd=width, n_head=heads, n_layer=layers)
        self.config = config
        for name, shape in shapes.items():
            self.register_parameter(name.replace(".", "__"), nn.Parameter(torch.zeros(shape), requires_grad=False))
        self._packed = None
        self._decode_plan = None  # the last single-token plan of `forward` / `logits_at`

    @classmethod
    def from_config(cls, config: dict):
        return cls(config)

    def load_tensors(self, tensors: dict) -> None:
        want = self.config.tensor_shapes()
        missing, extra = sorted(set(want) - set(tensors)), sorted(set(tensors) - set(want))
        if missing or extra:
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:4]}, unknown {extra[:4]}")
        with torch.no_grad():
            for name, shape in want.items():
                if tuple(tensors[name].shape) != shape:
                    raise ValueError(f"{name}: shape {tuple(tensors[name].shape)}, expected {shape}")
                self.tensor(name).copy_(tensors[name])

    def tensor(self, name: str) -> torch.Tensor:
        return getattr(self, name.replace(".", "__"))

    @property
    def embedding(self) -> torch.Tensor:
        return self.embed

    @property
    def device_type(self) -> str:
        return str(self.embed.device.type)

    def packed_weights(self):
        stamp = tuple((p.data_ptr(), p._version, p.dtype) for p in self.parameters())
        if self._packed is None or self._packed.stamp != stamp:
            with torch.no_grad():
                self._packed = self.pack(stamp)
        return self._packed

    @abstractmethod
    def pack(self, stamp: tuple):
        """Weights as the kernels want them, with `stamp` kept on the result."""

    @abstractmethod
    def new_plan(self, n_seq: int, T: int, **kw):
        ...

    @abstractmethod
    def step_binding(self, cache: RowCache, B: int, T: int):
        """How the next T tokens of each sequence are bound to a cache that has room for them."""

    # ---- forward behind a cache ----------------------------------------------------------------
    def _step(self, idx: torch.Tensor, cache: RowCache, rows: torch.Tensor | None, tap: Callable | None = None) -> torch.Tensor:
        B, T = idx.shape
        assert cache.batch_size == B
        cache.ensure(T)
        bind = self.step_binding(cache, B, T)
        n_rows = B * T if rows is None else rows.numel()
        plan = self._decode_plan
        if T > 1 or plan is None or plan.n_seq != B or plan.xn.shape[0] != n_rows or plan.dt != self.embedding.dtype:
            plan = self.new_plan(B, T, rows=n_rows)
            if T == 1:
                self._decode_plan = plan
        logits = plan.run(idx.reshape(-1).to(torch.int32), bind, None if rows is None else rows.to(torch.int32), tap)
        if T > 1:
            cache.state.flip()
        cache.pos += T
        if int(plan.status.item()):
            raise RuntimeError(f"device-side status {int(plan.status.item())}: a cache slot was out of range, or a bounded wait ran out")
        return logits

    @torch.inference_mode()
    def logits_at(self, idx, cache, rows):
        return self._step(idx, cache, rows)

    def forward(self, idx: torch.Tensor, targets: torch.Tensor | None = None, kv_cache: RowCache | None = None):
        if not idx.is_cuda:
            raise RuntimeError(f"diff_gpt_b200.{type(self).__name__} runs on CUDA only; there is no CPU path")
        B, T = idx.shape
        with torch.inference_mode():
            cache = self.new_cache(B, T) if kv_cache is None else kv_cache
            logits = self._step(idx, cache, None).view(B, T, self.vocab_size).clone()
        loss = None
        if targets is not None:
            loss = F.cross_entropy(logits.view(-1, self.vocab_size).float(), targets.view(-1))
        return logits, loss

    @torch.inference_mode()
    def generate(self, idx: torch.Tensor, max_new_tokens: int, sampler, seed: int | None = None):
        """Prompt, then one token at a time through a cache."""
        rng = None
        if seed is not None:
            rng = torch.Generator(device=idx.device)
            rng.manual_seed(seed)
        B, T = idx.shape
        out = torch.zeros((B, T + max_new_tokens), dtype=torch.int64, device=idx.device)
        out[:, :T] = idx
        cache = self.new_cache(B, T + max_new_tokens)
        new = idx
        for cur in range(T, T + max_new_tokens):
            logits = self(new, kv_cache=cache)[0][:, -1]
            if sampler is not None:
                new = sampler(logits, rng=rng).reshape(B, 1)
            else:
                new = torch.multinomial(F.softmax(logits.float(), dim=-1), num_samples=1, generator=rng)
            out[:, cur] = new.reshape(-1)
        return out
