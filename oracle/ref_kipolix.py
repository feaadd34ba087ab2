"""Plain CPU restatement of the Kipolix decoder (test infrastructure).

One function per mechanism, written for clarity: whole sequences, dense score matrices, the recurrence token by token,
no cache, no fusion.  The product never imports this file and this file imports nothing of the product.  Everything runs
in the dtype of the weights it is given (tests use float64).

Notation: T tokens, C channels, H heads, G key/value heads, d query/key size, e value size, S residual streams.
A weight `name` is stored [out, in] and applied as `x @ w.T`.  A model is (cfg, w): cfg the parsed configuration, w a
dict of tensors.
"""

from __future__ import annotations

import math

import torch


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_one_plus(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * (1 + w)


def bigram_rows(ids: torch.Tensor, buckets: int, mul_prev: int, mul_cur: int) -> torch.Tensor:
    """Row of the bigram table for every token of a sequence; the first token has a row of its own, the last one."""
    rows = torch.full_like(ids, buckets)
    rows[1:] = (ids[:-1] * mul_prev + ids[1:] * mul_cur) % buckets
    return rows


def embed(ids: torch.Tensor, table: torch.Tensor, bigram: torch.Tensor, mul_prev: int, mul_cur: int) -> torch.Tensor:
    return table[ids] + bigram[bigram_rows(ids, bigram.shape[0] - 1, mul_prev, mul_cur)]


def angles(T: int, dims: int, base: float, first: int = 0) -> torch.Tensor:
    """[T, dims / 2] in float64: position times base^(-2 i / dims)."""
    f = torch.tensor(base, dtype=torch.float64) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    return (first + torch.arange(T, dtype=torch.float64))[:, None] * f


def rotate_half(x: torch.Tensor, dims: int, base: float, first: int = 0) -> torch.Tensor:
    """x [T, heads, d]: dimension i < dims/2 is paired with i + dims/2; dimensions from `dims` on pass."""
    a = angles(x.shape[0], dims, base, first)[:, None]
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., : dims // 2], x[..., dims // 2 : dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def rotate_pairs(x: torch.Tensor, dims: int, base: float, first: int = 0) -> torch.Tensor:
    """x [T, heads, d]: dimension 2 i is paired with 2 i + 1."""
    a = angles(x.shape[0], dims, base, first)[:, None]
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def retention(q, k, v, decay, state=None):
    """o_t = S_t^T q_t with S_t = decay S_(t-1) + k_t v_t^T per head; q, k [T, H, d] (k scaled), v [T, H, e], decay [H].
    Returns (o [T, H, e], S [H, d, e])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    lam = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    out = []
    for t in range(T):
        S = lam * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def retention_mixer(h, m: dict, w_q, w_k, w_v, w_g, w_o, eps: float) -> torch.Tensor:
    T, H, d = h.shape[0], m["heads"], m["dim"]
    rot = m["rot"]
    q = rotate_half((h @ w_q.T).view(T, H, d), rot["dims"], rot["base"])
    k = rotate_half((h @ w_k.T).view(T, H, d), rot["dims"], rot["base"]) * d**-0.5
    o, _ = retention(q, k, (h @ w_v.T).view(T, H, m["vdim"]), m["decay"])
    g = h @ w_g.T
    return (unit_rms(o, eps).reshape(T, -1) * silu(g)) @ w_o.T


def visible(T: int, size: int, keep_first: int) -> torch.Tensor:
    """[T, T] bool: query i (row) sees key j (column) when j <= i and (i - j < size or j < keep_first)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_attention(q, k, v, seen, scale: float) -> torch.Tensor:
    """q [Tq, H, d], k [T, G, d], v [T, G, e], seen [Tq, T]; query head n reads key/value head n // (H / G)."""
    H, per = q.shape[1], q.shape[1] // k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for n in range(H):
        s = (q[:, n] @ k[:, n // per].T) * scale
        out[:, n] = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ v[:, n // per]
    return out


def attention_mixer(h, m: dict, w_q, w_k, w_v, q_norm, k_norm, w_o, eps: float) -> torch.Tensor:
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    rot = m["rot"]
    q = (unit_rms(h @ w_q.T, eps) * q_norm).view(T, H, d)
    k = (unit_rms(h @ w_k.T, eps) * k_norm).view(T, G, d)
    q, k = (rotate_pairs(x, rot["dims"], rot["base"]) for x in (q, k))
    seen = visible(T, m["mask"]["size"], m["mask"]["keep_first"])
    return softmax_attention(q, k, (h @ w_v.T).view(T, G, m["vdim"]), seen, m["scale"]).reshape(T, -1) @ w_o.T


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def feed_forward(h, w_gate, w_up, w_down) -> torch.Tensor:
    return (silu(h @ w_gate.T) * (h @ w_up.T)) @ w_down.T


def stream_in(x: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """x [S, T, C] -> sum_s a[s] x_s."""
    return torch.einsum("s,stc->tc", a, x)


def stream_out(x: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """New stream t = sum_s mix[s, t] x_s + out[t] y, from the old streams."""
    return torch.einsum("su,stc->utc", mix, x) + out[:, None, None] * y


def runs(cfg: dict) -> list[int]:
    """The layers in the order in which they run; a looped stretch is there as often as it runs."""
    n, loop = len(cfg["layers"]), cfg["loop"]
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg: dict, w: dict, ids, keep_layers: bool = False):
    """Logits [T, V] of one sequence; with keep_layers also the sum of the streams after every layer run, [runs, T, C]."""
    eps, big = cfg["norm"]["eps"], cfg["embedding"]["bigram"]
    e = embed(torch.as_tensor(ids, dtype=torch.long), w["embed"], w["bigram"], big["mul_prev"], big["mul_cur"])
    x = e.expand(cfg["streams"], *e.shape)
    after = []
    for i in runs(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        m = layer["mixer"]

        def sub(x, q, fn):
            hc = f"{p}hc{q}."
            y = fn(norm_one_plus(stream_in(x, w[hc + "in"]), w[f"{p}norm{q}"], eps))
            return stream_out(x, w[hc + "mix"], w[hc + "out"], y)

        mix = [w[p + "mix." + n] for n in ("q", "k", "v")]
        if layer["type"] == "retention":
            x = sub(x, 1, lambda h: retention_mixer(h, m, *mix, w[p + "mix.g"], w[p + "mix.o"], eps))
        else:
            assert layer["type"] == "attention"
            x = sub(x, 1, lambda h: attention_mixer(h, m, *mix, w[p + "mix.q.norm"], w[p + "mix.k.norm"], w[p + "mix.o"], eps))
        if layer.get("mlp") is not None:
            x = sub(x, 2, lambda h: feed_forward(h, *[w[p + "mlp." + n] for n in ("gate", "up", "down")]))
        after.append(x.sum(0))
    logits = norm_one_plus(x.sum(0), w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(after)) if keep_layers else logits


# ---- small random models for the tests -------------------------------------------------
def random_model(cfg: dict, seed: int, std: float = 0.4) -> dict:
    """Weights for a configuration, float32 but representable in bfloat16, so that both number formats start from the
    same numbers.  Norm weights scatter around 0 (1 for the query and key norms); the streams differ from the first
    sublayer on."""
    g = torch.Generator().manual_seed(seed)
    C, S = cfg["width"], cfg["streams"]

    def lin(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (2.0 * gain * std / math.sqrt(i))

    def near(v, *s):
        return v + 0.2 * torch.randn(*s, generator=g)

    w = {"embed": torch.randn(cfg["vocab"], C, generator=g), "final.norm": near(0.0, C), "head": lin(cfg["vocab"], C),
         "bigram": 0.7 * torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, C, generator=g)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, e = m["heads"], m["dim"], m["vdim"]
        G = H if layer["type"] == "retention" else m["kv_heads"]
        w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"] = lin(H * d, C), lin(G * d, C), lin(G * e, C)
        if layer["type"] == "retention":
            w[p + "mix.g"] = lin(H * e, C)
        else:
            w[p + "mix.q.norm"], w[p + "mix.k.norm"] = near(1.3, H * d), near(1.3, G * d)
        w[p + "mix.o"] = lin(C, H * e)
        w[p + "norm1"] = near(0.0, C)
        subs = (1,)
        if layer.get("mlp") is not None:
            f, subs = layer["mlp"]["ff"], (1, 2)
            w[p + "norm2"] = near(0.0, C)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = lin(f, C), lin(f, C), lin(C, f)
        for q in subs:
            w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"] = near(1.0 / S, S), 0.5 * near(0.8, S)
            w[f"{p}hc{q}.mix"] = 0.9 * torch.eye(S) + 0.1 * torch.randn(S, S, generator=g)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}
