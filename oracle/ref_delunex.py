"""Plain CPU restatement of the Delunex decoder (test infrastructure).

One function per mechanism, written for clarity: whole sequences, dense score
matrices, no cache, no fusion.  The product never imports this file and this
file imports nothing of the product.  Everything runs in the dtype of the
weights it is given (tests use float64 or float32).

Notation: T tokens, C channels, H heads, d query/key size, e value size, r
latent size.  A weight `name` is stored [out, in] and applied as `x @ w.T`.
A model is (cfg, w): cfg the parsed configuration, w a dict of tensors.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def embed(ids: torch.Tensor, table: torch.Tensor, scale: float) -> torch.Tensor:
    return table[ids] * scale


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """out[t, c] = sum_j w[c, j] x[t - (taps - 1) + j, c], zeros before the first token; x [T, C], w [C, taps]."""
    T, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x])
    out = torch.zeros_like(x)
    for j in range(taps):
        out += w[:, j] * padded[j : j + T]
    return out


def window_mask(T: int, size: int) -> torch.Tensor:
    """[T, T] bool: query i (row) sees key j (column) when 0 <= i - j < size."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def latent(h: torch.Tensor, w_dkv: torch.Tensor, w_norm: torch.Tensor, eps: float) -> torch.Tensor:
    """[T, r]: what a layer's cache holds."""
    return rms_norm(h @ w_dkv.T, w_norm, eps)


def latent_attention(h, c, w_q, w_uk, w_uv, w_g, w_o, heads: int, scale: float, size: int) -> torch.Tensor:
    """Softmax attention over the last `size` tokens with keys and values expanded from the latent c, one output gate
    per head read from h."""
    T = h.shape[0]
    q = (h @ w_q.T).view(T, heads, -1)
    k = (c @ w_uk.T).view(T, heads, -1)
    v = (c @ w_uv.T).view(T, heads, -1)
    gate = torch.sigmoid(h @ w_g.T)  # [T, H]
    seen = window_mask(T, size)
    out = torch.zeros(T, heads, v.shape[-1], dtype=h.dtype)
    for n in range(heads):
        s = (q[:, n] @ k[:, n].T) * scale
        p = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1)
        out[:, n] = (p @ v[:, n]) * gate[:, n : n + 1]
    return out.reshape(T, -1) @ w_o.T


def xielu(z: torch.Tensor, pq: torch.Tensor) -> torch.Tensor:
    """softplus(p) z^2 + z/2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z/2 at and below it."""
    ap = torch.nn.functional.softplus(pq[0])
    an = 0.5 + torch.nn.functional.softplus(pq[1])
    low = torch.clamp(z, max=0.0)
    return torch.where(z > 0, ap * z * z, an * (torch.expm1(low) - low)) + z / 2


def feed_forward(x, w_up, w_down, pq) -> torch.Tensor:
    return xielu(x @ w_up.T, pq) @ w_down.T


def depth_average(states: list, a: torch.Tensor) -> torch.Tensor:
    out = torch.zeros_like(states[0])
    for j, s in enumerate(states):
        out = out + a[j] * s
    return out


def forward(cfg: dict, w: dict, ids, keep_layers: bool = False):
    """Logits [T, V] of one sequence; with keep_layers also what leaves every layer, [L, T, C]."""
    eps = cfg["norm"]["eps"]
    x = embed(torch.as_tensor(ids, dtype=torch.long), w["embed"], cfg["embedding"]["scale"])
    states, latents, after = [x], {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        assert layer["type"] == "latent_attention"
        h = x + causal_conv(x, w[p + "canon1"])
        if m.get("kv_from") is None:
            latents[i] = latent(h, w[p + "mix.dkv"], w[p + "mix.dkv.norm"], eps)
        c = latents[i if m.get("kv_from") is None else m["kv_from"]]
        y = latent_attention(h, c, w[p + "mix.q"], w[p + "mix.uk"], w[p + "mix.uv"], w[p + "mix.g"], w[p + "mix.o"],
                             m["heads"], m["scale"], m["mask"]["size"])
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(x, w[p + "mlp.up"], w[p + "mlp.down"], w[p + "mlp.act"])
            x = x + rms_norm(y, w[p + "norm2"], eps)
        states.append(x)
        x = depth_average(states, w[p + "dwa"])
        after.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
    return (logits, torch.stack(after)) if keep_layers else logits


# ---- small random models for the tests -------------------------------------------------
def random_model(cfg: dict, seed: int, std: float = 0.4) -> dict:
    """Weights for a configuration, float32 but representable in bfloat16, so that both number formats start from the
    same numbers.  Norm weights scatter around 1, the averages' last weight around 1 and the others around 0."""
    g = torch.Generator().manual_seed(seed)
    C, taps = cfg["width"], cfg["canon"]["taps"]

    def lin(o, i):
        return torch.randn(o, i, generator=g) * (std * 2.0 / math.sqrt(i))

    def near(v, *s):
        return v + 0.2 * torch.randn(*s, generator=g)

    w = {"embed": torch.randn(cfg["vocab"], C, generator=g) * (std / 4), "final.norm": near(1.0, C)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, e, r = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        w[p + "norm1"] = near(0.7, C)
        w[p + "mix.q"] = lin(H * d, C)
        if m.get("kv_from") is None:
            w[p + "mix.dkv"] = lin(r, C)
            w[p + "mix.dkv.norm"] = near(1.0, r)
        w[p + "mix.uk"], w[p + "mix.uv"] = lin(H * d, r) * 2, lin(H * e, r) * 2
        w[p + "mix.g"], w[p + "mix.o"] = lin(H, C), lin(C, H * e)
        if layer.get("mlp") is not None:
            f = layer["mlp"]["ff"]
            w[p + "norm2"] = near(0.7, C)
            w[p + "mlp.up"], w[p + "mlp.down"] = lin(f, C), lin(C, f)
            w[p + "mlp.act"] = near(0.3, 2)
        w[p + "canon1"] = 0.3 * torch.randn(C, taps, generator=g)
        a = 0.2 * torch.randn(i + 2, generator=g)
        a[-1] += 1.0
        w[p + "dwa"] = a
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}
