"""Small Delunex configurations shared by the tests, and the comparison they use."""

import torch

from oracle import ref_delunex as ref


def mixer(heads, dim, vdim, rank, window, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim**-0.5 if scale is None else scale,
         "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def config(width, vocab, taps, layers, embed_scale=3.0, logit_scale=0.5, eps=1e-5):
    """layers: (mixer, ff or None) each."""
    return {
        "architecture": "Delunex", "width": width, "vocab": vocab, "canon": {"taps": taps}, "norm": {"eps": eps},
        "embedding": {"scale": embed_scale}, "logit_scale": logit_scale,
        "layers": [{"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
                   for m, ff in layers],
    }


CASES = {
    # nothing divides anything: 3 heads, dim != vdim, latent not a multiple of 8, windows that differ along a chain of
    # layers reading one latent (the reader's window larger than the owner's), layers without feed-forward, odd vocabulary
    "odd": config(52, 77, 4, [
        (mixer(3, 12, 20, 20, 9), 70), (mixer(2, 20, 12, 28, 33, scale=0.31), None), (mixer(5, 12, 36, 20, 40, kv_from=0), 44),
        (mixer(1, 44, 8, 28, 1, kv_from=1), 90),
    ], eps=3e-3),
    # tensor-core head sizes, a latent larger than a head, more than 16 heads, one layer's window beyond every sequence
    "wide": config(192, 160, 3, [
        (mixer(18, 32, 32, 144, 70), 256), (mixer(2, 64, 64, 144, 10**6, kv_from=0), None), (mixer(3, 100, 128, 64, 130), 320),
    ], embed_scale=9.0, logit_scale=1.0),
    # one tap (a plain channel gain), one layer, one head
    "tiny": config(16, 24, 1, [(mixer(1, 8, 8, 8, 4), 32)], embed_scale=1.0, logit_scale=2.0),
    # heads larger than the attention kernels that expand keys and values take, many taps, no feed-forward at all
    "big_heads": config(64, 48, 6, [(mixer(2, 160, 136, 40, 50), None), (mixer(2, 136, 160, 40, 25, kv_from=0), None)]),
}


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def build(cfg, seed, dtype, device="cuda", weights=None):
    """(model on the device, the same weights in float64 for the oracle)"""
    from diff_gpt_b200.model.registry import model_class

    w = ref.random_model(cfg, seed) if weights is None else weights
    m = model_class(cfg).from_config(cfg).to(dtype)
    m.load_tensors(w)
    return m.to(device).eval(), {k: v.double() for k, v in w.items()}


TOL = {torch.float32: 1e-4, torch.bfloat16: 8e-2}  # of the rms, worst row


def error(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest over the rows of rms(got - want) / rms over all of want."""
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape
    return ((got - want).pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt()).item()
