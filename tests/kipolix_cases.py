"""Small Kipolix configurations shared by the tests, and the comparison they use."""

import torch

from delunex_cases import TOL, error, tokens  # noqa: F401  (the same comparison)
from oracle import ref_kipolix as ref


def retention(heads, dim, vdim, decay, rot=None, base=10000.0):
    return "retention", {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay),
                         "rot": {"dims": dim if rot is None else rot, "base": base}}


def attention(heads, kv_heads, dim, vdim, window, keep_first, scale=None, rot=None, base=10000.0):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                         "scale": dim**-0.5 if scale is None else scale, "rot": {"dims": dim if rot is None else rot, "base": base},
                         "mask": {"size": window, "keep_first": keep_first}}


def config(width, vocab, layers, streams=3, loop=(0, 0, 1), buckets=61, mul=(31, 5), eps=1e-5):
    """layers: ((type, mixer), ff or None) each."""
    return {
        "architecture": "Kipolix", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps},
        "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}},
        "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]},
        "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers],
    }


CASES = {
    # nothing divides anything: odd sizes, value size != key size both ways, partial rotation, three query heads per key/value
    # head, one stream too many for a power of two, windows and kept tokens that differ between layers, a looped stretch that
    # starts at the first layer and holds both kinds of mixer, layers without feed-forward, an odd vocabulary, a strong decay
    "odd": config(52, 77, [
        (attention(6, 2, 12, 20, 9, 3, scale=0.31, rot=6, base=500.0), 70), (retention(3, 20, 12, (0.9, 0.99, 0.3), rot=14), None),
        (attention(5, 5, 20, 12, 33, 0, rot=8), 44), (retention(2, 10, 36, (0.95, 1.0)), 90), (attention(3, 1, 36, 8, 1, 11), None),
    ], streams=5, loop=(0, 2, 3), eps=3e-3),
    # tensor-core head sizes, key/value heads shared by 4, 9 and 1 query heads, chunked retention with two blocks of key and
    # value columns, one window beyond every sequence, a stretch run twice in the middle
    "wide": config(192, 160, [
        (retention(4, 64, 48, (0.97, 0.99, 0.999, 0.8)), 256), (attention(8, 2, 64, 64, 70, 5), 320),
        (retention(2, 96, 104, (0.95, 0.9995), rot=64), None), (attention(9, 1, 32, 24, 10**6, 4), 256),
        (attention(2, 2, 128, 100, 130, 140), 256),
    ], streams=4, loop=(1, 3, 2)),
    # one stream, one layer run once, one head, sizes of one and two
    "tiny": config(16, 24, [(attention(1, 1, 8, 8, 4, 1, rot=2), 32)], streams=1, loop=(0, 1, 1), buckets=1, mul=(1, 1)),
    # heads beyond the prefill attention kernels and the chunked retention, more value columns than one slice, two streams,
    # the whole model looped
    "big_heads": config(64, 48, [
        (retention(2, 136, 40, (0.9, 0.98)), None), (attention(2, 1, 160, 136, 50, 7), None), (retention(1, 32, 200, (0.99,)), 96),
    ], streams=2, loop=(0, 3, 2)),
}


def build(cfg, seed, dtype, device="cuda", weights=None):
    """(model on the device, the same weights in float64 for the oracle)"""
    from diff_gpt_b200.model.registry import model_class

    w = ref.random_model(cfg, seed) if weights is None else weights
    m = model_class(cfg).from_config(cfg).to(dtype)
    m.load_tensors(w)
    return m.to(device).eval(), {k: v.double() for k, v in w.items()}
