"""Delunex on the host: configuration, checkpoint folders, caches' bookkeeping, the plain implementation itself."""

import copy
import json
import math

import pytest
import torch

from delunex_cases import CASES, build, config, mixer, tokens
from oracle import ref_delunex as ref


def test_configuration_is_read_and_refused():
    from diff_gpt_b200.model.delunex import DelunexConfig

    cfg = DelunexConfig.from_dict(CASES["odd"])
    assert [l.mixer.window for l in cfg.layers] == [9, 33, 40, 1] and [l.ff for l in cfg.layers] == [70, None, 44, 90]
    assert cfg.layers[2].mixer.kv_from == 0 and cfg.taps == 4 and cfg.eps == 3e-3

    def broken(change):
        c = copy.deepcopy(CASES["odd"])
        change(c)
        with pytest.raises((ValueError, KeyError)):
            DelunexConfig.from_dict(c)

    broken(lambda c: c["layers"][0].update(type="something else"))
    broken(lambda c: c["layers"][0]["mixer"].update(sink=4))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].update(first=4))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=2))  # layer 2 has no latent of its own
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=3))
    broken(lambda c: c["layers"][2]["mixer"].update(kv_rank=24))  # not the owner's size
    broken(lambda c: c.update(layers=[]))
    broken(lambda c: c.pop("logit_scale"))


def test_checkpoint_folder_round_trip(tmp_path):
    from diff_gpt_b200 import Delunex, GPT, load_model
    from diff_gpt_b200.model.registry import model_class
    from diff_gpt_b200.weights import read_safetensors, write_safetensors

    cfg = CASES["odd"]
    w = {k: v.to(torch.bfloat16) for k, v in ref.random_model(cfg, 1).items()}
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), {**w})
    back = read_safetensors(str(tmp_path / "model.safetensors"))
    assert set(back) == set(w) and all(torch.equal(back[k], w[k]) for k in w)
    for dtype in (torch.float32, torch.bfloat16):
        m = load_model(str(tmp_path), dtype, "cpu")
        assert isinstance(m, Delunex) and m.embedding.dtype == dtype
        assert all(torch.equal(m.tensor(k).to(torch.bfloat16), w[k]) for k in w)
    write_safetensors(str(tmp_path / "model.safetensors"), {k: v for k, v in w.items() if k != "l1.dwa"})
    with pytest.raises(ValueError, match="missing"):
        load_model(str(tmp_path), torch.float32, "cpu")
    assert model_class({"architecture": "GPT"}) is GPT
    with pytest.raises(ValueError, match="unknown architecture"):
        model_class({"architecture": "nothing"})
    # the other registered class goes through the same folder
    g = GPT(vocab_size=64, n_embd=32, block_size=16, n_head=4, n_layer=2)
    (tmp_path / "config.json").write_text(json.dumps(dict(architecture="GPT", vocab_size=64, n_embd=32, block_size=16, n_head=4, n_layer=2)))
    write_safetensors(str(tmp_path / "model.safetensors"), {k: v for k, v in g.state_dict().items() if k != "lm_head.weight"})
    h = load_model(str(tmp_path), torch.float32, "cpu")
    assert all(torch.equal(a, b) for a, b in zip(g.state_dict().values(), h.state_dict().values()))


def test_reader_refuses_a_header_that_lies(tmp_path):
    from diff_gpt_b200.weights import read_safetensors, write_safetensors

    p = tmp_path / "x.safetensors"
    write_safetensors(str(p), {"a": torch.arange(6, dtype=torch.int32).view(2, 3), "b": torch.ones(3)})
    assert read_safetensors(str(p))["a"].tolist() == [[0, 1, 2], [3, 4, 5]]
    p.write_bytes(p.read_bytes()[:-4])
    with pytest.raises(ValueError, match="does not fit"):
        read_safetensors(str(p))


def test_packed_weights_pad_with_zeros_only():
    """Padded heads, latents and gate columns must not change any product."""
    m, w = build(CASES["odd"], 3, torch.float32, "cpu")
    h = torch.randn(5, 52, generator=torch.Generator().manual_seed(0))
    c = torch.randn(5, 20, generator=torch.Generator().manual_seed(1))
    p = m.packed_weights().layers[2]
    assert (p.H, p.D, p.r, p.owner, p.dkv_norm) == (5, 64, 24, 0, None)
    q = (h @ p.w_in_t)[:, : 5 * 64].view(5, 5, 64)
    assert torch.allclose(q[..., :12], (h @ w["l2.mix.q"].float().T).view(5, 5, 12), atol=1e-5) and bool((q[..., 12:] == 0).all())
    assert torch.allclose((h @ p.w_in_t)[:, p.gate_col : p.gate_col + 5], h @ w["l2.mix.g"].float().T, atol=1e-5)
    cp = torch.nn.functional.pad(c, (0, 4), value=7.0)  # what lies in the padding columns must not matter
    kv = (cp @ p.w_kv_t).view(5, 2, 5, 64)
    assert torch.allclose(kv[:, 0, :, :12], (c @ w["l2.mix.uk"].float().T).view(5, 5, 12), atol=1e-5)
    assert torch.allclose(kv[:, 1, :, :36], (c @ w["l2.mix.uv"].float().T).view(5, 5, 36), atol=1e-5)
    assert bool((kv[:, 0, :, 12:] == 0).all()) and bool((kv[:, 1, :, 36:] == 0).all())
    assert m.packed_weights() is m.packed_weights()
    m.tensor("l0.dwa").mul_(2.0)
    assert torch.equal(m.packed_weights().layers[0].dwa, 2 * w["l0.dwa"].float())


def test_latent_cache_slides_without_losing_what_can_be_seen():
    """Latents are tagged with their position; whatever the portions, the last `keep` tokens before each new one are in
    place, also after the slots were taken over by another request."""
    from diff_gpt_b200.model.kv_cache import LatentCache

    keep = 37
    cache = LatentCache(2, {0: 8, 3: 16}, keep, n_layer=4, taps=3, width=5, dtype=torch.float32, device="cpu")
    g = torch.Generator().manual_seed(5)
    moved = 0
    for _ in range(3):
        cache.reset()
        assert cache.get_pos() == 0 and cache.slot == 0
        while cache.pos < 6000:
            T = int(torch.randint(1, 3, (1,), generator=g)) if cache.pos % 5 else int(torch.randint(1, 400, (1,), generator=g))
            cache.ensure(T)
            slot, before = cache.slot, min(cache.pos, keep)
            moved += cache.base > 0
            for layer in (0, 3):
                assert slot + T <= cache.latents[layer].shape[1] == cache.capacity
                seen = cache.span(layer, slot - before, slot).view(2, before, cache.ranks[layer])
                assert torch.equal(seen[:, :, 0], torch.arange(cache.pos - before, cache.pos, dtype=torch.float32).expand(2, -1))
                cache.latents[layer][:, slot : slot + T] = torch.arange(cache.pos, cache.pos + T, dtype=torch.float32)[None, :, None]
            cache.pos += T
    assert moved and cache.capacity < 3000  # bounded by the window, not by the sequence


def test_latent_cache_without_a_window_keeps_everything():
    from diff_gpt_b200.model.kv_cache import LatentCache

    cache = LatentCache(1, {0: 8}, None, n_layer=1, taps=2, width=4, dtype=torch.float32, device="cpu")
    for T in (700, 1, 900, 2000):
        cache.ensure(T)
        assert cache.base == 0
        cache.latents[0][:, cache.slot : cache.slot + T] = torch.arange(cache.pos, cache.pos + T, dtype=torch.float32)[None, :, None]
        cache.pos += T
    assert torch.equal(cache.span(0, 0, 3601)[:, 0], torch.arange(3601.0))


@pytest.mark.parametrize("keep,pt,G", [(0, 4, 30), (3, 4, 30), (4, 4, 30), (5, 4, 30), (63, 64, 400), (200, 16, 90), (None, 8, 40)])
def test_ring_of_own_pages_never_overwrites_a_visible_token(keep, pt, G):
    """Walk through G generated tokens writing each one's number at the place its table entry names: the last `keep`
    before a new one must still be there."""
    from diff_gpt_b200.model.kv_cache import PagedLatentCache

    c = PagedLatentCache({1: 8}, keep, n_layer=2, taps=2, width=4, n_series=2, rows_per_series=3, prefix_len=9, max_new=G,
                         dtype=torch.float32, device="cpu", page_tokens=pt)
    assert c.suffix_slot0 == -(-9 // pt) * pt and c.row_table.shape == (6, c.suffix_slot0 // pt + -(-G // pt))
    assert c.row_table[0, 0] == c.row_table[2, 0] != c.row_table[3, 0]
    store = {}

    def place(row, g):
        slot = c.suffix_slot0 + g
        return int(c.row_table[row, slot // pt]), slot % pt

    for g in range(G):
        for row in range(6):
            store[place(row, g)] = (row, g)
        lo = 0 if keep is None else max(0, g - keep)
        for row in range(6):
            assert all(store[place(row, k)] == (row, k) for k in range(lo, g + 1))
    n_prefix = 2 * (c.suffix_slot0 // pt)
    assert int(c.row_table[:, c.suffix_slot0 // pt :].min()) >= n_prefix and c.pools[1].shape[0] == n_prefix + 6 * c.ring_pages
    if keep is not None:
        assert c.ring_pages <= -(-keep // pt) + 1


def test_rows_start_from_their_prompts_convolution_state():
    from diff_gpt_b200.model.kv_cache import PagedLatentCache

    c = PagedLatentCache({0: 8}, 3, n_layer=2, taps=3, width=4, n_series=3, rows_per_series=2, prefix_len=5, max_new=4,
                         dtype=torch.float32, device="cpu")
    a, b = c.prompt_states([0, 2]), c.prompt_states([1])
    a[:, 0], a[:, 1], b[:, 0] = 1.0, 3.0, 2.0
    c.prompts_ready()
    assert c.rows[1, :, 1, 2].tolist() == [1, 1, 2, 2, 3, 3]
    c.begin_prompts()
    assert bool((a == 0).all()) and bool((b == 0).all())


def test_split_policy():
    from diff_gpt_b200.model.delunex import pick_latent_splits

    assert pick_latent_splits(4096, 1, 1024) == 1
    assert pick_latent_splits(1, 1, 128) == 1
    assert pick_latent_splits(1, 1, 1024) == 8  # one tile each
    assert pick_latent_splits(32, 1, 4096) == 4 and pick_latent_splits(1, 1, 10**6) == 64


# ---- the plain implementation: facts that do not depend on the product ------------------------
def test_plain_window_and_convolution_by_hand():
    assert ref.window_mask(4, 2).tolist() == [[True, False, False, False], [True, True, False, False],
                                              [False, True, True, False], [False, False, True, True]]
    x = torch.arange(1.0, 5.0)[:, None].double()
    w = torch.tensor([[10.0, 1.0, 0.1]]).double()
    assert ref.causal_conv(x, w)[:, 0].tolist() == pytest.approx([0.1, 1.2, 10 + 2 + 0.3, 20 + 3 + 0.4])
    z = torch.tensor([-3.0, 0.0, 2.0]).double()
    sp = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.4))
    want = [sp[1] * (math.exp(-3) - 1 + 3) - 1.5, 0.0, sp[0] * 4 + 1]
    assert ref.xielu(z, torch.tensor([0.3, -0.4]).double()).tolist() == pytest.approx(want)


def test_plain_forward_is_causal_and_limited_by_the_windows():
    """A token changes nothing before it, and nothing past the reach of one layer (window and taps)."""
    cfg = config(20, 30, 3, [(mixer(2, 6, 6, 8, 5), 24)])
    w = {k: v.double() for k, v in ref.random_model(cfg, 2).items()}
    ids = tokens(cfg, 30, 3)
    other = list(ids)
    other[10] = (other[10] + 1) % 30
    a, b = ref.forward(cfg, w, ids), ref.forward(cfg, w, other)
    changed = ((a - b).abs().amax(-1) > 1e-12).nonzero().flatten().tolist()
    # token 10 reaches the latents of 10..12 (taps) and those the queries up to 16 (window of 5)
    assert changed == list(range(10, 17))


def test_planted_mistakes_are_visible():
    """Each mechanism matters at the tolerance the comparison with the product uses."""
    from delunex_cases import TOL, error

    cfg = CASES["odd"]
    w = {k: v.double() for k, v in ref.random_model(cfg, 4).items()}
    ids = tokens(cfg, 60, 5)
    base = ref.forward(cfg, w, ids)

    def changed(edit_cfg=None, edit_w=None):
        c, v = copy.deepcopy(cfg), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(v)
        return error(ref.forward(c, v, ids), base)

    floor = 2 * TOL[torch.float32]
    assert changed(lambda c: c["layers"][0]["mixer"]["mask"].update(size=10)) > floor
    assert changed(lambda c: c["layers"][3]["mixer"]["mask"].update(size=2)) > floor
    assert changed(lambda c: c["layers"][2]["mixer"].update(scale=0.2)) > floor
    assert changed(lambda c: c["norm"].update(eps=1e-6)) > floor
    for name in ("l0.canon1", "l2.mix.g", "l1.mix.dkv.norm", "l0.norm2", "l3.mlp.act"):
        assert changed(edit_w=lambda v, n=name: v.update({n: v[n] * 1.1})) > floor
    assert changed(edit_w=lambda v: v.update({"l3.dwa": torch.cat([v["l3.dwa"][:1] * 1.1, v["l3.dwa"][1:]])})) > floor


def test_models_refuse_the_host():
    from diff_gpt_b200 import Engine

    m, _ = build(CASES["tiny"], 0, torch.float32, "cpu")
    with pytest.raises(RuntimeError, match="CUDA only"):
        m(torch.zeros(1, 3, dtype=torch.long))
    with pytest.raises(RuntimeError, match="CUDA only"):
        Engine(m).generate_batch([1, 2], num_samples=1, max_tokens=2)
