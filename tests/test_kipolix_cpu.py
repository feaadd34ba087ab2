"""Kipolix on the host: configuration, checkpoint folders, caches' bookkeeping, the plain implementation itself."""

import copy
import json
import math

import pytest
import torch

from kipolix_cases import CASES, TOL, attention, build, config, error, retention, tokens
from oracle import ref_kipolix as ref


def test_configuration_is_read_and_refused():
    from diff_gpt_b200.model.kipolix import Attention, KipolixConfig, Retention

    cfg = KipolixConfig.from_dict(CASES["odd"])
    assert [type(l.mixer) for l in cfg.layers] == [Attention, Retention, Attention, Retention, Attention]
    assert [l.ff for l in cfg.layers] == [70, None, 44, 90, None] and cfg.streams == 5 and cfg.eps == 3e-3
    assert cfg.runs == (0, 1, 0, 1, 0, 1, 2, 3, 4) == tuple(ref.runs(CASES["odd"]))
    assert [KipolixConfig.from_dict(CASES[n]).runs for n in ("wide", "tiny")] == [(0, 1, 2, 1, 2, 3, 4), (0,)]
    m = cfg.layers[0].mixer
    assert (m.window, m.keep_first, m.rot.dims, m.rot.base, m.scale, m.head) == (9, 3, 6, 500.0, 0.31, 32)
    assert cfg.layers[1].mixer.decay == (0.9, 0.99, 0.3)
    assert (cfg.buckets, cfg.mul_prev, cfg.mul_cur) == (61, 31, 5)

    def broken(change):
        c = copy.deepcopy(CASES["odd"])
        change(c)
        with pytest.raises((ValueError, KeyError)):
            KipolixConfig.from_dict(c)

    broken(lambda c: c["layers"][0].update(type="something else"))
    broken(lambda c: c["layers"][0]["mixer"].update(bias=True))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].update(chunk=4))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda c: c["layers"][0]["mixer"]["mask"].pop("keep_first"))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=4))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(stretch=2))
    broken(lambda c: c["layers"][1]["mixer"].update(decay=[0.9, 0.99]))
    broken(lambda c: c["layers"][1]["mixer"].update(decay=[0.9, 0.99, 1.5]))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda c: c["loop"].update(stop=6))
    broken(lambda c: c["loop"].update(times=0))
    broken(lambda c: c.update(layers=[]))
    broken(lambda c: c.update(streams=0))
    broken(lambda c: c["embedding"].update(scale=2.0))
    broken(lambda c: c["embedding"]["bigram"].pop("mul_cur"))


def test_checkpoint_folder_round_trip(tmp_path):
    from diff_gpt_b200 import Kipolix, load_model
    from diff_gpt_b200.weights import write_safetensors

    cfg = CASES["odd"]
    w = {k: v.to(torch.bfloat16) for k, v in ref.random_model(cfg, 1).items()}
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    for dtype in (torch.float32, torch.bfloat16):
        m = load_model(str(tmp_path), dtype, "cpu")
        assert isinstance(m, Kipolix) and m.embedding.dtype == dtype
        assert all(torch.equal(m.tensor(k).to(torch.bfloat16), w[k]) for k in w)
    for change in ({"l1.norm2": torch.zeros(52)}, {"l0.hc2.in": None}, {"head": torch.zeros(76, 52)}):
        t = {**w, **change}
        write_safetensors(str(tmp_path / "model.safetensors"), {k: v for k, v in t.items() if v is not None})
        with pytest.raises(ValueError):
            load_model(str(tmp_path), torch.float32, "cpu")


def test_packed_weights_pad_with_zeros_only():
    """Padded heads, sections and interleaved feed-forward rows must not change any product."""
    m, w = build(CASES["odd"], 3, torch.float32, "cpu")
    h = torch.randn(5, 52, generator=torch.Generator().manual_seed(0))
    W = m.packed_weights()
    p = W.layers[0]  # 6 query and 2 key/value heads, 12 and 20 wide, padded to 32
    x = h @ p.w_in_t
    q, k, v = (x[:, a:b].view(5, -1, 32) for a, b in ((0, 192), (192, 256), (256, 320)))
    assert p.cols == (0, 192, 256)
    for t, name, n in ((q, "q", 12), (k, "k", 12), (v, "v", 20)):
        assert torch.allclose(t[..., :n].flatten(1), h @ w[f"l0.mix.{name}"].float().T, atol=1e-5) and bool((t[..., n:] == 0).all())
    assert torch.equal(p.q_norm.view(6, 32)[:, :12].flatten(), w["l0.mix.q.norm"].float()) and bool((p.q_norm.view(6, 32)[:, 12:] == 0).all())
    o = torch.randn(5, 6, 32)
    assert torch.allclose(o.flatten(1) @ p.w_o_t, o[..., :20].flatten(1) @ w["l0.mix.o"].float().T, atol=1e-4)
    gu = h @ p.w_gu.T
    assert torch.allclose(gu[:, 0::2], h @ w["l0.mlp.gate"].float().T, atol=1e-5) and torch.allclose(gu[:, 1::2], h @ w["l0.mlp.up"].float().T, atol=1e-5)
    assert torch.equal(p.sub1.norm, 1 + w["l0.norm1"].float())
    r = W.layers[1]  # retention, 3 heads of 20 and 12: sections of 60, 60, 36, 36 columns start at multiples of 8
    x = h @ r.w_in_t
    assert r.cols == (0, 64, 128, 168)
    for at, name, n in zip(r.cols, "qkvg", (60, 60, 36, 36)):
        assert torch.allclose(x[:, at : at + n], h @ w[f"l1.mix.{name}"].float().T, atol=1e-5)
    assert r.sub2 is None and r.w_gu is None
    assert W.head is not None and torch.equal(W.head.float(), w["head"].float())
    assert m.packed_weights() is W
    m.tensor("l0.hc1.out").mul_(2.0)
    assert torch.equal(m.packed_weights().layers[0].sub1.out, 2 * w["l0.hc1.out"].float())


def test_every_layer_run_has_rows_or_a_state_of_its_own():
    m, _ = build(CASES["odd"], 0, torch.float32, "cpu")
    assert sorted(m.row_widths) == [0, 2, 4, 6, 8] and m.row_widths[0] == 2 * 2 * 32 and m.row_widths[8] == 2 * 64
    assert sorted(m.state_specs) == ["prev", "ret1", "ret3", "ret5", "ret7"]
    assert m.state_specs["ret1"].shape == (3, 20, 12) and m.state_specs["ret7"].shape == (2, 10, 36)
    assert (m.keep, m.keep_first) == (32, 11)
    only_retention = config(16, 20, [(retention(1, 8, 8, (0.9,)), 16)])
    m, _ = build(only_retention, 0, torch.float32, "cpu")
    assert m.row_widths == {} and (m.keep, m.keep_first) == (0, 0)
    c = m.new_cache(2, 5)
    assert c.state.source["prev"].tolist() == [[-1, -1]]
    c.state.target["prev"].fill_(4)
    c.state.flip()
    c.state.source["ret0"].fill_(1.0)
    c.reset()
    assert c.state.current == 0 and all(int(b["prev"].max()) == -1 and bool((b["ret0"] == 0).all()) for b in c.state.buffers)


def test_rotation_tables_grow_and_stay_exact():
    from diff_gpt_b200.model.rope import rotation_table

    m, _ = build(CASES["odd"], 0, torch.float32, "cpu")
    a = m.tables(10)
    assert set(a) == {(500.0, 6), (10000.0, 14), (10000.0, 8), (10000.0, 10), (10000.0, 36)} and all(t.shape[0] == 1024 for t in a.values())
    assert m.tables(1024)[500.0, 6] is a[500.0, 6]
    b = m.tables(5000)
    assert b[500.0, 6].shape == (8192, 3, 2) and torch.equal(b[500.0, 6][:1024], a[500.0, 6]) and a[500.0, 6].shape[0] == 1024
    t = rotation_table(1e4, 64, 40000, "cpu")
    p, i = 39999, 3
    x = p * 1e4 ** (-2 * i / 64)
    assert t[p, i].tolist() == pytest.approx([math.cos(x), math.sin(x)], abs=6e-8)


@pytest.mark.parametrize("keep,keep_first", [(37, 0), (37, 5), (10, 200), (0, 1), (64, 64)])
def test_row_cache_slides_behind_the_kept_tokens(keep, keep_first):
    """Rows are tagged with their position; whatever the portions, the first `keep_first` and the last `keep` tokens before
    each new one are in place, and what is dropped lies farther than `keep` slots back."""
    from diff_gpt_b200.model.kv_cache import RowCache, StateSpec

    cache = RowCache(2, {0: 8, 3: 16}, keep, {"s": StateSpec(1, (3,))}, torch.float32, "cpu", keep_first)
    g = torch.Generator().manual_seed(5)
    moved = 0
    for _ in range(3):
        cache.reset()
        assert cache.get_pos() == 0 and cache.slot == 0
        while cache.pos < 5000:
            T = int(torch.randint(1, 3, (1,), generator=g)) if cache.pos % 5 else int(torch.randint(1, 400, (1,), generator=g))
            cache.ensure(T)
            slot = cache.slot
            moved += cache.base > 0
            for key in (0, 3):
                t = cache.store[key]
                assert slot + T <= t.shape[1] == cache.capacity
                first = min(cache.pos, keep_first)
                assert torch.equal(t[:, :first, 0], torch.arange(first, dtype=torch.float32).expand(2, -1))
                last = min(cache.pos - first, keep)
                seen = cache.span(key, slot - last, slot).view(2, last, cache.widths[key])
                assert torch.equal(seen[:, :, 0], torch.arange(cache.pos - last, cache.pos, dtype=torch.float32).expand(2, -1))
                # behind the kept tokens slots are as far apart as positions; a kept token that looks nearer than it is
                # must still look farther than any window reaches
                assert torch.equal(slot - torch.arange(first, slot), cache.pos - t[0, first:slot, 0].long())
                if cache.base and first:
                    assert slot - (first - 1) > keep
                t[:, slot : slot + T] = torch.arange(cache.pos, cache.pos + T, dtype=torch.float32)[None, :, None]
            cache.pos += T
    assert moved and cache.capacity < 3000


@pytest.mark.parametrize("keep,first,pt,G,P", [(0, 3, 4, 30, 1), (5, 6, 4, 40, 2), (63, 100, 64, 400, 30), (20, 1, 16, 90, 5), (3, 9, 4, 30, 9), (7, 50, 8, 60, 1)])
def test_ring_of_own_pages_never_overwrites_a_kept_token(keep, first, pt, G, P):
    """Prompts shorter than the number of kept tokens: the generated ones among the kept must survive the ring."""
    from diff_gpt_b200.model.kv_cache import PagedRowCache

    c = PagedRowCache({1: 8}, keep, {}, n_series=2, rows_per_series=2, prefix_len=P, max_new=G, dtype=torch.float32, device="cpu",
                      page_tokens=pt, keep_first=first)
    store = {}

    def place(row, g):
        slot = c.suffix_slot0 + g
        return int(c.row_table[row, slot // pt]), slot % pt

    for prompt in (1, P):  # every prompt of a run may be shorter than the longest
        for g in range(G):
            for row in range(4):
                store[place(row, g)] = (row, g)
            for row in range(4):
                seen = set(range(max(0, g - keep), g + 1)) | {k for k in range(g + 1) if prompt + k < first}
                assert all(store[place(row, k)] == (row, k) for k in seen)
    n_prefix = 2 * (c.suffix_slot0 // pt)
    assert int(c.row_table[:, c.suffix_slot0 // pt :].min()) >= n_prefix and int(c.row_table.max()) < c.pools[1].shape[0]
    assert c.ring_pages <= -(-keep // pt) + 1 + -(-first // pt)


def test_rows_start_from_their_prompts_state():
    from diff_gpt_b200.model.kv_cache import PagedRowCache, StateSpec

    specs = {"prev": StateSpec(1, (), torch.int32, -1), "ret2": StateSpec(1, (2, 3, 4))}
    c = PagedRowCache({0: 8}, 3, specs, n_series=3, rows_per_series=2, prefix_len=5, max_new=4, dtype=torch.float32, device="cpu")
    a, b = c.prompt_states([0, 2]), c.prompt_states([1])
    assert a["prev"].tolist() == [[-1, -1]] and a["ret2"].shape == (1, 2, 2, 3, 4)
    a["prev"][0] = torch.tensor([7, 9])
    a["ret2"][:, 0], a["ret2"][:, 1], b["ret2"][:, 0] = 1.0, 3.0, 2.0
    c.prompts_ready()
    assert c.states["prev"].tolist() == [[7, 7, -1, -1, 9, 9]] and c.states["ret2"][0, :, 1, 2, 3].tolist() == [1, 1, 2, 2, 3, 3]
    c.begin_prompts()
    assert a["prev"].tolist() == [[-1, -1]] and bool((a["ret2"] == 0).all()) and bool((b["ret2"] == 0).all())


# ---- the plain implementation: facts that do not depend on the product ------------------------
def test_plain_mechanisms_by_hand():
    assert ref.visible(5, 2, 1).tolist() == [
        [True, False, False, False, False], [True, True, False, False, False], [True, True, True, False, False],
        [True, False, True, True, False], [True, False, False, True, True],
    ]
    assert ref.bigram_rows(torch.tensor([4, 0, 3]), 11, 5, 2).tolist() == [11, (4 * 5) % 11, (0 + 6) % 11]
    x = torch.arange(1.0, 7.0).view(1, 1, 6).double()
    c, s = math.cos(3.0), math.sin(3.0)
    c2, s2 = math.cos(3.0 * 100.0**-0.5), math.sin(3.0 * 100.0**-0.5)
    assert ref.rotate_half(x, 4, 100.0, 3)[0, 0].tolist() == pytest.approx(
        [c - 3 * s, 2 * c2 - 4 * s2, 3 * c + s, 4 * c2 + 2 * s2, 5, 6])
    assert ref.rotate_pairs(x, 4, 100.0, 3)[0, 0].tolist() == pytest.approx(
        [c - 2 * s, 2 * c + s, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 5, 6])
    q = torch.tensor([1.0, 2.0, -1.0]).view(3, 1, 1).double()
    k = torch.tensor([3.0, 1.0, 2.0]).view(3, 1, 1).double()
    v = torch.tensor([1.0, 5.0, 7.0]).view(3, 1, 1).double()
    o, S = ref.retention(q, k, v, [0.5])
    assert o.flatten().tolist() == [3.0, 2 * 6.5, -17.25] and S.item() == 17.25
    x = torch.tensor([[[1.0]], [[10.0]]]).double()
    mix, out = torch.tensor([[0.5, 2.0], [3.0, 0.25]]).double(), torch.tensor([1.0, -1.0]).double()
    assert ref.stream_out(x, mix, out, torch.tensor([[100.0]]).double()).flatten().tolist() == [0.5 + 30 + 100, 2 + 2.5 - 100]


def test_plain_forward_reaches_back_as_far_as_the_layers_allow():
    """One attention layer: a token reaches the queries of its window, the kept ones every later query, and each the bigram
    of the next token."""
    cfg = config(20, 30, [(attention(2, 1, 6, 6, 5, 2), 24)])
    w = {k: v.double() for k, v in ref.random_model(cfg, 2).items()}
    ids = tokens(cfg, 30, 3)

    def changed(at):
        other = list(ids)
        other[at] = (other[at] + 1) % 30
        d = (ref.forward(cfg, w, ids) - ref.forward(cfg, w, other)).abs().amax(-1)
        return (d > 1e-12).nonzero().flatten().tolist()

    assert changed(10) == list(range(10, 16))  # itself and the next token's bigram, five queries each
    assert changed(1) == list(range(1, 30)) and changed(0) == list(range(30))
    assert changed(2) == list(range(2, 8))


def test_planted_mistakes_are_visible():
    """Each mechanism matters at the tolerance the comparison with the product uses."""
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
    assert changed(lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=4)) > floor
    assert changed(lambda c: c["layers"][4]["mixer"]["mask"].update(keep_first=10)) > floor
    assert changed(lambda c: c["layers"][2]["mixer"].update(scale=0.2)) > floor
    assert changed(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10)) > floor
    assert changed(lambda c: c["layers"][1]["mixer"]["rot"].update(base=5000.0)) > floor
    assert changed(lambda c: c["layers"][3]["mixer"].update(decay=[0.951, 1.0])) > floor
    assert changed(lambda c: c["loop"].update(times=2)) > floor
    assert changed(lambda c: c["norm"].update(eps=1e-6)) > floor
    assert changed(lambda c: c["embedding"]["bigram"].update(mul_prev=30)) > floor
    for name in ("l0.hc1.in", "l1.hc1.out", "l4.hc1.mix", "l0.mix.q.norm", "l2.mix.k.norm", "l1.mix.g", "l0.norm2", "l3.mlp.up", "final.norm"):
        assert changed(edit_w=lambda v, n=name: v.update({n: v[n] * 1.1})) > floor, name
    assert changed(edit_w=lambda v: v.update({"l0.hc2.mix": v["l0.hc2.mix"].T.contiguous()})) > floor
    assert changed(edit_w=lambda v: v.update(bigram=torch.cat([v["bigram"][:-1], v["bigram"][:1]]))) > floor  # the first token's row


def test_models_refuse_the_host():
    from diff_gpt_b200 import Engine

    m, _ = build(CASES["tiny"], 0, torch.float32, "cpu")
    with pytest.raises(RuntimeError, match="CUDA only"):
        m(torch.zeros(1, 3, dtype=torch.long))
    with pytest.raises(RuntimeError, match="CUDA only"):
        Engine(m).generate_batch([1, 2], num_samples=1, max_tokens=2)
