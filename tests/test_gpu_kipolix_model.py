"""Kipolix models on the GPU against the plain implementation: prompts, portions, decoding, batches, the Engine, the
command line."""

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

from kipolix_cases import CASES, TOL, attention, build, config, error, retention, tokens
from oracle import ref_kipolix as ref

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def run_portions(model, ids, cuts, cache=None):
    """Logits at every token of one request, its tokens handed over in portions."""
    cache = model.new_cache() if cache is None else cache
    cache.reset()
    out, at = [], 0
    for n in cuts:
        part = torch.tensor([ids[at : at + n]], device="cuda")
        out.append(model.logits_at(part, cache, torch.arange(n, device="cuda")).float().cpu().clone())
        at += n
    assert at == len(ids) and cache.get_pos() == at
    return torch.cat(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_layers_prompts_portions_and_decoding(name, dtype):
    cfg = CASES[name]
    model, w = build(cfg, 7, dtype)
    ids = tokens(cfg, 230, 8)
    want, layers = ref.forward(cfg, w, ids, keep_layers=True)
    # the sum of the streams after every layer run
    got = {}
    with torch.inference_mode():
        model._step(torch.tensor([ids], device="cuda"), model.new_cache(), None, lambda i, x: got.update({i: x.clone()}))
    assert sorted(got) == list(range(len(layers)))
    for i in got:
        assert error(got[i], layers[i]) <= TOL[dtype], i
    # the whole prompt, one by one, and portions around the sizes where the kernels change (16, 32, 64, a multiple of a tile)
    cache = model.new_cache()
    for cuts in ([230], [1] * 230, [2] * 115, [15, 16, 17, 31, 32, 33, 64, 22], [100] + [1] * 30 + [3, 60, 7, 30], [1, 229], [128, 102]):
        assert error(run_portions(model, ids, cuts, cache), want) <= TOL[dtype], cuts[:4]
    # logits in the model's dtype through the module's own call
    full, loss = model(torch.tensor([ids[:40]], device="cuda"), targets=torch.tensor([ids[1:41]], device="cuda"))
    assert full.dtype == dtype and error(full[0], want[:40]) <= TOL[dtype] and torch.isfinite(loss)


@pytest.mark.parametrize("dtype", DTYPES)
def test_how_a_prompt_is_cut_changes_only_rounding(dtype):
    cfg = CASES["wide"]
    model, _ = build(cfg, 3, dtype)
    ids = tokens(cfg, 150, 4)
    base = run_portions(model, ids, [150])
    for cuts in ([1] * 150, [70, 80], [2, 3, 40, 105]):
        assert error(run_portions(model, ids, cuts), base.double()) <= TOL[dtype]


@pytest.mark.parametrize("window,keep", [(5, 2), (64, 1), (65, 70), (128, 6), (129, 0), (200, 33)])
def test_window_and_kept_token_edges_show(window, keep):
    """With sharp attention a window, or a number of kept tokens, of one more or less moves some logits by far more than the
    tolerance (checked on the plain implementation), and the product sides with the right one, in a prompt and in decoding."""
    layer = attention(4, 2, 32, 32, window, keep, scale=0.6, rot=16)
    cfg = config(64, 50, [(layer, 96), (layer, 96)], streams=2)
    model, w = build(cfg, window, torch.float32)
    ids = tokens(cfg, window + keep + 90, 9)
    want = ref.forward(cfg, w, ids)
    for change in ({"size": window - 1}, {"size": window + 1}, {"keep_first": keep + 1}) + (({"keep_first": keep - 1},) if keep else ()):
        wrong = copy.deepcopy(cfg)
        for l in wrong["layers"]:
            l["mixer"]["mask"].update(change)
        assert error(ref.forward(wrong, w, ids), want) > 20 * TOL[torch.float32], change
    n = len(ids)
    for cuts in ([n], [window + 10] + [1] * (n - window - 10), [window - 1] + [1] * 4 + [40, n - window - 43], [keep + 1, 2, n - keep - 3]):
        assert error(run_portions(model, ids, cuts), want) <= TOL[torch.float32]
    bf, _ = build(cfg, window, torch.bfloat16)
    assert torch.isfinite(run_portions(bf, ids, [n])).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_tokens(dtype):
    """One token changed among hundreds: through the retained state, a kept first token and the window's chain the later
    logits change as the plain implementation's do, and the bigram carries it one token on."""
    cfg = config(64, 40, [(retention(2, 32, 32, (0.995, 0.9)), 48), (attention(2, 1, 32, 32, 24, 3), 48)], streams=2, loop=(0, 2, 2))
    model, w = build(cfg, 5, dtype)
    ids = tokens(cfg, 420, 6)
    base = ref.forward(cfg, w, ids)
    for at in (0, 2, 3, 57):
        other = list(ids)
        other[at] = (other[at] + 7) % 40
        want = ref.forward(cfg, w, other)
        effect = error(want, base)
        assert effect > 3 * TOL[dtype]
        for cuts in ([420], [at + 1] + [1] * 60 + [359 - at]):
            got = run_portions(model, other, cuts)
            assert error(got, want) <= min(TOL[dtype], effect / 3)
            if dtype == torch.float32:  # the difference itself, far behind the token
                d = (got - run_portions(model, ids, cuts)).double()[at + 150 :]
                e = (want - base)[at + 150 :]
                assert e.abs().max() > 1e-3 and (d - e).abs().max() <= 2e-2 * e.abs().max()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_slides_the_cache(dtype):
    """Thousands of tokens through a cache of a few windows, mostly one by one: the rows slide behind the kept ones, the
    states run on, positions pass the tables' first size."""
    cfg = config(32, 40, [(attention(2, 1, 16, 16, 20, 4), 48), (retention(2, 16, 16, (0.9, 0.98)), None), (attention(2, 2, 16, 16, 30, 9), 48)],
                 streams=2)
    model, w = build(cfg, 5, dtype)
    ids = tokens(cfg, 2600, 6)
    cache = model.new_cache()
    got = run_portions(model, ids, [700] + [1] * 900 + [500] + [1] * 500, cache)
    assert cache.base > 0 and cache.capacity < 2600 and cache.slot < 2600
    want = ref.forward(cfg, w, ids)
    for end in (700, 1100, 1599, 1601, 2101, 2600):
        assert error(got[end - 20 : end], want[end - 20 : end]) <= TOL[dtype], end
    assert error(got, want) <= 2 * TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_step_runner_gives_caches_back_and_takes_them_again(dtype):
    """Unequal requests one after the other and interleaved; what an earlier request left in a cache must not show."""
    from diff_gpt_b200 import StepRunner

    cfg = CASES["odd"]
    model, w = build(cfg, 2, dtype)
    runner = StepRunner(model)
    reqs = {f"r{k}": tokens(cfg, n, 20 + k) for k, n in enumerate((90, 3, 1, 55, 140))}
    want = {k: ref.forward(cfg, w, v) for k, v in reqs.items()}
    for k, ids in reqs.items():  # one after the other: every request takes over the cache before it
        got = [runner.step(k, ids[:50], list(range(len(ids[:50]))))]
        for t in ids[50:]:
            got.append(runner.step(k, [t], [0]))
        assert error(torch.cat(got), want[k]) <= TOL[dtype]
        runner.finish(k)
    assert len(runner._free) == 1 and not runner._live
    got = {k: [] for k in reqs}
    at = {k: 0 for k in reqs}
    turn = 0
    while any(at[k] < len(v) for k, v in reqs.items()):
        for k, ids in reqs.items():
            n = min((1, 2, 37, 5)[turn % 4], len(ids) - at[k])
            turn += 1
            if n > 0:
                got[k].append(runner.step(k, ids[at[k] : at[k] + n], list(range(n))))
                at[k] += n
    for k in reqs:
        assert error(torch.cat(got[k]), want[k]) <= TOL[dtype]
    # places asked for in any order, or none
    runner.finish("r0")
    assert runner.step("x", reqs["r0"][:7], []).shape == (0, cfg["vocab"])
    picked = runner.step("x", reqs["r0"][7:12], [4, 0])
    assert error(picked, want["r0"][[11, 7]]) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_forward_equals_each_alone(dtype):
    cfg = CASES["wide"]
    model, w = build(cfg, 2, dtype)
    rows = [tokens(cfg, 120, 30 + b) for b in range(3)]
    cache = model.new_cache(3)
    idx = torch.tensor(rows, device="cuda")
    got = torch.cat([model(idx[:, a:b], kv_cache=cache)[0] for a, b in ((0, 50), (50, 51), (51, 53), (53, 100), (100, 120))], dim=1)
    for b in range(3):
        assert error(got[b], ref.forward(cfg, w, rows[b])) <= TOL[dtype]


# ---- the Engine -------------------------------------------------------------------------
def plain_greedy(cfg, w, prompt, G):
    """Greedy continuation and, per step, how far the best logit leads (a lead below rounding decides nothing)."""
    ids, lead = list(prompt), []
    for _ in range(G):
        z = ref.forward(cfg, w, ids)[-1]
        top = z.topk(2).values
        lead.append(((top[0] - top[1]) / z.std()).item())
        ids.append(int(z.argmax()))
    return ids[len(prompt) :], lead


ENGINE_CFG = config(48, 64, [
    (attention(4, 2, 16, 24, 11, 12), 64), (retention(2, 24, 16, (0.9, 0.97)), 64), (attention(3, 1, 32, 32, 7, 0), None),
], streams=3, loop=(0, 2, 2))


def same_stream(got, want, lead):
    """Equal token by token, up to a place where rounding may decide (the streams part there)."""
    at = next((i for i, (a, b) in enumerate(zip(got, want)) if a != b), len(want))
    return at == len(want) or lead[at] < 1e-3


@pytest.mark.parametrize("N,use_graph", [(1, True), (1, False), (17, True)])
def test_engine_greedy_generation(N, use_graph):
    """`generate_many` over prompts of unequal length (one of a single token, two shorter than the kept tokens), far past
    the ring of own pages."""
    from diff_gpt_b200 import Engine, TemperatureSampler

    model, w = build(ENGINE_CFG, 8, torch.float32)
    lens, G = (1, 9, 40, 9), 60
    prompts = [tokens(ENGINE_CFG, n, 40 + n + i // 3) for i, n in enumerate(lens)]
    eng = Engine(model)
    kw = dict(num_samples=N, max_tokens=G, sampler=TemperatureSampler(0.0), page_tokens=4, use_graph=use_graph)
    got, masks = eng.generate_many(prompts, **kw)
    assert got.shape == (4, N, G) and bool((masks == 1).all())
    run = eng._run
    assert run.cache.ring_pages < run.cache.own_pages and (run.graph is not None) == use_graph
    for s, p in enumerate(prompts):
        want, lead = plain_greedy(ENGINE_CFG, w, p, G)
        for n in range(N):
            assert same_stream(got[s, n].tolist(), want, lead), (s, n)
        first = next((i for i, x in enumerate(lead) if x < 1e-3), G)
        assert first > 20 and len(set(want)) > 5
    # the same run reused with other prompts of the same lengths: pages, states and the captured step are used again
    again = [tokens(ENGINE_CFG, n, 80 + 3 * n + i) for i, n in enumerate(lens)]
    got2, _ = eng.generate_many(again, **kw)
    assert eng._run is run
    for s, p in enumerate(again):
        want, lead = plain_greedy(ENGINE_CFG, w, p, G)
        assert same_stream(got2[s, 0].tolist(), want, lead), s
    alone, _ = eng.generate_many([prompts[2]], **kw)
    assert torch.equal(alone[0], got[2])


def test_engine_streaming_forcing_and_samplers():
    from diff_gpt_b200 import Engine, NucleusSampler, TemperatureSampler

    model, w = build(ENGINE_CFG, 8, torch.float32)
    eng = Engine(model)
    prompt = tokens(ENGINE_CFG, 12, 1)
    sched = [None if g % 3 else (5 * g) % 64 for g in range(20)]
    res, masks = eng.generate_batch(prompt, num_samples=2, max_tokens=20, sampler=TemperatureSampler(0.0), force_schedule=sched)
    assert masks[0] == [0] * 12 + [0 if s is not None else 1 for s in sched]
    ids = list(prompt)
    for g, s in enumerate(sched):
        want = s if s is not None else int(ref.forward(ENGINE_CFG, w, ids)[-1].argmax())
        assert res[0][12 + g] == res[1][12 + g] == want
        ids.append(want)
    stream = [c for c, _ in eng.generate(prompt, num_samples=2, max_tokens=20, sampler=TemperatureSampler(0.0), force_schedule=sched)]
    assert [c[0] for c in stream] == res[0][12:]
    # sampled streams are functions of (seed, trajectory): batch size does not change them
    for sampler in (TemperatureSampler(1.0), NucleusSampler(0.8, TemperatureSampler(0.7))):
        a, _ = eng.generate_many([prompt], 6, 15, sampler, seed=7)
        b, _ = eng.generate_many([prompt], 2, 15, sampler, seed=7, traj_offset=4)
        assert torch.equal(a[0, 4:], b[0]) and len({tuple(r) for r in a[0].tolist()}) > 1
    # a sampler that is only a Python callable sees the device logits
    c, _ = eng.generate_many([prompt], 1, 15, lambda z, rng=None: z.argmax(-1, keepdim=True))
    d, _ = eng.generate_many([prompt], 1, 15, TemperatureSampler(0.0))
    assert torch.equal(c, d)
    out = model.generate(torch.tensor([prompt], device="cuda"), 15, TemperatureSampler(0.0))
    assert out[0, 12:].tolist() == d[0, 0].tolist()


def test_engine_bf16_decode_logits_and_fused_head():
    """bf16: per-step logits of a forced decode against the plain implementation (a prompt long enough for the tensor-core
    kernels and their segments, 40 trajectories, a head of its own), and the draw in the head's epilogue."""
    from diff_gpt_b200 import TemperatureSampler
    from diff_gpt_b200.model.engine import DecodeRun

    cfg = config(128, 96, [
        (retention(2, 64, 64, (0.97, 0.998)), 256), (attention(8, 2, 32, 32, 50, 5), 256), (attention(4, 1, 64, 64, 300, 20), 192),
    ], streams=4, loop=(1, 2, 2))
    model, w = build(cfg, 6, torch.bfloat16)
    prompt, stream = tokens(cfg, 1100, 2), tokens(cfg, 40, 3)
    want = ref.forward(cfg, w, prompt + stream)[1099:]
    run = DecodeRun(model, [prompt], 40, 40, TemperatureSampler(0.0), 42, [stream], fused_head=False, page_tokens=16)
    run.start()
    assert error(run.logits0, want[:1]) <= TOL[torch.bfloat16]
    for g in range(1, 40):
        run.advance(1)
        assert error(run.logits, want[g : g + 1].expand(40, -1)) <= TOL[torch.bfloat16], g
    run.check_status()
    free = DecodeRun(model, [prompt], 300, 30, TemperatureSampler(0.0), 42, None)
    assert free.lmhead and free.head_ws is not None and free.plan.fused_ff
    free.start()
    free.advance(30)
    free.check_status()
    rows = free.history.cpu()
    assert bool((rows == rows[:1]).all())
    z = ref.forward(cfg, w, prompt + rows[0].tolist())[1099:-1]
    chosen = z.gather(1, rows[0][:, None].long())[:, 0]
    assert bool((chosen >= z.max(-1).values - 0.2 * z.std()).all())  # the arg-max up to rounding


def test_forecasting_facade_over_a_kipolix_model():
    import numpy as np
    import pandas as pd

    from diff_gpt_b200 import TemperatureSampler
    from diff_gpt_b200.diff_gpt import DiffGPT
    from diff_gpt_b200.encoder_decoder import get_domain_of_definition

    model, _ = build(ENGINE_CFG, 8, torch.float32)
    df = pd.DataFrame({"a": np.cumsum(np.random.default_rng(0).normal(size=50))})
    f = DiffGPT(model, 1, get_domain_of_definition(df.to_numpy(), 1, use_decimal=False), False)
    a = f.predict_samples(df, 8, 3, TemperatureSampler(0.0))
    assert a.shape == (3, 8, 1) and np.isfinite(a).all() and (a[0] == a[1]).all()
    scores = f.anomaly_scores(df)
    assert np.isfinite(scores.to_numpy()[2:]).all()


# ---- the command line ---------------------------------------------------------------------
def test_command_line_generates_and_replays_a_trace(tmp_path):
    from diff_gpt_b200.weights import write_safetensors

    cfg = CASES["odd"]
    w = ref.random_model(cfg, 9)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()})
    w = {k: v.double() for k, v in w.items()}
    a, b = tokens(cfg, 45, 1), tokens(cfg, 12, 2)
    lines = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [3, 39]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[40:41], "want": [0]}], "end": []},
        {"step": 3, "entries": [{"id": "a", "tokens": a[41:], "want": [3]}, {"id": "b", "tokens": b, "want": [11, 0]}], "end": ["a", "b"]},
    ]
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run(
        [os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
        input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True, text=True, timeout=300,
    )
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {k}" for k in range(4)]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
    za, zb = ref.forward(cfg, w, a), ref.forward(cfg, w, b)
    for name, want in (("0", za[[3, 39]]), ("2", za[[40]]), ("3", torch.cat([za[[44]], zb[[11, 0]]]))):
        got = torch.frombuffer(bytearray((out / f"{name}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert error(got, want) <= TOL[torch.float32]
    p = subprocess.run(
        [sys.executable, "-m", "diff_gpt_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--tokens",
         ",".join(map(str, b)), "--max-tokens", "6"],
        cwd=ROOT, capture_output=True, text=True, timeout=300,
    )
    assert p.returncode == 0, p.stderr[-2000:]
    want, lead = plain_greedy(cfg, w, b, 6)
    assert same_stream([int(t) for t in p.stdout.split()], want, lead)
