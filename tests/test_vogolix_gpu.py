"""Vogolix through the engine against the plain implementation (tests/plain_vogolix.py): whole prompts, prefill
against token-by-token decoding, portions down to two tokens, unequal requests in one batch against each alone
with pages and state slots used again, keys just inside and just outside of chunks and windows in prompts and in
decoding, a far key among hundreds, a sink that takes most of the weight, a token that the state must carry over
hundreds of others, the first tokens of a sequence, long decoding, keys shared under the same chunk and under another,
models of one kind of layer only, sizes that are multiples of neither 8 nor 16, configurations drawn at random, greedy
generation through the scheduler, and the programs."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import vogolix_configs as C
import plain_vogolix as P
from gpu_utils import random_tokens, rel_max
from vogolix_utils import Reference, check, engine_for, make_model, oracle
from test_replay_gpu import mixed_schedule

pytestmark = pytest.mark.gpu

CASES = [("mix", "float32"), ("mix", "bfloat16"), ("spaces", "bfloat16"), ("chunks", "bfloat16"), ("windows", "bfloat16")]


class Models(dict):
    def __missing__(self, key):
        name, dtype = key
        self[key] = make_model(self.tmp, C.ALL[name], seed=3 + list(C.ALL).index(name) + (0 if dtype == "float32" else 10))
        return self[key]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    m = Models()
    m.tmp = tmp_path_factory.mktemp("vogolix")
    return m


@pytest.fixture(scope="module")
def engines(models):
    cache = {}

    def get(name, dtype, **kw):
        key = (name, dtype, tuple(sorted(kw.items())))
        if key not in cache:
            cache[key] = engine_for(models[name, dtype][0], dtype, **kw)
        return cache[key]

    yield get
    cache.clear()


def in_steps(eng, key, toks, sizes):
    """The logits of every token, the sequence cut into steps of the given sizes (the last one takes the rest)."""
    outs, i = [], 0
    for s in list(sizes) + [len(toks)]:
        s = min(s, len(toks) - i)
        if s <= 0:
            break
        outs.append(eng.step_tokens([(key, toks[i:i + s], list(range(s)))]).cpu().numpy())
        i += s
    eng.close_request(key)
    return np.concatenate(outs)


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_then_decoding_then_portions(name, dtype, models, engines):
    eng, (_, w) = engines(name, dtype), models[name, dtype]
    cfg = C.ALL[name]
    toks = random_tokens(cfg["vocab"], 150, 1)
    ref = Reference(cfg, w, toks, dtype)
    check(in_steps(eng, "w", toks, []), cfg, w, toks, dtype, ref=ref)
    # most of it in one step, then token by token
    check(in_steps(eng, "d", toks, [80] + [1] * 70), cfg, w, toks, dtype, ref=ref)
    # everything one token at a time, from the first
    check(in_steps(eng, "e", toks[:60], [1] * 60), cfg, w, toks, dtype, rows=range(60), ref=ref)
    # portions of changing size
    check(in_steps(eng, "p", toks, [17, 5, 2, 31, 2, 1, 33, 2, 16, 3, 7, 2]), cfg, w, toks, dtype, ref=ref)
    eng.runner.cache.check_invariants()


@pytest.mark.parametrize("name,dtype", [("mix", "float32"), ("mix", "bfloat16"), ("spaces", "float32"), ("spaces", "bfloat16")])
def test_long_prompts_in_chunks(name, dtype, models, engines):
    """Prompts long enough that the recurrences are cut into chunks that run side by side, and what they leave."""
    eng, (_, w) = engines(name, dtype), models[name, dtype]
    cfg = C.ALL[name]
    toks = random_tokens(cfg["vocab"], 470, 5)
    ref = Reference(cfg, w, toks, dtype)
    check(in_steps(eng, "w", toks, []), cfg, w, toks, dtype, ref=ref)
    check(in_steps(eng, "p", toks, [300, 2, 1, 1, 100, 26]), cfg, w, toks, dtype, ref=ref)
    check(in_steps(eng, "q", toks, [3, 257, 1]), cfg, w, toks, dtype, ref=ref)


@pytest.mark.parametrize("name,dtype", [("mix", "float32"), ("mix", "bfloat16"), ("chunks", "float32")])
def test_unequal_requests_together_with_pages_and_slots_used_again(name, dtype, models, engines):
    lengths = [129, 70, 40, 97, 33, 150, 64, 5, 2]
    pool = 384
    eng, (_, w) = engines(name, dtype, kv_cache_tokens=pool, max_num_seqs=4), models[name, dtype]
    cfg = C.ALL[name]
    toks = {i: random_tokens(cfg["vocab"], n, 100 + i) for i, n in enumerate(lengths)}
    got = {i: [] for i in toks}
    pages, slots = {}, {}
    reused = set()
    for entries, ends in mixed_schedule(lengths, pool, seed=11):
        batch = [(f"r{i}", toks[i][s:s + n], list(range(n))) for i, s, n in entries]
        out = eng.step_tokens(batch).cpu().numpy()
        r = 0
        for i, s, n in entries:
            got[i].append(out[r:r + n])
            r += n
            rc = eng.runner.cache.get(f"r{i}")
            if slots.setdefault(rc.state_slot, i) != i:
                reused.add("slot")
            for p in (p for table in rc.tables for p in table):
                if p and pages.setdefault(p, i) != i:
                    reused.add("page")
        for i in ends:
            eng.close_request(f"r{i}")
        eng.runner.cache.check_invariants()
    assert reused == {"slot", "page"}
    assert eng.runner.cache.num_open() == 0
    for i in toks:
        check(np.concatenate(got[i]), cfg, w, toks[i], dtype)


@pytest.mark.parametrize("name,dtype", [("mix", "float32"), ("mix", "bfloat16")])
def test_long_decoding(name, dtype, models, engines):
    """Single tokens for hundreds of steps: chunks begin and windows move on over decoded tokens, pages go back and are
    handed out again, the states are carried all the way."""
    eng, (_, w) = engines(name, dtype), models[name, dtype]
    cfg = C.ALL[name]
    toks = random_tokens(cfg["vocab"], 420, 9)
    eng.step_tokens([("l", toks[:50], [])])
    outs, rows = [], []
    for i in range(50, len(toks)):
        want = [0] if (i % 37 == 0 or i % 50 in (0, 49) or i % 83 in (0, 82) or i in (127, 128, 129, 256, 384, 419)) else []
        o = eng.step_tokens([("l", toks[i:i + 1], want)])
        if want:
            outs.append(o.cpu().numpy())
            rows.append(i)
    eng.close_request("l")
    check(np.concatenate(outs), cfg, w, toks, dtype, rows=rows)


@pytest.mark.parametrize("name,dtype", CASES)
def test_first_tokens_of_a_sequence(name, dtype, models, engines):
    eng, (_, w) = engines(name, dtype), models[name, dtype]
    toks = random_tokens(C.ALL[name]["vocab"], 6, 4)
    check(in_steps(eng, "f", toks, [1, 1, 1]), C.ALL[name], w, toks, dtype)
    one = eng.step_tokens([("g", toks[:1], [0, 0])]).cpu().numpy()
    eng.close_request("g")
    assert np.array_equal(one[0], one[1])
    check(one[:1], C.ALL[name], w, toks[:1], dtype)
    check(in_steps(eng, "h", toks[:2], [2]), C.ALL[name], w, toks[:2], dtype)
    # a sequence of one token, then another request in the same slot: nothing of the first is left
    check(in_steps(eng, "i", toks[3:5], [1]), C.ALL[name], w, toks[3:5], dtype)


# ---------------------------------------------------------------------------- what a position sees

def standout_model(tmp, cfg, seeds, patch, make_tokens, row, least=0.05):
    """A model and two tokens (A, B) such that in a sequence of A's with one B the logits at ``row`` differ from those
    of A's alone by more than ``least`` of the largest: whether B is seen decides them."""
    V = cfg["vocab"]
    for seed in seeds:
        d, w = make_model(tmp, cfg, seed, patch=patch)
        for A, B in ((seed % V, (seed * 7 + 3) % V), ((seed * 5 + 1) % V, (seed * 11 + 2) % V)):
            if A != B and rel_max(oracle(cfg, w, make_tokens(A, B))[row], oracle(cfg, w, make_tokens(A, A))[row]) > least:
                return d, w, A, B
    raise AssertionError("no seed gave a token that stands out")


def sharper(w):
    """Queries and keys scaled so that single scores stand out."""
    for name in list(w):
        if name.endswith(("mix.uk", "mix.q.norm", "mix.k.norm")):
            w[name] = w[name] * 3.0
        if name.endswith("mix.dkv") or (name.endswith("mix.q") and name[:-1] + "q.norm" not in w):
            w[name] = w[name] * 2.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("at", [0, 1, 15, 16, 17])
def test_a_far_key_among_hundreds(dtype, kind, at, tmp_path):
    """One attention layer that sees everything: one key near the start (around the first page's border) must reach
    queries hundreds of tokens later, in a prompt's tiles and over the partitions of a decoding token's context."""
    n = 500
    if kind == "attention":
        cfg = C.one_layer(kind, C.attention(2, 1, 16, 16, n, rot_dims=4, base=2e5))
    else:
        cfg = C.one_layer(kind, C.latent(2, 16, 8, 16, 32, n, base=2e5))

    def toks_of(A, B):
        t = [A] * n
        t[at] = B
        return t
    d, w, A, B = standout_model(tmp_path, cfg, range(60, 120), sharper, toks_of, n - 1)
    toks = toks_of(A, B)
    ref = Reference(cfg, w, toks, dtype)
    eng = engine_for(d, dtype, max_num_batched_tokens=1024)
    rows = sorted({0, 1, 2, at, at + 1, 127, 128, 129, 255, 256, 498, 499})
    out = eng.step_tokens([("w", toks, rows)]).cpu().numpy()
    eng.close_request("w")
    check(out, cfg, w, toks, dtype, rows=rows, ref=ref)
    outs = [eng.step_tokens([("d", toks[:460], [459])]).cpu().numpy()]
    for i in range(460, n):
        outs.append(eng.step_tokens([("d", toks[i:i + 1], [0])]).cpu().numpy())
    eng.close_request("d")
    check(np.concatenate(outs), cfg, w, toks, dtype, rows=range(459, n), ref=ref)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,size,at", [("attention", 48, 95), ("attention", 48, 96), ("attention", 40, 79), ("attention", 40, 80),
                                          ("attention", 7, 90), ("latent_attention", 48, 95), ("latent_attention", 37, 80),
                                          ("latent_attention", 16, 79)])
def test_a_key_at_the_edge_of_a_chunk_or_window(dtype, kind, size, at, tmp_path):
    """One attention layer over equal tokens but one, whose key stands out: the first and the last token that sees it, and
    their neighbours that do not, in prompts cut before, at and behind those places and token by token."""
    n = at + size + 12
    if kind == "attention":
        cfg = C.one_layer(kind, C.attention(2, 1, 16, 16, size, rot_dims=4, base=2e5))
        first, last = at, (at // size + 1) * size - 1
    else:
        cfg = C.one_layer(kind, C.latent(2, 16, 8, 16, 32, size, base=2e5))
        first, last = at, at + size - 1

    def toks_of(A, B):
        t = [A] * n
        t[at] = B
        return t
    probe = last if last > at else at
    d, w, A, B = standout_model(tmp_path, cfg, range(60, 120), sharper, toks_of, probe)
    toks = toks_of(A, B)
    # the plain implementation itself: what is not seen changes nothing
    plain = [oracle(cfg, w, t) for t in (toks, [A] * n)]
    for i in range(n):
        assert (i < first or i > last) == bool(np.array_equal(plain[0][i], plain[1][i]) or rel_max(plain[0][i], plain[1][i]) < 1e-9), i
    ref = Reference(cfg, w, toks, dtype)
    eng = engine_for(d, dtype)
    check(in_steps(eng, "w", toks, []), cfg, w, toks, dtype, ref=ref)
    for cuts in ([at, 2], [at + 1], [last, 2], [last + 1, 2], [at - 1, 2, 2]):
        check(in_steps(eng, "p", toks, cuts), cfg, w, toks, dtype, ref=ref)
    check(in_steps(eng, "d", toks, [at - 2] + [1] * (n - at + 2)), cfg, w, toks, dtype, ref=ref)
    eng.runner.cache.check_invariants()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sinks_that_take_much_and_nothing(dtype, tmp_path):
    """Sinks so large that a head's keys hardly count, and so small that they do not count themselves; where a chunk
    begins, one key stands against the sink."""
    cfg = C.one_layer("attention", C.attention(4, 2, 16, 16, 20, rot_dims=8))

    def patch(w):
        w["l0.mix.sink"] = torch.tensor([4.0, -40.0, 1.0, 30.0])
    d, w = make_model(tmp_path, cfg, 5, patch=patch)
    toks = random_tokens(cfg["vocab"], 90, 2)
    w0 = dict(w)
    w0["l0.mix.sink"] = torch.full((4,), -100.0)
    assert rel_max(oracle(cfg, w0, toks), oracle(cfg, w, toks)) > 0.02
    ref = Reference(cfg, w, toks, dtype)
    eng = engine_for(d, dtype)
    check(in_steps(eng, "w", toks, []), cfg, w, toks, dtype, ref=ref)
    check(in_steps(eng, "d", toks, [38] + [1] * 52), cfg, w, toks, dtype, ref=ref)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_token_carried_by_the_state(dtype, tmp_path):
    """One state-space layer that hardly forgets: a single other token stays visible hundreds of tokens later, through
    chunks, portions, the cuts between them and decoding; were a state lost or taken from another request, it would
    not be."""
    cfg = C.one_layer("mamba2", C.ssm(4, 16, 32, groups=2, norm_groups=2, conv=4))
    n, at = 420, 37

    def patch(w):
        w["l0.mix.A_log"] = w["l0.mix.A_log"] * 0.1 - 7.0                  # decays next to 1
        w["l0.mix.in"][-4:] *= 3.0                                        # steps that differ from token to token
        w["l0.mix.D"] = w["l0.mix.D"] * 0.1

    def toks_of(A, B):
        t = [A] * n
        t[at] = B
        return t
    d, w, A, B = standout_model(tmp_path, cfg, range(20, 80), patch, toks_of, n - 1, least=5e-3)
    toks = toks_of(A, B)
    ref = Reference(cfg, w, toks, dtype)
    eng = engine_for(d, dtype)
    check(in_steps(eng, "w", toks, []), cfg, w, toks, dtype, ref=ref)
    check(in_steps(eng, "p", toks, [at, 2, 300, 1, 1, 60]), cfg, w, toks, dtype, ref=ref)
    check(in_steps(eng, "q", toks, [at + 1, 64, 17] + [1] * 60), cfg, w, toks, dtype, ref=ref)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_convolutions_last_inputs_are_carried(dtype, tmp_path):
    """One state-space layer of eight taps without memory of its own: a token is seen by the seven behind it through the
    convolution alone, wherever the portions are cut."""
    cfg = C.one_layer("mamba2", C.ssm(2, 16, 16, conv=8))
    n, at = 40, 17

    def patch(w):
        w["l0.mix.A_log"] = w["l0.mix.A_log"] * 0.0 + 5.0                  # everything is forgotten at once
        w["l0.mix.dt_bias"] = w["l0.mix.dt_bias"] * 0.0 + 2.0

    def toks_of(A, B):
        t = [A] * n
        t[at] = B
        return t
    d, w, A, B = standout_model(tmp_path, cfg, range(20, 60), patch, toks_of, at + 7, least=0.02)
    toks = toks_of(A, B)
    assert rel_max(oracle(cfg, w, toks)[at + 8], oracle(cfg, w, [A] * n)[at + 8]) < 1e-6
    ref = Reference(cfg, w, toks, dtype)
    eng = engine_for(d, dtype)
    for cuts in ([], [at], [at + 1, 2, 2], [at + 1] + [1] * 12, [at + 4, 3], [2] * 20, [1] * 40):
        check(in_steps(eng, "c", toks, cuts), cfg, w, toks, dtype, ref=ref)


# ---------------------------------------------------------------------------- other shapes of model

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_are_no_multiples_of_8(dtype, models, engines):
    name = "odd"
    eng, (_, w) = engines(name, dtype), models[name, dtype]
    cfg = C.ALL[name]
    toks = random_tokens(cfg["vocab"], 290, 21)
    ref = Reference(cfg, w, toks, dtype)
    check(in_steps(eng, "o", toks, [40, 2, 17, 1, 1, 29]), cfg, w, toks, dtype, ref=ref)
    check(in_steps(eng, "p", toks, []), cfg, w, toks, dtype, ref=ref)


def test_shared_keys_and_the_stream_after_every_layer(tmp_path):
    """Layers that use an earlier layer's keys and values write none of their own; the residual stream after every
    layer is compared with the plain implementation's."""
    cfg = C.clone(C.CHUNKS)
    d, w = make_model(tmp_path, cfg, 17)
    eng = engine_for(d, "float32")
    assert [g.owners for g in eng.runner.groups] == [[0], [2]]
    toks = random_tokens(cfg["vocab"], 40, 6)
    snaps = []
    for blk in eng.runner.model.blocks:
        def wrapped(residual, pending, ctx, cache, state, _o=blk.forward):
            out = _o(residual, pending, ctx, cache, state)
            snaps.append((residual + (out.float() if out is not None else 0.0)).clone().cpu().double())
            return out
        blk.forward = wrapped
    eng.step_tokens([("a", toks, [])])
    eng.close_request("a")
    for blk in eng.runner.model.blocks:
        del blk.forward
    layers = []
    P.forward(cfg, w, toks, layers)
    assert len(snaps) == len(layers) == 4
    for got, want in zip(snaps, layers):
        assert float((got - want).abs().max() / want.abs().max()) < 1e-5
    check(in_steps(eng, "b", toks, [25] + [1] * 15), cfg, w, toks, "float32")


@pytest.mark.parametrize("first,second", [(12, 50), (50, 12), (33, 33)])
def test_keys_shared_under_another_chunk(first, second, tmp_path):
    """The layer that owns the keys has the shorter chunk, the longer one, or the same as the layer that borrows them; the
    pool is just large enough for the requests, so pages that go back too early would be overwritten."""
    cfg = C.model([("attention", C.attention(2, 1, 16, 16, first, rot_dims=8), None),
                   ("attention", C.attention(4, 1, 16, 16, second, rot_dims=8, kv_from=0), 32)], vocab=64, width=64)
    d, w = make_model(tmp_path, cfg, 9, patch=sharper)
    eng = engine_for(d, "float32", kv_cache_tokens=192, max_seq_len=192)
    seqs = {k: random_tokens(64, 96, 40 + i) for i, k in enumerate("ab")}
    got = {k: [] for k in seqs}
    at = 0
    for n in [1, 2, 9, 1, 1, 17, 2, 1, 30, 1, 1, 30]:
        n = min(n, 96 - at)
        out = eng.step_tokens([(k, t[at:at + n], list(range(n))) for k, t in seqs.items()]).cpu().numpy()
        got["a"].append(out[:n])
        got["b"].append(out[n:])
        at += n
        eng.runner.cache.check_invariants()
    assert at == 96
    for k, t in seqs.items():
        eng.close_request(k)
        check(np.concatenate(got[k]), cfg, w, t, "float32")


@pytest.mark.parametrize("seed", [1, 2, 3, 5, 8, 13])
def test_configurations_drawn_at_random(seed, tmp_path):
    for dtype in ("float32", "bfloat16"):
        cfg = C.random_config(seed)
        toks = random_tokens(cfg["vocab"], 330, seed)
        d, w = make_model(tmp_path, cfg, seed + (0 if dtype == "float32" else 100), sharpen=1.5)
        eng = engine_for(d, dtype)
        ref = Reference(cfg, w, toks, dtype)
        check(in_steps(eng, "p", toks, [130, 2, 1, 70, 1, 1, 1, 3, 121]), cfg, w, toks, dtype, ref=ref)
        check(in_steps(eng, "w", toks, []), cfg, w, toks, dtype, ref=ref)
        del eng


def test_decoding_as_cuda_graphs(models):
    """Single-token steps padded and replayed as CUDA graphs; the states advance once per step."""
    for name in ("mix", "spaces"):
        cfg = C.ALL[name]
        d, w = models[name, "float32"]
        eng = engine_for(d, "float32", cuda_graphs=True)
        toks = random_tokens(cfg["vocab"], 90, 6)
        before = eng.runner.num_graph_steps
        outs = [eng.step_tokens([("d", toks[:50], [49])], graphs=True).cpu().numpy()]
        for i in range(50, len(toks)):
            outs.append(eng.step_tokens([("d", toks[i:i + 1], [0])], graphs=True).cpu().numpy())
        eng.close_request("d")
        assert eng.runner.num_graph_steps - before == 40
        check(np.concatenate(outs), cfg, w, toks, "float32", rows=range(49, len(toks)))


# ---------------------------------------------------------------------------- generation and programs

@pytest.mark.parametrize("name,dtype,opts", [
    ("mix", "float32", dict(async_scheduling=True, cuda_graphs=True, max_num_batched_tokens=48)),
    ("mix", "float32", dict(async_scheduling=False, cuda_graphs=False, max_num_batched_tokens=48)),
    ("chunks", "float32", dict(async_scheduling=True, cuda_graphs=True, max_num_batched_tokens=64)),
    ("mix", "bfloat16", dict(async_scheduling=False, max_num_batched_tokens=32)),
])
def test_greedy_generation_through_the_scheduler(name, dtype, opts, models):
    """The framework's own entry point: requests of unequal length admitted by the scheduler, prompts in portions
    under a small token budget, decoding beside them; every generated token is the oracle's arg max given the
    tokens before it (or within the dtype's margin of it)."""
    from redline_b200.runtime import Engine
    d, w = models[name, dtype]
    cfg = C.ALL[name]
    prompts = [random_tokens(cfg["vocab"], n, 30 + i) for i, n in enumerate((5, 70, 33, 1, 18, 90))]
    eng = Engine(d, dtype=dtype, max_seqs=4, max_seq_len=256, kv_cache_tokens=512, **opts)
    outs = eng.generate(prompts, max_new_tokens=12, ignore_eos=True)
    margin = 1e-3 if dtype == "float32" else 0.25
    assert (eng._engine.runner.num_graph_steps > 0) == bool(opts.get("cuda_graphs", True))
    for p, o in zip(prompts, outs):
        assert len(o["output_ids"]) == 12
        seq = p + o["output_ids"]
        ref = oracle(cfg, w, seq[:-1], None if dtype == "float32" else torch.bfloat16)
        for i, tok in enumerate(o["output_ids"]):
            row = ref[len(p) - 1 + i]
            assert row[tok] >= row.max() - margin, (name, dtype, i, tok, int(row.argmax()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(dtype, models, tmp_path):
    name = "mix"
    model_dir, w = models[name, dtype]
    cfg = C.ALL[name]
    V = cfg["vocab"]
    a, b = random_tokens(V, 70, 11), random_tokens(V, 45, 12)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[40:42], "want": [1]},
                                {"id": "b", "tokens": b[:45], "want": [44]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[42:43], "want": []}], "end": []},
        {"step": 3, "entries": [{"id": "a", "tokens": a[43:70], "want": [26]},
                                {"id": "c", "tokens": b[:2], "want": [1, 0]}], "end": ["a", "c"]},
    ]
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", model_dir,
                           "--dtype", dtype, "--out", str(out), "--max-tokens", "256"],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                          timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (out / "2.f32").exists()
    f = {i: np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V) for i in (0, 1, 3)}
    check(np.concatenate([f[0], f[1][:1], f[3][:1]]), cfg, w, a, dtype, rows=[0, 39, 41, 69])
    check(f[1][1:], cfg, w, b, dtype, rows=[44])
    check(f[3][1:], cfg, w, b[:2], dtype, rows=[1, 0])


def test_command_line_with_random_weights(tmp_path):
    """`bin/redline_generate --random-weights`: the framework writes a seeded Vogolix model from a config.json,
    generates greedily, and the plain implementation, reading that folder, agrees with every token."""
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(C.MIX))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "redline_generate"), "--random-weights", str(cfg_path),
                        "--weights-seed", "5", "--model", str(tmp_path / "rand"), "--dtype", "float32", "--prompt-ids",
                        "1,2,3,50,9", "--prompt-ids", "7", "--max-new-tokens", "8", "--ignore-eos", "--max-seq-len", "64",
                        "--kv-cache-tokens", "256", "--max-seqs", "2"], capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(x) for x in r.stdout.splitlines() if x.startswith("{")]
    assert [x["id"] for x in lines] == [0, 1] and all(len(x["output_ids"]) == 8 for x in lines)
    cfg, w = P.read_model_dir(str(tmp_path / "rand"))
    for prompt, line in zip(([1, 2, 3, 50, 9], [7]), lines):
        seq = prompt + line["output_ids"]
        ref = oracle(cfg, w, seq[:-1])
        for i, tok in enumerate(line["output_ids"]):
            row = ref[len(prompt) - 1 + i]
            assert row[tok] >= row.max() - 1e-3, (i, tok, int(row.argmax()))
