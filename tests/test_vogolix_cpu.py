"""Vogolix's host side and its plain implementation: configuration round trip and errors, tensor names, shared keys
in the run order and in the cache groups, what a chunk's pages are kept for, states, the random-weights writer; and each
mechanism of the plain implementation against a second way to compute it."""

import math

import pytest
import torch

import plain_vogolix as P
import vogolix_configs as C
from redline_b200.cache.manager import CacheManager, GroupInfo
from redline_b200.config import ConfigError, config_from_dict, model_spec
from redline_b200.engine.model import DecoderModel
from redline_b200.parts.base import Runtime
from redline_b200.parts.spec import CacheSpec
from redline_b200.weights import write_random_model
from redline_b200.weights.safetensors_io import CheckpointReader


def model_of(cfg_dict, dtype=torch.float32):
    rt = Runtime(device=torch.device("cpu"), dtype=dtype, max_tokens=64, max_seqs=4, max_seq_len=256, page_size=16)
    return DecoderModel(model_spec(config_from_dict(cfg_dict)), rt)


@pytest.mark.parametrize("name", list(C.ALL))
def test_configuration_round_trip_and_tensor_names(name):
    cfg = C.ALL[name]
    c = config_from_dict(cfg)
    assert config_from_dict(c.to_hf()) == c
    assert {k: tuple(v.shape) for k, v in model_of(cfg).expected_tensors().items()} == P.tensor_shapes(cfg)


def test_what_the_configuration_leaves_out():
    cfg = C.clone(C.MIX)
    del cfg["logit_scale"], cfg["layers"][0]["mixer"]["kv_heads"], cfg["layers"][6]["mixer"]["mask"]
    cfg["layers"][3]["mixer"]["kv_heads"] = cfg["layers"][5]["mixer"]["kv_heads"] = 4
    cfg["layers"][3]["mixer"]["heads"] = cfg["layers"][5]["mixer"]["heads"] = 4
    c = config_from_dict(cfg)
    assert c.logit_scale == 1.0 and c.layers[0].mixer.kv_heads == 4 and c.layers[6].mixer.window == 0
    assert config_from_dict(c.to_hf()) == c
    assert c.layers[2].ff == 0 and "l2.norm2" not in model_of(cfg).expected_tensors()


@pytest.mark.parametrize("change,where", [
    (lambda c: c["layers"][0].update(type="wkv"), r"layers\[0\]"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=64), r"layers\[0\].mixer: rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), r"layers\[0\].mixer: rot.dims"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=32), "vdim"),
    (lambda c: c["layers"][2]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_errors_name_the_key(change, where):
    cfg = C.clone(C.MIX)
    change(cfg)
    with pytest.raises(ConfigError, match=where):
        config_from_dict(cfg)


def test_shared_keys_and_what_they_are_kept_for():
    m = model_of(C.MIX)
    assert [c.cache_of for c in m.spec.order] == [None, None, None, 0, None, 0, None]
    # three layers read the first one's keys under chunks of 50, 50 and 83 positions: a window of 83 holds them all
    assert {(g.spec.kind, g.spec.window): g.owners for g in m.cache_groups()} == {("window", 83): [0], ("window", 37): [2],
                                                                                  ("window", 64): [6]}
    assert {(g.spec.kind, g.spec.window): g.owners for g in model_of(C.CHUNKS).cache_groups()} == {("chunk", 33): [0], ("chunk", 128): [2]}
    open_ended = C.clone(C.CHUNKS)
    del open_ended["layers"][1]["mixer"]["mask"]
    assert [(g.spec.kind, g.owners) for g in model_of(open_ended).cache_groups()] == [("full", [0]), ("chunk", [2])]
    states = model_of(C.MIX).state_specs()
    assert sorted(states) == [1, 4]
    assert [s.shape for s in states[1]] == [(4 * 32 * 16,), (2 * (64 + 2 * 2 * 32),)]
    assert model_of(C.ODD).state_specs()[0].shape == (3 * 10 * 7,)              # one tap: no inputs are carried


def test_a_chunks_pages_go_back_when_the_next_one_begins():
    def group(kind, size):
        return GroupInfo(CacheSpec.keys_values(kind, 1, 8, size), [0])
    m = CacheManager([group("chunk", 40), group("window", 40), group("chunk", 8)], [40, 40, 40], 16, 2)
    rc = m.open("a")
    held = []
    for n in range(1, 200):
        assert m.reserve(rc, n)
        m.release_passed(rc, n)
        m.check_invariants()
        held.append([sum(1 for p in rc.table(g) if p) for g in range(3)])
        for g, first in ((0, n // 40 * 40), (1, max(0, n - 39)), (2, n // 8 * 8)):
            # every key that token n sees has its page; pages that lie before its first key as a whole have gone
            table = rc.table(g)
            assert all(table[j // 16] for j in range(first, n)), (g, n)
            assert not any(table[b] for b in range(first // 16)), (g, n)
    assert max(h[0] for h in held) == 3 and max(h[1] for h in held) <= 4 and max(h[2] for h in held) == 1
    m.close("a")
    assert [m.num_free_pages(g) for g in range(3)] == [39, 39, 39]
    m.check_invariants()


def test_random_weights_are_what_the_model_expects(tmp_path):
    write_random_model(str(tmp_path), config_from_dict(C.MIX), seed=3)
    cfg, w = P.read_model_dir(str(tmp_path))
    assert config_from_dict(cfg) == config_from_dict(C.MIX)
    assert {k: tuple(v.shape) for k, v in w.items()} == P.tensor_shapes(C.MIX)
    m = model_of(C.MIX)
    m.load_weights(CheckpointReader(str(tmp_path)))
    att, shared = m.blocks[0].mixer, m.blocks[3].mixer
    assert torch.equal(att.w_qkv, torch.cat([w["l0.mix.q"], w["l0.mix.k"], w["l0.mix.v"]]))
    assert torch.equal(att.b_qkv, torch.cat([w["l0.mix.q.b"], w["l0.mix.k.b"], w["l0.mix.v.b"]]))
    assert torch.equal(shared.w_qkv, w["l3.mix.q"]) and torch.equal(shared.b_qkv, w["l3.mix.q.b"]) and shared.w_knorm is None
    lat = m.blocks[2].mixer
    assert torch.equal(lat.w_proj, torch.cat([w["l2.mix.q"], w["l2.mix.dkv"], w["l2.mix.g"]]))
    space = m.blocks[1].mixer
    assert torch.equal(space.w_in, w["l1.mix.in"]) and torch.equal(space.b_conv, w["l1.mix.conv.b"])
    # the factor on the logits joins the final norm's weight
    assert torch.allclose(m.final_norm.weight, w["final.norm"] * 0.7)
    assert torch.isfinite(P.forward(C.MIX, w, [1, 5, 9])).all()


# ---------------------------------------------------------------------------- the plain implementation's mechanisms

def test_the_recurrence_written_out():
    """y_t as a sum over the tokens up to t with products of decays."""
    g = torch.Generator().manual_seed(2)
    T, e, N = 7, 3, 5
    x, B, Cm = (torch.randn(T, n, generator=g, dtype=torch.float64) for n in (e, N, N))
    dt, a, D = torch.rand(T, generator=g, dtype=torch.float64), torch.tensor(0.3, dtype=torch.float64), torch.tensor(-0.7, dtype=torch.float64)
    y, S = P.state_space_recurrence(x, B, Cm, dt, a, D)
    decay = torch.exp(-math.exp(0.3) * dt)
    for t in range(T):
        want = D * x[t]
        for s in range(t + 1):
            want = want + (Cm[t] @ B[s]) * decay[s + 1:t + 1].prod() * dt[s] * x[s]
        assert torch.allclose(y[t], want)
    # cut in two, the state carried over
    y0, S0 = P.state_space_recurrence(x[:4], B[:4], Cm[:4], dt[:4], a, D)
    y1, S1 = P.state_space_recurrence(x[4:], B[4:], Cm[4:], dt[4:], a, D, S0)
    assert torch.allclose(torch.cat([y0, y1]), y) and torch.allclose(S1, S)


def test_the_recurrence_in_blocks():
    """The identities the block form rests on: with l the running sums of the decays' logarithms, the state before a
    block is read out once, pairs within it by their own products, and moved on by weighted values."""
    g = torch.Generator().manual_seed(3)
    T, e, N = 9, 4, 6
    x, B, Cm = (torch.randn(T, n, generator=g, dtype=torch.float64) for n in (e, N, N))
    dt, a, D = torch.rand(T, generator=g, dtype=torch.float64), torch.tensor(-0.2, dtype=torch.float64), torch.tensor(0.4, dtype=torch.float64)
    S0 = torch.randn(N, e, generator=g, dtype=torch.float64)
    want, S1 = P.state_space_recurrence(x, B, Cm, dt, a, D, S0)
    logs = torch.cumsum(-torch.exp(a) * dt, 0)
    M = (Cm @ B.T) * torch.exp(logs[:, None] - logs[None, :]).tril() * dt[None, :] + D * torch.eye(T, dtype=torch.float64)
    assert torch.allclose(torch.exp(logs)[:, None] * (Cm @ S0) + M @ x, want)
    assert torch.allclose(torch.exp(logs[-1]) * S0 + B.T @ (x * (dt * torch.exp(logs[-1] - logs))[:, None]), S1)


def test_the_convolution_written_out():
    u, w, b = torch.randn(5, 2, dtype=torch.float64), torch.randn(2, 3, dtype=torch.float64), torch.randn(2, dtype=torch.float64)
    y = P.causal_conv(u, w, b)
    assert torch.allclose(y[0], w[:, 2] * u[0] + b)
    assert torch.allclose(y[4], w[:, 0] * u[2] + w[:, 1] * u[3] + w[:, 2] * u[4] + b)


def test_the_gate_comes_before_the_norm_and_parts_are_normed_by_themselves():
    y, z, w = (torch.randn(2, 8, dtype=torch.float64) for _ in range(3))
    got = P.grouped_gated_norm(y, z, w[0], 2, 1e-5)
    u = y * torch.nn.functional.silu(z)
    for part in (slice(0, 4), slice(4, 8)):
        assert torch.allclose(got[:, part], u[:, part] / torch.sqrt((u[:, part] ** 2).mean(-1, keepdim=True) + 1e-5) * w[0, part])
    assert not torch.allclose(P.grouped_gated_norm(y, z, w[0], 1, 1e-5), got)


def test_masks():
    c = P.chunk_mask(9, 4)
    assert c.sum(1).tolist() == [1, 2, 3, 4, 1, 2, 3, 4, 1] and bool(c[5, 4]) and not bool(c[4, 3]) and not bool(c[4, 5])
    w = P.window_mask(6, 3)
    assert w.sum(1).tolist() == [1, 2, 3, 3, 3, 3] and bool(w[5, 3]) and not bool(w[5, 2])


def test_a_sink_counts_once_and_is_no_key():
    s, sink = torch.tensor([[1.0, 9.0], [2.0, 0.5]], dtype=torch.float64), torch.tensor(1.5, dtype=torch.float64)
    p = P.masked_softmax(s, P.window_mask(2, None), sink)
    assert torch.allclose(p[0], torch.tensor([math.e / (math.e + math.exp(1.5)), 0.0], dtype=torch.float64))
    assert torch.allclose(p[1].sum(), 1 - math.exp(1.5) / (math.exp(2.0) + math.exp(0.5) + math.exp(1.5)) * torch.ones((), dtype=torch.float64))


def test_rotations():
    g = torch.Generator().manual_seed(4)
    x, y = torch.randn(5, 10, generator=g, dtype=torch.float64), torch.randn(5, 10, generator=g, dtype=torch.float64)
    rot = {"base": 50.0, "dims": 6}
    for f in (P.rotate_halves, P.rotate_pairs):
        a, b = f(x, rot, [3] * 5), f(y, rot, [9] * 5)
        c, d = f(x, rot, [103] * 5), f(y, rot, [109] * 5)
        assert torch.allclose((a * b).sum(-1), (c * d).sum(-1))                # the distance alone counts
        assert torch.equal(a[:, 6:], x[:, 6:])
    h, n = P.rotate_halves(x, rot, [2] * 5), P.rotate_pairs(x, rot, [2] * 5)
    a = 2 * 50.0 ** (-2.0 / 6)                                                 # pair 1: entries (1, 4), or (2, 3)
    assert torch.allclose(h[:, 1], x[:, 1] * math.cos(a) - x[:, 4] * math.sin(a))
    assert torch.allclose(n[:, 3], x[:, 3] * math.cos(a) + x[:, 2] * math.sin(a))


def test_attention_over_latents_needs_no_keys():
    """The identities that let the engine attend over the cached rows; a gate per entry comes behind W_uv."""
    g = torch.Generator().manual_seed(6)
    T, d, e, rank = 5, 4, 3, 6
    q, c = torch.randn(T, d, generator=g, dtype=torch.float64), torch.randn(T, rank, generator=g, dtype=torch.float64)
    uk, uv = torch.randn(d, rank, generator=g, dtype=torch.float64), torch.randn(e, rank, generator=g, dtype=torch.float64)
    gate, seen = torch.rand(T, e, generator=g, dtype=torch.float64), P.window_mask(T, 3)
    direct = (P.masked_softmax(q @ (c @ uk.T).T, seen) @ (c @ uv.T)) * gate
    absorbed = ((P.masked_softmax((q @ uk) @ c.T, seen) @ c) @ uv.T) * gate
    assert torch.allclose(direct, absorbed)
