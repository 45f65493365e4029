"""Lakatar's host side and its plain implementation: configuration round trip and errors, tensor names, the shared
latent in the run order and in the cache groups, states, the random-weights writer; and each mechanism of the
plain implementation against a second way to compute it."""

import json
import math
import os

import numpy as np
import pytest
import torch

import lakatar_configs as C
import plain_lakatar as P
from redline_b200.config import ConfigError, config_from_dict, load_config, model_spec
from redline_b200.engine.model import DecoderModel
from redline_b200.parts.base import Runtime
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
    m = model_of(cfg)
    assert {k: tuple(v.shape) for k, v in m.expected_tensors().items()} == P.tensor_shapes(cfg)


def test_what_the_configuration_leaves_out():
    cfg = C.clone(C.MIX)
    f = cfg["layers"][0]["mlp"]
    del f["router"]["groups"], f["router"]["scale"], f["shared"]
    c = config_from_dict(cfg)
    m = c.layers[0].mlp
    assert (m.groups, m.group_keep, m.scale, m.shared_ff) == (1, 1, 1.0, 0)
    assert c.layers[2].mixer.rot.scaling is None and c.layers[2].mlp is None
    # the inner size of the decays' products comes from the file's tensor shapes
    del cfg["layers"][1]["mixer"]["decay_rank"]
    with pytest.raises(ConfigError, match="decay_rank"):
        config_from_dict(cfg)


def test_the_inner_size_of_the_decays_products_is_the_tensors_shape(tmp_path):
    w = P.random_weights(C.WKVS, 1)
    bare = C.clone(C.WKVS)
    for layer in bare["layers"]:
        del layer["mixer"]["decay_rank"]
    P.write_model_dir(str(tmp_path), bare, w)
    assert [l.mixer.decay_rank for l in load_config(str(tmp_path)).layers] == [24, 8, 16]


@pytest.mark.parametrize("change,where", [
    (lambda c: c["layers"][0].update(type="mamba"), r"layers\[0\]"),
    (lambda c: c["layers"][3]["mixer"].update(decay=[0.5]), r"layers\[3\].mixer"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(dims=64), r"layers\[3\].mixer: rot.dims"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=4), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_rank=48), "kv_rank"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "dense"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c.pop("postln_alpha"), "postln_alpha"),
])
def test_errors_name_the_key(change, where):
    cfg = C.clone(C.MIX)
    change(cfg)
    with pytest.raises(ConfigError, match=where):
        config_from_dict(cfg)


def test_a_shared_latent_owns_no_cache():
    m = model_of(C.LATENTS)
    assert [c.cache_of for c in m.spec.order] == [None, 0, None, 0]
    groups = {g.spec.tensors[0].shape: g.owners for g in m.cache_groups()}
    assert groups == {(1, 64): [0], (1, 96): [2]}
    states = model_of(C.MIX).state_specs()
    assert sorted(states) == [1, 3, 5]
    assert [s.shape for s in states[1]] == [(3 * 16 * 16,), (96,)] and states[3].shape == (2, 32, 48)


def test_random_weights_are_what_the_model_expects(tmp_path):
    write_random_model(str(tmp_path), config_from_dict(C.MIX), seed=3)
    cfg, w = P.read_model_dir(str(tmp_path))
    assert cfg == C.MIX or config_from_dict(cfg) == config_from_dict(C.MIX)
    assert {k: tuple(v.shape) for k, v in w.items()} == P.tensor_shapes(C.MIX)
    m = model_of(C.MIX)
    m.load_weights(CheckpointReader(str(tmp_path)))
    norm = m.blocks[0].mixer_post_norm
    assert torch.allclose(norm.weight, 1.0 + w["l0.norm1"]) and torch.allclose(norm.scale, w["l0.ls1"])
    mix = m.blocks[1].mixer
    assert torch.equal(mix.w_each[2], w["l1.mix.v"]) and torch.equal(mix.mu[4], w["l1.mix.mu.w"])
    moe = m.blocks[0].ffn
    assert torch.equal(moe.w_router[6:7], w["l0.mlp.shared.sg"]) and torch.equal(moe.w_router[:6], w["l0.mlp.router"])
    lat = m.blocks[4].mixer
    assert lat.w_norm is None and torch.equal(lat.w_proj, torch.cat([w["l4.mix.dq"], w["l4.mix.g"]]))
    logits = P.forward(C.MIX, w, [1, 5, 9])
    assert torch.isfinite(logits).all()


# ---------------------------------------------------------------------------- the plain implementation's mechanisms

def test_time_mixing_written_out():
    """o_t from the definition as a sum over earlier tokens with products of decays."""
    g = torch.Generator().manual_seed(2)
    T, d = 7, 5
    r, k, v = (torch.randn(T, d, generator=g, dtype=torch.float64) for _ in range(3))
    w, u = torch.rand(T, d, generator=g, dtype=torch.float64), torch.randn(d, generator=g, dtype=torch.float64)
    got = P.channel_decay_recurrence(r, k, v, w, u)
    for t in range(T):
        want = (r[t] * u * k[t]).sum() * v[t]
        for s in range(t):
            want = want + (r[t] * k[s] * w[s + 1:t].prod(0)).sum() * v[s]
        assert torch.allclose(got[t], want)


def test_retention_written_out():
    g = torch.Generator().manual_seed(3)
    T, d, e, c = 6, 4, 3, 0.8
    q, k, v = (torch.randn(T, n, generator=g, dtype=torch.float64) for n in (d, d, e))
    got = P.scalar_decay_recurrence(q, k, v, c)
    for t in range(T):
        assert torch.allclose(got[t], sum(c ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1)))


def test_the_first_token_is_mixed_with_zeros():
    x = torch.randn(3, 4, dtype=torch.float64)
    s = P.shifted(x)
    assert torch.equal(s[0], torch.zeros(4, dtype=torch.float64)) and torch.equal(s[1:], x[:2])


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


def test_stretched_frequencies():
    from redline_b200.parts.rope import RotaryPairsParams, yarn_frequencies
    for base, dims, s in ((10000.0, 32, (4.0, 64, 8.0, 1.0)), (100.0, 6, (2.5, 30, 4.0, 0.5)), (5e5, 64, (16.0, 4096, 32.0, 1.0)),
                          (1e4, 16, (1.0, 100, 32.0, 1.0))):
        sc = dict(zip(("factor", "original", "fast", "slow"), s))
        f, mag = P.stretched_frequencies(base, dims, sc)
        g, mag2 = yarn_frequencies(RotaryPairsParams(dims, base, 10, *s))
        assert np.allclose(f, g) and math.isclose(mag, mag2)
        plain = P.plain_frequencies(base, dims)
        assert f[0] <= plain[0] + 1e-12 and f[-1] >= plain[-1] / s[0] - 1e-15
        assert math.isclose(mag, 0.1 * math.log(s[0]) + 1.0)


def test_groups_keep_their_negative_choices():
    """All choice scores may be negative: the other groups count as minus infinity, not as 0."""
    s = torch.tensor([[0.1, 0.2, 0.3, 0.4]], dtype=torch.float64)
    corr = torch.tensor([-1.0, -1.0, -2.0, -2.0], dtype=torch.float64)
    pick = P.choose(s, corr, {"top": 2, "groups": {"count": 2, "keep": 1}})
    assert sorted(pick[0].tolist()) == [0, 1]
    # the group of the single best choice score stays, whatever the other scores in it
    s = torch.tensor([[0.5, 0.0, 0.3, 0.3]], dtype=torch.float64)
    assert sorted(P.choose(s, torch.zeros(4, dtype=torch.float64), {"top": 2, "groups": {"count": 2, "keep": 1}})[0].tolist()) == [0, 1]


def test_attention_over_latents_needs_no_keys():
    """The identities that let the engine attend over the cached rows: keys and values formed per head, or the query
    taken through W_uk and the attended latents through W_uv; the head's gate commutes with W_uv."""
    g = torch.Generator().manual_seed(6)
    T, d, e, rank = 5, 4, 3, 6
    q, c = torch.randn(T, d, generator=g, dtype=torch.float64), torch.randn(T, rank, generator=g, dtype=torch.float64)
    uk, uv = torch.randn(d, rank, generator=g, dtype=torch.float64), torch.randn(e, rank, generator=g, dtype=torch.float64)
    gate = torch.rand(T, 1, generator=g, dtype=torch.float64)
    direct = (P.causal_softmax(q @ (c @ uk.T).T) @ (c @ uv.T)) * gate
    absorbed = ((P.causal_softmax((q @ uk) @ c.T) @ c) * gate) @ uv.T
    assert torch.allclose(direct, absorbed)


def test_the_norm_is_of_the_sum():
    x, y, s, w = (torch.randn(2, 8, dtype=torch.float64) for _ in range(4))
    got = P.summed_norm(x, y, 1.7, s, w, 1e-5)
    u = 1.7 * x + s * y
    assert torch.allclose(got, u / torch.sqrt((u ** 2).mean(-1, keepdim=True) + 1e-5) * (1 + w))
    assert not torch.allclose(P.summed_norm(x, y, 1.0, s, w, 1e-5), got)
