"""``Lakatar`` laid out as parts: a token embedding; "postnorm" blocks (the stream is RMS-normed after every sum,
h = norm(alpha h + s * sublayer(h)), weights stored around zero, ``rmsnorm_sum``) whose mixer is RWKV-style time
mixing (``time_mix``), retention (``linear_attention`` without activations: rotated queries and keys, keys scaled
by dim^(-1/2), every head's output divided by its root mean square, a SiLU gate) or attention over a cached
latent (``latent_attention``: queries from a latent of their own, a rotated key part in neighbouring pairs with
YaRN scaling, a sigmoid gate per head; a layer may read an earlier one's cache, ``LayerCall.cache_of``); routed
SiLU-gated experts (``routed_experts``: softmax scores, a corrected choice within the best groups, scaled
weights, a shared expert with a gate per token), or none; a final RMS norm and a head of its own.  Tensor names:
``embed``, ``l<i>.norm1|norm2|ls1|ls2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import math
from typing import Iterator, Tuple

import torch

from ..config.model_config import LakatarConfig, LakatarRotation
from ..config.registry import Architecture, register_architecture
from ..parts.embedding import EmbeddingParams, HeadParams
from ..parts.latent_attention import LatentAttentionParams
from ..parts.linear_attention import LinearAttentionParams
from ..parts.moe import RoutedExpertsParams
from ..parts.rmsnorm import RMSNormParams, RMSNormSumParams
from ..parts.rope import RotaryHalvesParams, RotaryPairsParams
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..parts.time_mix import MIXES, TimeMixParams

GROUP_TOP = 1                  # a group of experts is scored by its best one


def _rotation(kind: str, params: type, r: LakatarRotation, max_positions: int) -> PartSpec:
    s = r.scaling
    return PartSpec(kind, params(r.dims, r.base, max_positions, *((s.factor, s.original, s.fast, s.slow) if s else ())))


def lakatar_spec(c: LakatarConfig) -> ModelSpec:
    W = c.hidden_size

    def closing(p: str, n: int) -> PartSpec:
        return PartSpec("rmsnorm_sum", RMSNormSumParams(W, c.norm_eps, c.alpha, zero_centred=True, scaled=True),
                        {"weight": f"{p}norm{n}", "scale": f"{p}ls{n}"})

    layers = []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        m = layer.mixer
        if layer.type == "wkv":
            names = {n: f"{p}mix.{n}" for n in ("r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o")}
            names.update({f"mu_{s}": f"{p}mix.mu.{s}" for s in MIXES})
            mixer = PartSpec("time_mix", TimeMixParams(W, m.heads, m.dim, m.decay_rank, c.norm_eps), names)
        elif layer.type == "retention":
            mixer = PartSpec("linear_attention", LinearAttentionParams(
                hidden_size=W, num_heads=m.heads, dim=m.dim, vdim=m.vdim, decay=m.decay, eps=c.norm_eps,
                activation="none", gate_activation="silu", head_norm=True, k_scale=m.dim ** -0.5,
                position=_rotation("rope_halves", RotaryHalvesParams, m.rot, c.max_position_embeddings)
                if m.rot is not None else None),
                {n: f"{p}mix.{n}" for n in ("q", "k", "v", "g", "o")})
        else:
            own = m.kv_from is None
            names = {n: f"{p}mix.{n}" for n in ("dq", "uq", "uk", "uv", "g", "o")}
            names["dq_norm"] = p + "mix.dq.norm"
            if own:
                names.update({"dkv": p + "mix.dkv", "dkv_norm": p + "mix.dkv.norm"})
            mixer = PartSpec("latent_attention", LatentAttentionParams(
                hidden_size=W, num_heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.kv_rank,
                scale=m.scale, eps=c.norm_eps, q_rank=m.q_rank, gate="head", own_latent=own,
                position=_rotation("rope_pairs", RotaryPairsParams, m.rot, c.max_position_embeddings)
                if m.rot_dim > 0 else None), names)
        f = layer.mlp
        ffn = None
        if f is not None:
            names = {"router": p + "mlp.router", "choice_bias": p + "mlp.correction"}
            for e in range(f.experts):
                names.update({f"{n}{e}": f"{p}mlp.e{e}.{n}" for n in ("gate", "up", "down")})
            if f.shared_ff > 0:
                names.update({f"shared_{n}": f"{p}mlp.shared.{n}" for n in ("gate", "up", "down", "sg")})
            ffn = PartSpec("routed_experts", RoutedExpertsParams(
                hidden_size=W, intermediate_size=f.ff, num_experts=f.experts, top=f.top, groups=f.groups,
                group_keep=f.group_keep, group_top=GROUP_TOP, score="softmax", activation="silu", gated=True,
                choice_bias=True, weight_scale=f.scale, shared_intermediate_size=f.shared_ff,
                shared_gate=f.shared_ff > 0), names)
        layers.append(LayerSpec(arrangement="postnorm", mixer_norm=None, mixer=mixer, ffn_norm=None, ffn=ffn,
                                mixer_post_norm=closing(p, 1), ffn_post_norm=closing(p, 2) if ffn is not None else None))
    order = tuple(LayerCall(i, cache_of=getattr(layer.mixer, "kv_from", None)) for i, layer in enumerate(c.layers))
    return ModelSpec(
        hidden_size=W, vocab_size=c.vocab_size, max_positions=c.max_position_embeddings,
        embedding=PartSpec("token_embedding", EmbeddingParams(c.vocab_size, W), {"weight": "embed"}),
        layers=tuple(layers), order=order,
        final_norm=PartSpec("rmsnorm", RMSNormParams(W, c.norm_eps, zero_centred=True), {"weight": "final.norm"}),
        head=PartSpec("lm_head", HeadParams(c.vocab_size, W, False), {"weight": "head"}))


def lakatar_random_tensors(c: LakatarConfig, seed: int, dtype: torch.dtype) -> Iterator[Tuple[str, tuple, object]]:
    """Yields (name, shape, make) in file order: matrices N(0, 1 / fan_in), the embedding N(0, 1), zero-centred norm
    weights N(0, 0.1^2), the others and layer scales 1 + N(0, 0.1^2), mixing weights around 1/2, the decays' w0 around
    -3, choice corrections N(0, 0.02^2); one seeded generator run in order."""
    g = torch.Generator().manual_seed(seed)
    W = c.hidden_size

    def mat(n, k, std=None):
        return (n, k), lambda: (torch.randn(n, k, generator=g) * (std if std is not None else 1.0 / math.sqrt(k))).to(dtype)

    def vec(n, mean, std):
        return (n,), lambda: (mean + std * torch.randn(n, generator=g)).to(dtype)

    def emit(name, shape_make):
        return name, shape_make[0], shape_make[1]

    yield emit("embed", mat(c.vocab_size, W, 1.0))
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        m = layer.mixer
        q = p + "mix."
        yield emit(p + "norm1", vec(W, 0.0, 0.1))
        yield emit(p + "ls1", vec(W, 1.0, 0.1))
        if layer.type == "wkv":
            n = m.heads * m.dim
            for s in MIXES:
                yield emit(q + "mu." + s, vec(W, 0.5, 0.2))
            for s in ("r", "k", "v", "g"):
                yield emit(q + s, mat(n, W))
            yield emit(q + "w1", mat(m.decay_rank, W))
            yield emit(q + "w2", mat(n, m.decay_rank))
            yield emit(q + "w0", vec(n, -3.0, 1.0))
            yield emit(q + "u", mat(m.heads, m.dim, 0.5))
            yield emit(q + "norm", vec(n, 1.0, 0.1))
            yield emit(q + "o", mat(W, n))
        elif layer.type == "retention":
            for s, rows in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)):
                yield emit(q + s, mat(rows, W))
            yield emit(q + "o", mat(W, m.heads * m.vdim))
        else:
            yield emit(q + "dq", mat(m.q_rank, W))
            yield emit(q + "dq.norm", vec(m.q_rank, 1.0, 0.1))
            yield emit(q + "uq", mat(m.heads * (m.dim + m.rot_dim), m.q_rank))
            if m.kv_from is None:
                yield emit(q + "dkv", mat(m.kv_rank + m.rot_dim, W))
                yield emit(q + "dkv.norm", vec(m.kv_rank, 1.0, 0.1))
            yield emit(q + "uk", mat(m.heads * m.dim, m.kv_rank))
            yield emit(q + "uv", mat(m.heads * m.vdim, m.kv_rank))
            yield emit(q + "g", mat(m.heads, W))
            yield emit(q + "o", mat(W, m.heads * m.vdim))
        f = layer.mlp
        if f is None:
            continue
        yield emit(p + "norm2", vec(W, 0.0, 0.1))
        yield emit(p + "ls2", vec(W, 1.0, 0.1))
        widths = [(f"e{e}", f.ff) for e in range(f.experts)] + ([("shared", f.shared_ff)] if f.shared_ff > 0 else [])
        for name, ff in widths:
            yield emit(f"{p}mlp.{name}.gate", mat(ff, W))
            yield emit(f"{p}mlp.{name}.up", mat(ff, W))
            yield emit(f"{p}mlp.{name}.down", mat(W, ff))
        if f.shared_ff > 0:
            yield emit(p + "mlp.shared.sg", mat(1, W))
        yield emit(p + "mlp.router", mat(f.experts, W))
        yield emit(p + "mlp.correction", vec(f.experts, 0.0, 0.02))
    yield emit("final.norm", vec(W, 0.0, 0.1))
    yield emit("head", mat(c.vocab_size, W))


register_architecture(Architecture(
    name="Lakatar",
    config_from_hf=LakatarConfig.from_hf,
    build_spec=lakatar_spec,
    random_tensors=lakatar_random_tensors,
))
