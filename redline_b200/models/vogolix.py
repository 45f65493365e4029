"""``Vogolix`` laid out as parts: a token embedding; "prenorm" blocks whose mixer is a state-space layer
(``state_space``: Mamba-2), attention over a cached latent (``latent_attention``: a window, a rotated key part whose
entries turn with the one half away, a gate per output entry) or grouped attention within chunks of positions
(``maps_attention`` with one map: biases, queries and keys normed over the whole projection, the heads' first
entries rotated in neighbouring pairs, a sink; a layer may use an earlier one's keys and values,
``LayerCall.cache_of``), and whose feed-forward is dense and gated by a ReLU, or absent; a final RMS norm and a head
of its own, whose logits are multiplied by a constant (formed with the final norm's weight).  Tensor names:
``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import math
from typing import Iterator, Tuple

import torch

from ..config.model_config import VogolixConfig, VogolixRotation
from ..config.registry import Architecture, register_architecture
from ..parts.attention_maps import MapsAttentionParams
from ..parts.embedding import EmbeddingParams, HeadParams
from ..parts.latent_attention import LatentAttentionParams
from ..parts.mlp import GatedMLPParams
from ..parts.rmsnorm import RMSNormParams
from ..parts.rope import RotaryHalvesParams, RotaryPairsParams
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..parts.state_space import StateSpaceParams


def _kept_span(c: VogolixConfig, owner: int) -> Tuple[str, int]:
    """What the keys of attention layer ``owner`` must be kept for: the chunk, if every layer that reads them has the
    same one, else a window as long as the largest chunk (every chunk's visible keys lie in it)."""
    spans = {layer.mixer.chunk for i, layer in enumerate(c.layers)
             if i == owner or getattr(layer.mixer, "kv_from", None) == owner}
    if 0 in spans:
        return "full", 0
    return ("chunk" if len(spans) == 1 else "window"), max(spans)


def vogolix_spec(c: VogolixConfig) -> ModelSpec:
    W = c.hidden_size

    def rotation(kind: str, params: type, r: VogolixRotation) -> PartSpec:
        return PartSpec(kind, params(r.dims, r.base, c.max_position_embeddings))

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", RMSNormParams(W, c.norm_eps), {"weight": name})

    layers = []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        m = layer.mixer
        if layer.type == "mamba2":
            names = {n: f"{p}mix.{n}" for n in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}
            names["conv_bias"] = p + "mix.conv.b"
            mixer = PartSpec("state_space", StateSpaceParams(
                hidden_size=W, num_heads=m.heads, vdim=m.vdim, state=m.state, groups=m.groups, conv_taps=m.conv,
                norm_groups=m.norm_groups, eps=c.norm_eps), names)
        elif layer.type == "latent_attention":
            names = {n: f"{p}mix.{n}" for n in ("q", "dkv", "uk", "uv", "g", "o")}
            names["dkv_norm"] = p + "mix.dkv.norm"
            mixer = PartSpec("latent_attention", LatentAttentionParams(
                hidden_size=W, num_heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.kv_rank, scale=m.scale,
                eps=c.norm_eps, gate="entry", window=m.window,
                position=rotation("rope_halves", RotaryHalvesParams, m.rot) if m.rot_dim > 0 else None), names)
        else:
            own = m.kv_from is None
            names = {n: f"{p}mix.{n}" for n in ("q", "sink", "o")}
            names.update({"q_bias": p + "mix.q.b", "q_norm": p + "mix.q.norm"})
            if own:
                names.update({"k": p + "mix.k", "v": p + "mix.v", "k_bias": p + "mix.k.b", "v_bias": p + "mix.v.b",
                              "k_norm": p + "mix.k.norm"})
            mixer = PartSpec("maps_attention", MapsAttentionParams(
                hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, bias=True, scale=m.scale,
                eps=c.norm_eps, head_norm="whole", sink=True, chunk=m.chunk, own_kv=own,
                keep_for=_kept_span(c, i if own else m.kv_from),
                position=rotation("rope_pairs", RotaryPairsParams, m.rot) if m.rot is not None else None), names)
        ffn = None
        if layer.ff > 0:
            ffn = PartSpec("swiglu_mlp", GatedMLPParams(W, layer.ff, activation="relu"),
                           {n: f"{p}mlp.{n}" for n in ("gate", "up", "down")})
        layers.append(LayerSpec(arrangement="prenorm", mixer_norm=norm(p + "norm1"), mixer=mixer,
                                ffn_norm=norm(p + "norm2") if ffn is not None else None, ffn=ffn))
    return ModelSpec(
        hidden_size=W, vocab_size=c.vocab_size, max_positions=c.max_position_embeddings,
        embedding=PartSpec("token_embedding", EmbeddingParams(c.vocab_size, W), {"weight": "embed"}),
        layers=tuple(layers),
        order=tuple(LayerCall(i, cache_of=getattr(layer.mixer, "kv_from", None)) for i, layer in enumerate(c.layers)),
        # (logits = s W_head N(x): the factor joins the norm's weight)
        final_norm=PartSpec("rmsnorm", RMSNormParams(W, c.norm_eps, scale=c.logit_scale), {"weight": "final.norm"}),
        head=PartSpec("lm_head", HeadParams(c.vocab_size, W, False), {"weight": "head"}))


def vogolix_random_tensors(c: VogolixConfig, seed: int, dtype: torch.dtype) -> Iterator[Tuple[str, tuple, object]]:
    """Yields (name, shape, make) in file order: matrices N(0, 1 / fan_in), the embedding N(0, 1), norm weights
    1 + N(0, 0.1^2), biases N(0, 0.1^2), sinks and D N(0, 1), step biases around -3, A_log around 1; one seeded
    generator run in order."""
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
        yield emit(p + "norm1", vec(W, 1.0, 0.1))
        if layer.type == "mamba2":
            inner, channels = m.heads * m.vdim, m.heads * m.vdim + 2 * m.groups * m.state
            yield emit(q + "in", mat(inner + channels + m.heads, W))
            yield emit(q + "conv", mat(channels, m.conv))
            yield emit(q + "conv.b", vec(channels, 0.0, 0.1))
            yield emit(q + "dt_bias", vec(m.heads, -3.0, 1.0))
            yield emit(q + "A_log", vec(m.heads, 1.0, 0.7))
            yield emit(q + "D", vec(m.heads, 0.0, 1.0))
            yield emit(q + "norm", vec(inner, 1.0, 0.1))
            yield emit(q + "o", mat(W, inner))
        elif layer.type == "latent_attention":
            yield emit(q + "q", mat(m.heads * (m.dim + m.rot_dim), W))
            yield emit(q + "dkv", mat(m.kv_rank + m.rot_dim, W))
            yield emit(q + "dkv.norm", vec(m.kv_rank, 1.0, 0.1))
            yield emit(q + "uk", mat(m.heads * m.dim, m.kv_rank))
            yield emit(q + "uv", mat(m.heads * m.vdim, m.kv_rank))
            yield emit(q + "g", mat(m.heads * m.vdim, W))
            yield emit(q + "o", mat(W, m.heads * m.vdim))
        else:
            parts = [("q", m.heads * m.dim, True)]
            if m.kv_from is None:
                parts += [("k", m.kv_heads * m.dim, True), ("v", m.kv_heads * m.vdim, False)]
            for s, rows, normed in parts:
                yield emit(q + s, mat(rows, W))
                yield emit(q + s + ".b", vec(rows, 0.0, 0.1))
                if normed:
                    yield emit(q + s + ".norm", vec(rows, 1.0, 0.1))
            yield emit(q + "sink", vec(m.heads, 0.0, 1.0))
            yield emit(q + "o", mat(W, m.heads * m.vdim))
        if layer.ff > 0:
            yield emit(p + "norm2", vec(W, 1.0, 0.1))
            yield emit(p + "mlp.gate", mat(layer.ff, W))
            yield emit(p + "mlp.up", mat(layer.ff, W))
            yield emit(p + "mlp.down", mat(W, layer.ff))
    yield emit("final.norm", vec(W, 1.0, 0.1))
    yield emit("head", mat(c.vocab_size, W))


register_architecture(Architecture(
    name="Vogolix",
    config_from_hf=VogolixConfig.from_hf,
    build_spec=vogolix_spec,
    random_tensors=vogolix_random_tensors,
))
