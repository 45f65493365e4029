"""Causal attention whose keys and values come from one latent vector per token.

Per token the mixer projects its input to queries (per head ``dim`` unrotated and ``rot_dim`` rotated entries)
and to [c' | k_r]: a latent of ``kv_rank`` entries, RMS-normed with a weight into c, and one rotated key part
of ``rot_dim`` entries that all heads share.  Head h's key is [W_uk,h c | k_r], its value W_uv,h c; scores are
scale * q . k over every earlier token (or those of a window), ordinary softmax.  Only [c | k_r] is cached (one row per token, one
"key head" for all query heads), and the keys and values are never formed:

    q_n . (W_uk,h c_j) = (W_uk,h^T q_n) . c_j          sum_j p_j W_uv,h c_j = W_uv,h (sum_j p_j c_j)

so the attention kernels (those of ``maps_attention``: csrc/attention_maps.cu) run over the cached rows with the
query [W_uk,h^T q_n | q_r] and the row's first ``kv_rank`` entries as the value, and W_uv,h is applied to what
they return.  The two per-head products and the kernel between projection and cache (norm, rotation, cache
write) are csrc/latent.cu.  The rotation is a ``rope_halves`` or ``rope_pairs`` position encoding over the
first ``rot_dims`` entries of the rotated part.  Norm, rotation, scores and softmax are float32 in both engine
types.

Further options: the queries may come from a latent of their own, q = W_uq rmsnorm(W_dq h) (``q_rank``); every
head's output may be multiplied by sigmoid(W_g h)_h (``gate`` "head"; applied by the attention kernels to what they
return, which W_uv,h maps linearly) or entry by entry ("entry": W_g h has a number per output entry; applied by the
product with W_uv,h to its result); ``window`` > 0: a token sees itself and the ``window`` - 1 tokens before it; a layer may attend over the rows that an earlier layer has cached
(``own_latent`` False: no W_dkv; its call of the run order names the other call in ``cache_of``).  What is
projected from h, [q or the queries' latent | latent | key part | gate], is one product.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch

from ..ops import kernels
from ..ops.linear import linear
from .base import LayerCache, Mixer, build_part, op_mark, register
from .spec import CacheSpec, CacheTensor, PartSpec, TensorSpec


@dataclass(frozen=True)
class LatentAttentionParams:
    hidden_size: int
    num_heads: int
    dim: int                     # unrotated entries of a head's query and key
    rot_dim: int                 # rotated entries (0: none); the key's are one vector for all heads
    vdim: int                    # size of a head's value
    kv_rank: int                 # size of the cached latent
    scale: float
    eps: float = 1e-6            # of the latent's RMS norm
    position: Optional[PartSpec] = None      # an encoding of the rotated part (needed if rot_dim > 0)
    q_rank: int = 0              # > 0: size of the latent the queries come from
    gate: str = "none"           # none | head | entry: a sigmoid gate per head or per output entry
    own_latent: bool = True      # False: another layer's cached rows are attended over
    window: int = 0              # 0: every earlier token


@register("mixer", "latent_attention")
class LatentAttention(Mixer):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = self.params
        self.key_size = p.kv_rank + p.rot_dim          # a cached row, and a head's query for the kernels
        if min(p.num_heads, p.dim, p.vdim, p.kv_rank) <= 0 or p.rot_dim < 0:
            raise ValueError("latent_attention: heads, dim, vdim and kv_rank must be positive")
        if self.key_size > kernels.MAPS_MAX_DIM or p.kv_rank > kernels.MAPS_MAX_VDIM:
            raise ValueError(f"latent_attention: kv_rank + rot_dim is {self.key_size}; the attention kernels take "
                             f"rows of up to {kernels.MAPS_MAX_DIM} entries of which {kernels.MAPS_MAX_VDIM} are the latent")
        if p.gate not in ("none", "head", "entry") or p.window < 0:
            raise ValueError(f"latent_attention: gate '{p.gate}' is not known (none, head, entry), or a negative window")
        self.cos = self.sin = None
        self.rot_dims = 0
        self.pairs = False
        if p.rot_dim > 0:
            if p.position is None:
                raise ValueError("latent_attention: a rotated part needs a position encoding")
            pos = build_part("position", p.position, rt)
            if getattr(pos, "pairing", None) not in ("halves", "neighbours") or pos.rotary_tables() is None:
                raise ValueError("latent_attention rotates entry i with entry i + half (rope_halves) or with its "
                                 "neighbour (rope_pairs)")
            self.pairs = pos.pairing == "neighbours"
            self.cos, self.sin = pos.rotary_tables()
            self.rot_dims = 2 * self.cos.shape[1]
            if self.rot_dims > p.rot_dim:
                raise ValueError(f"a rotation of {self.rot_dims} entries does not fit a rotated part of {p.rot_dim}")
        self.q_head = p.dim + p.rot_dim
        self.q_size = p.num_heads * self.q_head
        # columns of the projection from h: queries or their latent, then (own) latent and key part, then gates
        self.c_col = p.q_rank or self.q_size
        self.g_col = self.c_col + (self.key_size if p.own_latent else 0)
        self.gate_size = {"none": 0, "head": p.num_heads, "entry": p.num_heads * p.vdim}[p.gate]
        self.proj_size = self.g_col + self.gate_size
        self.qa_size = p.num_heads * self.key_size
        self.lat_size = p.num_heads * p.kv_rank
        self.out_size = p.num_heads * p.vdim

    def cache_spec(self) -> CacheSpec:
        tensors = (CacheTensor("k", (1, self.key_size)),)
        return CacheSpec("window", tensors, self.params.window) if self.params.window > 0 else CacheSpec("full", tensors)

    def tiling(self):
        return kernels.PREFILL_TILE_ROWS, kernels.DECODE_PARTITION

    def tensors(self) -> Dict[str, TensorSpec]:
        p = self.params
        t = {
            "uk": TensorSpec((p.num_heads * p.dim, p.kv_rank)),
            "uv": TensorSpec((self.out_size, p.kv_rank)),
            "o": TensorSpec((p.hidden_size, self.out_size)),
        }
        if p.q_rank > 0:
            t["dq"] = TensorSpec((p.q_rank, p.hidden_size))
            t["dq_norm"] = TensorSpec((p.q_rank,))
            t["uq"] = TensorSpec((self.q_size, p.q_rank))
        else:
            t["q"] = TensorSpec((self.q_size, p.hidden_size))
        if p.own_latent:
            t["dkv"] = TensorSpec((self.key_size, p.hidden_size))
            t["dkv_norm"] = TensorSpec((p.kv_rank,))
        if p.gate != "none":
            t["g"] = TensorSpec((self.gate_size, p.hidden_size))
        return t

    def _projected(self) -> list:
        p = self.params
        return ["dq" if p.q_rank > 0 else "q"] + (["dkv"] if p.own_latent else []) + (["g"] if p.gate != "none" else [])

    def fused(self) -> Dict[str, list]:
        return {"from_input": self._projected()}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p = self.params
        if "from_input" in tensors:
            self.w_proj = tensors["from_input"]
        else:
            ws = [tensors[n] for n in self._projected()]
            dt = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
            self.w_proj = torch.cat([w.to(dt) for w in ws], dim=0).contiguous()
        self.w_norm = tensors.get("dkv_norm")
        self.w_uq, self.w_dq_norm = tensors.get("uq"), tensors.get("dq_norm")
        if self.w_norm is not None and self.w_dq_norm is not None and self.w_norm.dtype != self.w_dq_norm.dtype:
            self.w_norm, self.w_dq_norm = self.w_norm.float(), self.w_dq_norm.float()
        # W_uk,h^T for every head: [heads, kv_rank, dim], the matrix the unrotated query part is multiplied by
        self.w_uk_t = tensors["uk"].view(p.num_heads, p.dim, p.kv_rank).transpose(1, 2).contiguous()
        self.w_uv = tensors["uv"].view(p.num_heads, p.vdim, p.kv_rank).contiguous()
        self.w_o = tensors["o"]

    def nbytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_proj, self.w_uq, self.w_uk_t, self.w_uv, self.w_o)
                   if w is not None)

    def forward(self, x, ctx, cache: Optional[LayerCache], state=None) -> torch.Tensor:
        p, rt = self.params, self.rt
        T = ctx.T
        ws = rt.workspace
        proj = ws.get("latent.proj", (rt.max_tokens, self.proj_size), rt.dtype)[:T]
        linear(x, self.w_proj, proj)
        op_mark(ctx, "q_dkv_proj", self.w_proj, T)
        g = ctx.groups[cache.group]
        k_cache = cache.tensors["k"]
        qa = ws.get("latent.qa", (rt.max_tokens, self.qa_size), rt.dtype)[:T]
        elem = proj.element_size()
        latent = proj[:, self.c_col:self.c_col + self.key_size] if p.own_latent and cache.write else None
        head = (p.num_heads, p.dim, p.rot_dim, p.kv_rank, self.rot_dims)
        cached = (g.slots if latent is not None else None, k_cache, rt.page_size, ctx.status, self.pairs)
        turn = None
        if p.q_rank > 0:
            # the latent into the cache beside the norm of the queries' latent; then the queries, whose rotated parts go along with the product below
            c_q = ws.get("latent.cq", (rt.max_tokens, p.q_rank), rt.dtype)[:T]
            kernels.latent_prep(None, latent, ctx.positions, T, *head, self.w_norm if latent is not None else None, p.eps,
                                self.cos, self.sin, None, *cached, dq=proj[:, :p.q_rank], dq_w=self.w_dq_norm, dq_out=c_q)
            op_mark(ctx, "latent_norm+rotate+write", nbytes=float(T * (2 * p.q_rank + 2 * self.key_size) * elem))
            q = ws.get("latent.q", (rt.max_tokens, self.q_size), rt.dtype)[:T]
            linear(c_q, self.w_uq, q)
            op_mark(ctx, "q_up_proj", self.w_uq, T)
            if p.rot_dim > 0:
                turn = (p.rot_dim, p.dim, p.kv_rank, self.cos, self.sin, ctx.positions, self.pairs, ctx.status)
        else:
            q = proj[:, :self.q_size]
            kernels.latent_prep(q, latent, ctx.positions, T, *head, self.w_norm, p.eps, self.cos, self.sin, qa, *cached)
            op_mark(ctx, "latent_norm+rotate+write", nbytes=float(T * (self.proj_size + 2 * self.key_size
                                                                       + p.num_heads * p.rot_dim) * elem))
        kernels.head_linear(q, 0, self.q_head, self.w_uk_t, qa, 0, self.key_size, tokens=T, turn=turn)
        op_mark(ctx, "q_absorb", nbytes=float(T * p.num_heads * (p.dim + p.kv_rank) * elem + self.w_uk_t.numel() * elem),
                flops=2.0 * T * p.num_heads * p.dim * p.kv_rank)
        gate = dict(gate=proj[:, self.g_col:], gate_mode=1) if p.gate == "head" else {}
        lat = ws.get("latent.out", (rt.max_tokens, self.lat_size), rt.dtype)[:T]
        v_stride = self.key_size if p.rot_dim > 0 else 0
        common = (p.num_heads, 1, self.key_size, p.kv_rank, 1, rt.page_size, p.window, 0, p.scale, 0.0, 0.0, 1.0, p.eps, False)
        if ctx.num_decode > 0:
            rows = ctx.max_items * p.num_heads * ctx.parts_capacity
            part_o = ws.get("mattn.part_o", (rows * p.kv_rank,), torch.float32)
            part_ml = ws.get("mattn.part_ml", (rows * 2,), torch.float32)
            kernels.maps_attn_decode(qa, self.qa_size, k_cache, k_cache, g.block_table, ctx.decode_info, part_o, part_ml,
                                     ctx.decode_parts, lat, ctx.num_decode, *common, v_stride=v_stride, **gate)
            self._mark(ctx, "attention_decode", "decode")
        if ctx.num_tiles > 0:
            kernels.maps_attn_prefill(qa, self.qa_size, k_cache, k_cache, g.block_table, ctx.tile_seq, ctx.tile_tok,
                                      ctx.tile_rows, ctx.positions, lat, ctx.num_tiles, kernels.PREFILL_TILE_ROWS,
                                      *common, v_stride=v_stride, **gate)
            self._mark(ctx, "attention_prefill", "prefill")
        heads_v = ws.get("latent.values", (rt.max_tokens, self.out_size), rt.dtype)[:T]
        kernels.head_linear(lat, 0, p.kv_rank, self.w_uv, heads_v, 0, p.vdim, tokens=T,
                            gate=proj[:, self.g_col:] if p.gate == "entry" else None)
        op_mark(ctx, "v_up", nbytes=float(T * p.num_heads * ((2 if p.gate == "entry" else 1) * p.vdim + p.kv_rank) * elem + self.w_uv.numel() * elem),
                flops=2.0 * T * p.num_heads * p.vdim * p.kv_rank)
        out = ws.get("mixer.out", (rt.max_tokens, p.hidden_size), rt.dtype)[:T]
        linear(heads_v, self.w_o, out)
        op_mark(ctx, "o_proj", self.w_o, T)
        return out

    def _mark(self, ctx, op: str, which: str) -> None:
        if ctx.profiler is None:
            return
        from ..engine.profiler import attention_work
        p = self.params
        elem = 2 if self.rt.dtype == torch.bfloat16 else 4
        nbytes, flops = attention_work(ctx.host, p.num_heads, 1, (self.key_size + p.kv_rank) // 2, p.window, elem)[which]
        ctx.profiler.mark(op, nbytes, flops)
