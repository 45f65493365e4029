"""Linear attention with a decaying state per head ("lightning" attention, retention).

q = f(W_q h), k = f(W_k h) (heads x dim), v = f(W_v h) (heads x vdim), f an activation (SiLU, or none); per head
S_t = decay_h S_(t-1) + k_t v_t^T and o_t = S_t^T q_t.  Then either the joined heads are RMS-normed with a
weight (``head_norm`` False), or every head's o is divided by its root mean square (``head_norm`` True, no
weight); the result is multiplied by sigmoid(W_g h) or silu(W_g h) and projected by W_o.  q and k may be rotated
by their positions (a ``rope_halves`` encoding) and k scaled: both happen in float32 inside the recurrence's
kernel.  The state S (float32, [heads, dim, vdim]) is this mixer's per-request state: zero for a new request,
carried from step to step in the request's slot; there is no cache of keys.  q, k, v and g come from one fused
projection [q | k | v | g]; the recurrence (csrc/linear_attention.cu), its output and the norm are float32.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Tuple

import torch

from ..ops import kernels
from ..ops.linear import linear
from .base import Mixer, build_part, op_mark, register
from .spec import PartSpec, StateSpec, TensorSpec


@dataclass(frozen=True)
class LinearAttentionParams:
    hidden_size: int
    num_heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]       # one per head
    eps: float = 1e-6
    activation: str = "silu"       # of q, k and v ("none": as projected)
    gated: bool = True             # multiply the normed output by gate_activation(W_g h)
    gate_activation: str = "sigmoid"       # or "silu"
    head_norm: bool = False        # every head divided by its root mean square instead of the joined norm
    k_scale: float = 1.0           # factor on k
    position: Optional[PartSpec] = None    # a ``rope_halves`` encoding of q and k


def run_recurrence(part, ctx, q, k, v, decay, state, y, heads: int, dim: int, vdim: int, gate, gate_mode: int,
                   norm_w=None, eps: float = 0.0, finish: bool = True, **kw) -> Optional[torch.Tensor]:
    """The recurrence of csrc/linear_attention.cu over the step, cut into chunks where sequences are long.  With
    ``finish`` the heads are normed (per head), weighed and gated into ``y``; without, the float32 sums are
    returned."""
    rt, T = part.rt, ctx.T
    ws = rt.workspace
    # (how a step is cut depends on its shape alone: single-token steps and full portions replay as graphs)
    longest = 1 if ctx.num_tiles == 0 else max(ctx.host.q_len)
    chunk, max_chunks = kernels.linear_attention_chunks(longest, blocks=rt.dtype == torch.bfloat16 and dim % 16 == 0 and vdim % 16 == 0)
    if max_chunks > 1:
        kw["chunk_state"] = ws.get("lin.chunks", (ctx.S * max_chunks * heads * dim * vdim,), torch.float32)
        if kw.get("bonus") is not None:
            kw["chunk_decay"] = ws.get("lin.chunk_decay", (ctx.S * max_chunks * heads * dim,), torch.float32)
    kw.update(chunk=chunk, max_chunks=max_chunks, status=ctx.status, longest=longest)
    o = ws.get("lin.o", (rt.max_tokens, heads * vdim), torch.float32)[:T]
    if finish:
        kw.update(y=y, gate=gate, gate_mode=gate_mode, norm_w=norm_w, eps=eps)
    kernels.linear_attention(q, k, v, ctx.seq_of_token, ctx.state_slot, decay, state, o, T, ctx.S, heads, dim, vdim, **kw)
    return None if finish else o


@register("mixer", "linear_attention")
class LinearAttention(Mixer):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = self.params
        if len(p.decay) != p.num_heads:
            raise ValueError(f"linear attention of {p.num_heads} heads needs as many decays, got {len(p.decay)}")
        if not 1 <= p.dim <= 256:
            raise ValueError(f"linear attention kernels take key sizes up to 256; got {p.dim}")
        if not p.gated:
            raise ValueError("linear attention without an output gate is not built")
        if p.gate_activation not in ("sigmoid", "silu") or (p.gate_activation == "silu" and not p.head_norm):
            raise ValueError("linear attention: the gate is a sigmoid, or with head_norm also silu")
        self.gate_mode = kernels.GATE_SILU if p.gate_activation == "silu" else kernels.GATE_SIGMOID
        self.cos = self.sin = None
        if p.position is not None:
            pos = build_part("position", p.position, rt)
            if getattr(pos, "pairing", None) != "halves" or 2 * pos.rotary_tables()[0].shape[1] > p.dim:
                raise ValueError("linear attention rotates up to dim entries, entry i with entry i + half (rope_halves)")
            self.cos, self.sin = pos.rotary_tables()
        self.qk_size = p.num_heads * p.dim
        self.v_size = p.num_heads * p.vdim
        self.proj_size = 2 * self.qk_size + 2 * self.v_size
        self.decay = torch.tensor(p.decay, dtype=torch.float32, device=rt.device)
        self.act = kernels.ACTIVATIONS[p.activation]

    def state_spec(self) -> StateSpec:
        p = self.params
        return StateSpec((p.num_heads, p.dim, p.vdim), "float32")

    def state_in_graphs(self) -> bool:
        return True

    def tensors(self) -> Dict[str, TensorSpec]:
        p = self.params
        t = {
            "q": TensorSpec((self.qk_size, p.hidden_size)),
            "k": TensorSpec((self.qk_size, p.hidden_size)),
            "v": TensorSpec((self.v_size, p.hidden_size)),
            "g": TensorSpec((self.v_size, p.hidden_size)),
            "o": TensorSpec((p.hidden_size, self.v_size)),
        }
        if not p.head_norm:
            t["norm"] = TensorSpec((self.v_size,))
        return t

    def fused(self) -> Dict[str, list]:
        return {"qkvg": ["q", "k", "v", "g"]}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        if "qkvg" in tensors:
            self.w_in = tensors["qkvg"]
        else:
            ws = [tensors[n] for n in ("q", "k", "v", "g")]
            dt = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
            self.w_in = torch.cat([w.to(dt) for w in ws], dim=0).contiguous()
        self.w_o = tensors["o"]
        self.w_norm = tensors.get("norm")

    def nbytes(self) -> int:
        return self.w_in.numel() * self.w_in.element_size() + self.w_o.numel() * self.w_o.element_size()

    def forward(self, x, ctx, cache, state) -> torch.Tensor:
        p, rt = self.params, self.rt
        T = ctx.T
        ws = rt.workspace
        proj = ws.get("lin.proj", (rt.max_tokens, self.proj_size), rt.dtype)[:T]
        linear(x, self.w_in, proj)
        if self.act != kernels.ACT_NONE:
            kernels.bias_act(proj, None, self.act, cols=2 * self.qk_size + self.v_size)
        op_mark(ctx, "qkvg_proj", self.w_in, T)
        n = self.qk_size
        q, k, v, g = proj[:, :n], proj[:, n:2 * n], proj[:, 2 * n:2 * n + self.v_size], proj[:, 2 * n + self.v_size:]
        y = ws.get("lin.y", (rt.max_tokens, self.v_size), rt.dtype)[:T]
        rotation = dict(cos=self.cos, sin=self.sin, positions=ctx.positions) if self.cos is not None else {}
        o = run_recurrence(self, ctx, q, k, v, self.decay, state, y, heads=p.num_heads, dim=p.dim, vdim=p.vdim, gate=g,
                           gate_mode=self.gate_mode, eps=p.eps, finish=p.head_norm, k_scale=p.k_scale, **rotation)
        nbytes = T * (self.proj_size * proj.element_size() + 4.0 * self.v_size) + 8.0 * ctx.S * n * p.vdim
        op_mark(ctx, "linear_attention", nbytes=nbytes,
                flops=4.0 * T * p.num_heads * p.dim * p.vdim)
        if not p.head_norm:
            kernels.gated_rmsnorm(o, g, self.w_norm, y, p.eps, rows=T)
        out = ws.get("mixer.out", (rt.max_tokens, p.hidden_size), rt.dtype)[:T]
        linear(y, self.w_o, out)
        op_mark(ctx, "o_proj", self.w_o, T)
        return out
