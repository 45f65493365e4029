"""RWKV-style time mixing: a matrix state per head with a decay per token and key channel.

Every one of r, k, v, the gate g and the decay w reads its own mix of the token's row and the row of the token
before it in the sequence, m_s = h_t + (h_(t-1) - h_t) * mu_s (zeros before the first token).  r = W_r m_r,
k = W_k m_k, v = W_v m_v, gate = silu(W_g m_g) (heads x dim each); the decay is
a = exp(-exp(W_2 tanh(W_1 m_w) + w0)).  Per head, with a bonus u per key channel,

    o_t = S_(t-1)^T r_t + (sum_i r_i u_i k_i) v_t;      S_t = diag(a_t) S_(t-1) + k_t v_t^T

so the read-out sees the token's own write through the bonus only.  Every head's o is divided by its root mean
square, the joined heads multiplied by a weight and by the gate, then projected by W_o.

The per-request state is S (float32 [heads, dim, dim]) and the last row h (float32 [width]): two pools.  Where
the block's sublayers read the residual stream itself, the mixes are formed from its float32 rows
(``ctx.block_stream``).  Products of at most 8 rows run as one launch (groups of features with an input each).  The
decays' two products have float32 results; mixes, tanh, decays, the recurrence,
norm and gate are float32 (csrc/stream_ops.cu, csrc/linear_attention.cu).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict

import torch

from ..ops import kernels
from ..ops.linear import linear
from .base import Mixer, op_mark, register
from .linear_attention import run_recurrence
from .spec import StateSpec, TensorSpec

MIXES = ("r", "k", "v", "g", "w")


@dataclass(frozen=True)
class TimeMixParams:
    hidden_size: int
    num_heads: int
    dim: int                     # of a head's key and of its value
    decay_rank: int              # inner size of the decays' two products
    eps: float = 1e-6            # of the heads' norm


@register("mixer", "time_mix")
class TimeMix(Mixer):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = self.params
        if not 1 <= p.dim <= 256:
            raise ValueError(f"time_mix: the recurrence's kernels take head sizes up to 256; got {p.dim}")
        self.size = p.num_heads * p.dim

    def state_spec(self):
        p = self.params
        return (StateSpec((p.num_heads * p.dim * p.dim,), "float32"), StateSpec((p.hidden_size,), "float32"))

    def state_in_graphs(self) -> bool:
        return True

    def tensors(self) -> Dict[str, TensorSpec]:
        p = self.params
        W, n = p.hidden_size, self.size
        t = {f"mu_{s}": TensorSpec((W,)) for s in MIXES}
        t.update({s: TensorSpec((n, W)) for s in MIXES if s != "w"})
        t.update({"w1": TensorSpec((p.decay_rank, W)), "w2": TensorSpec((n, p.decay_rank)), "w0": TensorSpec((n,)),
                  "u": TensorSpec((p.num_heads, p.dim)), "norm": TensorSpec((n,)), "o": TensorSpec((W, n))})
        return t

    def fused(self) -> Dict[str, list]:
        return {"rkvgw": ["r", "k", "v", "g", "w1"], "mu": [f"mu_{s}" for s in MIXES]}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        def joined(name, members):
            if name in tensors:
                return tensors[name]
            ws = [tensors[m] for m in members]
            dt = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
            return torch.cat([w.to(dt) for w in ws], dim=0).contiguous()

        n = self.size
        self.w_in = joined("rkvgw", ["r", "k", "v", "g", "w1"])
        self.w_each = [self.w_in[i * n:(i + 1) * n] for i in range(4)] + [self.w_in[4 * n:]]
        self.mu = joined("mu", [f"mu_{s}" for s in MIXES]).float().view(len(MIXES), -1).contiguous()
        self.w_2, self.w_o = tensors["w2"], tensors["o"]
        self.w_0 = tensors["w0"].float().contiguous()
        self.u = tensors["u"].float().reshape(-1).contiguous()
        self.w_norm = tensors["norm"].float().contiguous()

    def nbytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_2, self.w_o))

    def forward(self, x, ctx, cache, state) -> torch.Tensor:
        p, rt = self.params, self.rt
        T, n = ctx.T, self.size
        ws = rt.workspace
        s_state, shift_state = state
        elem = x.element_size()
        stream = ctx.block_stream if ctx.block_stream is not None else x
        mixes = ws.get("tmix.mixes", (len(MIXES), rt.max_tokens, p.hidden_size), rt.dtype)
        kernels.token_shift(stream, self.mu, mixes, ctx.seq_of_token, ctx.state_slot, shift_state, T)
        op_mark(ctx, "token_shift", nbytes=T * p.hidden_size * (stream.element_size() + len(MIXES) * elem))
        w4 = self.w_in[:4 * n]
        if kernels.gemm_skinny_grouped_ok(T, mixes, w4, n):          # a few rows: the four products are one launch
            rkvg = ws.get("tmix.rkvg", (rt.max_tokens, 4 * n), rt.dtype)[:T]
            kernels.gemm_skinny_grouped(mixes, w4, rkvg, T, n)
            r, k, v, g = (rkvg[:, i * n:(i + 1) * n] for i in range(4))
        else:
            rkvg = ws.get("tmix.rkvg", (4, rt.max_tokens, n), rt.dtype)
            for i in range(4):
                linear(mixes[i, :T], self.w_each[i], rkvg[i, :T])
            r, k, v, g = (rkvg[i, :T] for i in range(4))
        low = ws.get("tmix.low", (rt.max_tokens, p.decay_rank), torch.float32)[:T]
        linear(mixes[4, :T], self.w_each[4], low)
        op_mark(ctx, "rkvgw_proj", self.w_in, T)
        z = ws.get("tmix.z", (rt.max_tokens, n), torch.float32)[:T]
        if T <= kernels.LOW_RANK_ROWS and p.decay_rank <= kernels.LOW_RANK_MAX:
            kernels.low_rank(low, self.w_2, z, kernels.ACT_TANH)
        else:
            inner = ws.get("tmix.inner", (rt.max_tokens, p.decay_rank), rt.dtype)[:T]
            kernels.act_cast(low, inner, kernels.ACT_TANH)
            linear(inner, self.w_2, z)
        op_mark(ctx, "decay_proj", self.w_2, T)
        y = ws.get("tmix.y", (rt.max_tokens, n), rt.dtype)[:T]
        run_recurrence(self, ctx, r, k, v, z, s_state, y, heads=p.num_heads, dim=p.dim, vdim=p.dim, decay_bias=self.w_0,
                       bonus=self.u, gate=g, gate_mode=kernels.GATE_SILU, norm_w=self.w_norm, eps=p.eps)
        op_mark(ctx, "time_mix", nbytes=T * n * (5.0 * elem + 4.0) + 8.0 * ctx.S * n * p.dim, flops=6.0 * T * n * p.dim)
        out = ws.get("mixer.out", (rt.max_tokens, p.hidden_size), rt.dtype)[:T]
        linear(y, self.w_o, out)
        op_mark(ctx, "o_proj", self.w_o, T)
        return out
