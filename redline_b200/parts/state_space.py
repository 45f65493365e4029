"""State-space layers (Mamba-2, "state-space duality").

W_in h is laid out as [z | x | B | C | d]: the gate and the values (heads x vdim each), B and C (groups x state each)
and one number per head.  x, B and C pass a short causal convolution over time per channel, with a bias, and SiLU.
With dt = softplus(d + dt_bias), and head h using the B and C of group h // (heads / groups), per head

    S_t = exp(-exp(A_log_h) dt_t) S_(t-1) + dt_t B_t x_t^T,        y_t = S_t^T C_t + D_h x_t

The joined heads are multiplied by silu(z), RMS-normed in ``norm_groups`` equal parts (each by its own root mean
square), times a weight, and projected by W_o.

The per-request state is S (float32 [heads, state, vdim]) and the convolution's last taps - 1 inputs (float32): two
pools, zero for a new request.  The recurrence is csrc/linear_attention.cu with a decay per token (B as its keys, C as
its queries); softplus, decays, the recurrence, its output, gate and norm are float32.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict

import torch

from ..ops import kernels
from ..ops.linear import linear
from .base import Mixer, op_mark, register
from .spec import StateSpec, TensorSpec


@dataclass(frozen=True)
class StateSpaceParams:
    hidden_size: int
    num_heads: int
    vdim: int                    # channels of a head
    state: int                   # state entries per channel
    groups: int = 1              # groups of B and C
    conv_taps: int = 4
    norm_groups: int = 1         # equal parts of the joined heads, normed one by one
    eps: float = 1e-6


@register("mixer", "state_space")
class StateSpace(Mixer):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = self.params
        if p.num_heads % p.groups != 0:
            raise ValueError(f"state_space: heads {p.num_heads} is no multiple of the groups {p.groups}")
        if not 1 <= p.state <= 256:
            raise ValueError(f"the recurrence's kernels take state sizes up to 256; got {p.state}")
        if not 1 <= p.conv_taps <= kernels.MAX_CONV_TAPS:
            raise ValueError(f"a short convolution has 1 to {kernels.MAX_CONV_TAPS} taps; got {p.conv_taps}")
        self.inner = p.num_heads * p.vdim
        if self.inner % p.norm_groups != 0:
            raise ValueError(f"state_space: {self.inner} entries do not form {p.norm_groups} equal parts")
        self.bc_size = p.groups * p.state
        self.conv_size = self.inner + 2 * self.bc_size
        self.proj_size = self.inner + self.conv_size + p.num_heads

    def state_spec(self):
        p = self.params
        s = StateSpec((p.num_heads * p.state * p.vdim,), "float32")
        if p.conv_taps > 1:
            return (s, StateSpec(((p.conv_taps - 1) * self.conv_size,), "float32"))
        return s

    def state_in_graphs(self) -> bool:
        return True

    def tensors(self) -> Dict[str, TensorSpec]:
        p = self.params
        return {
            "in": TensorSpec((self.proj_size, p.hidden_size)), "conv": TensorSpec((self.conv_size, p.conv_taps)),
            "conv_bias": TensorSpec((self.conv_size,)), "dt_bias": TensorSpec((p.num_heads,)),
            "A_log": TensorSpec((p.num_heads,)), "D": TensorSpec((p.num_heads,)), "norm": TensorSpec((self.inner,)),
            "o": TensorSpec((p.hidden_size, self.inner)),
        }

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_in, self.w_conv, self.w_norm, self.w_o = tensors["in"], tensors["conv"], tensors["norm"], tensors["o"]
        self.b_conv, self.dt_bias, self.a_log, self.d = (tensors[n].float().contiguous()
                                                         for n in ("conv_bias", "dt_bias", "A_log", "D"))

    def nbytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_conv, self.w_o))

    def forward(self, x, ctx, cache, state) -> torch.Tensor:
        p, rt = self.params, self.rt
        T = ctx.T
        ws = rt.workspace
        s_state, conv_state = state if isinstance(state, (tuple, list)) else (state, None)
        proj = ws.get("ssm.proj", (rt.max_tokens, self.proj_size), rt.dtype)[:T]
        linear(x, self.w_in, proj)
        op_mark(ctx, "zxbcdt_proj", self.w_in, T)
        conv = ws.get("ssm.conv", (rt.max_tokens, self.conv_size), rt.dtype)[:T]
        if conv_state is None:           # one tap: a weight and a bias per channel, nothing carried
            conv_state = ws.get("ssm.no_state", (rt.max_seqs + 1, 1), torch.float32)
        kernels.short_conv(proj, self.inner, self.w_conv, None, conv, 0, kernels.ACT_SILU, ctx.seq_of_token, ctx.state_slot,
                           conv_state, T, single=ctx.num_decode == ctx.S == T, out_bias=self.b_conv)
        op_mark(ctx, "conv+act", nbytes=2.0 * T * self.conv_size * proj.element_size())
        n, bc, H = self.inner, self.bc_size, p.num_heads
        o = ws.get("ssm.o", (rt.max_tokens, n), torch.float32)[:T]
        # (how a step is cut depends on its shape alone: single-token steps and full portions replay as graphs)
        longest = 1 if ctx.num_tiles == 0 else max(ctx.host.q_len)
        blocks = rt.dtype == torch.bfloat16 and p.state % 16 == 0 and p.vdim % 16 == 0
        chunk, max_chunks = kernels.state_space_chunks(longest, T, H, p.vdim, blocks)
        work = {}
        if max_chunks > 1:
            work = dict(chunk_state=ws.get("lin.chunks", (ctx.S * max_chunks * H * p.state * p.vdim,), torch.float32),
                        chunk_decay=ws.get("lin.chunk_decay", (ctx.S * max_chunks * H,), torch.float32))
        kernels.state_space(conv[:, n + bc:], conv[:, n:n + bc], p.groups, conv[:, :n], proj[:, n + self.conv_size:],
                            self.dt_bias, self.a_log, self.d, ctx.seq_of_token, ctx.state_slot, s_state, o, T, ctx.S, H,
                            p.state, p.vdim, chunk=chunk, max_chunks=max_chunks, longest=longest, **work)
        op_mark(ctx, "state_space", nbytes=T * (self.conv_size * conv.element_size() + 4.0 * n) + 8.0 * ctx.S * n * p.state,
                flops=4.0 * T * n * p.state)
        y = ws.get("ssm.y", (rt.max_tokens, n), rt.dtype)[:T]
        kernels.group_gated_norm(o, proj[:, :n], self.w_norm, y, p.norm_groups, p.eps, rows=T)
        op_mark(ctx, "gate+group_norm", nbytes=T * n * (4.0 + 2.0 * y.element_size()))
        out = ws.get("mixer.out", (rt.max_tokens, p.hidden_size), rt.dtype)[:T]
        linear(y, self.w_o, out)
        op_mark(ctx, "o_proj", self.w_o, T)
        return out
