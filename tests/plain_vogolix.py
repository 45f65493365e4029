"""A plain, slow implementation of the Vogolix decoder, one function per mechanism, in float64 on whole
sequences (every token sees the full score matrix, recurrences run token by token; no cache, no portions).  It
shares no code with the package: it reads the configuration dictionary itself, makes its own random weights and
writes and reads its own safetensors files.  The GPU tests hold the engine to it.

Notation.  A linear map W is stored [out, in] and applied as W x.  x_t is the residual stream at token t
(position t, counted from 0).  N(u; w) = u / sqrt(mean u^2 + eps) * w.

    x_t = E[token_t]
    layer:  x <- x + mixer(N(x; w1));   x <- x + ff(N(x; w2))      (or no feed-forward)
    logits = c W_head N(x; w_f)                                     (c: one constant)

    state space ("mamba2", H heads of e channels, N state entries, G groups, taps, n norm groups; h the input):
        W_in h = [z | u | d],  u of H e + 2 G N channels;  u_t <- silu(sum_j w_j u_(t - taps + 1 + j) + b), zeros
        before the first token;  u = [x | B | C];  dt = softplus(d + dt_bias).  Head h reads group h // (H / G):
            S_t = exp(-exp(A_h) dt) S_(t-1) + dt B x^T,      y_t = S_t^T C + D_h x
        The joined heads times silu(z) are normed in n equal parts, times a weight; then W_o.
    latent attention (H heads):  q = W_q h, per head [q_n | q_r];  [c' | k_r] = W_dkv h, c = N(c'; w_c);  q_r and
        k_r turn by position (entry i with entry i + half), k_r is one vector for all heads;  k_n = W_uk c,
        v = W_uv c;  s_ij = scale (q_n,i . k_n,j + q_r,i . k_r,j) over 0 <= i - j < window;  softmax;  the joined
        heads times sigmoid(W_g h), entry by entry;  W_o.
    attention (H query heads, G key heads):  q, k, v = W h + b;  q and k normed over all their rows at once, then
        the first `dims` entries of every head turn in neighbouring pairs;  s_ij = scale q_i . k_j over j <= i in
        the same chunk of positions, i // size = j // size;  the softmax's denominator also holds exp(sink_h);
        W_o.  A layer may use the keys and values of an earlier one.
    feed-forward:  W_d (relu(W_g h) * (W_u h)).
"""

from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

F64 = torch.float64
STORE_DTYPE: Optional[torch.dtype] = None     # set to torch.bfloat16: round what a 16-bit engine stores in 16 bits


def stored(x: torch.Tensor) -> torch.Tensor:
    if STORE_DTYPE is None:
        return x
    return x.to(STORE_DTYPE).to(F64)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ---------------------------------------------------------------------------------------- rotation

def angles(rot: dict, positions: Sequence[int], like: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """cos and sin [T, 1, ..., dims / 2] of p * base^(-2i/dims)."""
    freq = [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    a = torch.tensor(list(positions), dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)[None, :]
    shape = [like.shape[0]] + [1] * (like.dim() - 2) + [len(freq)]
    return torch.cos(a).to(like.dtype).view(shape), torch.sin(a).to(like.dtype).view(shape)


def rotate_halves(x: torch.Tensor, rot: dict, positions: Sequence[int]) -> torch.Tensor:
    """x [T, ..., n]: the first rot.dims entries turned, entry i with entry i + dims/2; the rest unchanged."""
    half, dims = rot["dims"] // 2, rot["dims"]
    c, s = angles(rot, positions, x)
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def rotate_pairs(x: torch.Tensor, rot: dict, positions: Sequence[int]) -> torch.Tensor:
    """x [T, ..., n]: entries 2i and 2i + 1 of the first rot.dims turned."""
    dims = rot["dims"]
    c, s = angles(rot, positions, x)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ---------------------------------------------------------------------------------------- the state space

def causal_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, channels], w [channels, taps] (the last column belongs to the current token), b [channels]."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps)) + b


def state_space_recurrence(x, B, C, dt, a_log, D, S: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """One head: x [T, e], B and C [T, N], dt [T], a_log and D numbers, S [N, e] -> (y [T, e], S after the last token)."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=x.dtype) if S is None else S
    out = []
    for t in range(x.shape[0]):
        S = torch.exp(-torch.exp(a_log) * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        out.append(S.T @ C[t] + D * x[t])
    return torch.stack(out), S


def grouped_gated_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """The gate first, then the norm of every one of ``groups`` equal parts by itself."""
    u = y * silu(z)
    parts = u.view(u.shape[0], groups, -1)
    return (parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)).reshape(u.shape) * w


def mamba2(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, e, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    proj = stored(h @ w[p + "in"].T)
    z, u, d = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    u = stored(silu(causal_conv(u, w[p + "conv"], w[p + "conv.b"])))
    x = u[:, :inner].view(T, H, e)
    B, C = u[:, inner:inner + G * N].view(T, G, N), u[:, inner + G * N:].view(T, G, N)
    dt = softplus(d + w[p + "dt_bias"])
    y = torch.stack([state_space_recurrence(x[:, i], B[:, i // (H // G)], C[:, i // (H // G)], dt[:, i],
                                            w[p + "A_log"][i], w[p + "D"][i])[0] for i in range(H)], dim=1)
    y = stored(grouped_gated_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps))
    return stored(y @ w[p + "o"].T)


# ---------------------------------------------------------------------------------------- attention

def window_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T]: row i sees the columns j with 0 <= i - j < size (None: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else torch.ones(T, T, dtype=torch.bool))


def chunk_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T]: row i sees the columns j <= i with floor(i / size) = floor(j / size)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i // size == j // size) if size else torch.ones(T, T, dtype=torch.bool))


def masked_softmax(s: torch.Tensor, seen: torch.Tensor, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """s [T, T]; with ``sink`` (a number) exp(sink) joins every row's denominator."""
    s = s.masked_fill(~seen, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return e / den


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float,
                     positions: Sequence[int]) -> torch.Tensor:
    T = h.shape[0]
    H, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = stored(h @ w[p + "q"].T).view(T, H, dn + dr)
    raw = stored(h @ w[p + "dkv"].T)
    c = stored(rms_norm(raw[:, :rank], w[p + "dkv.norm"], eps))
    kr = stored(rotate_halves(raw[:, rank:], m["rot"], positions))
    qn, qr = q[:, :, :dn], stored(rotate_halves(q[:, :, dn:], m["rot"], positions))
    kn = stored(c @ w[p + "uk"].T).view(T, H, dn)
    v = stored(c @ w[p + "uv"].T).view(T, H, dv)
    seen = window_mask(T, (m.get("mask") or {}).get("size"))
    out = torch.stack([masked_softmax((qn[:, i] @ kn[:, i].T + qr[:, i] @ kr.T) * m["scale"], seen) @ v[:, i]
                       for i in range(H)], dim=1).reshape(T, H * dv)
    return stored(stored(out * sigmoid(stored(h @ w[p + "g"].T))) @ w[p + "o"].T)


def keys_and_values(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float,
                    positions: Sequence[int]) -> Tuple[torch.Tensor, torch.Tensor]:
    """-> (k [T, G, dim] normed and rotated, v [T, G, vdim])."""
    T, G = h.shape[0], m["kv_heads"]
    k = stored(h @ w[p + "k"].T + w[p + "k.b"])
    k = rms_norm(k, w[p + "k.norm"], eps).view(T, G, m["dim"])
    return stored(rotate_pairs(k, m["rot"], positions)), stored(h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, m["vdim"])


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, positions: Sequence[int],
              kv: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    k, v = kv
    q = rms_norm(stored(h @ w[p + "q"].T + w[p + "q.b"]), w[p + "q.norm"], eps).view(T, H, m["dim"])
    q = stored(rotate_pairs(q, m["rot"], positions))
    seen = chunk_mask(T, (m.get("mask") or {}).get("size"))
    out = torch.stack([masked_softmax((q[:, i] @ k[:, i // (H // G)].T) * m["scale"], seen, w[p + "sink"][i])
                       @ v[:, i // (H // G)] for i in range(H)], dim=1)
    return stored(stored(out.reshape(T, H * m["vdim"])) @ w[p + "o"].T)


# ---------------------------------------------------------------------------------------- the model

def relu_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    gate, up = stored(h @ w[p + "gate"].T), stored(h @ w[p + "up"].T)
    return stored(stored(torch.clamp(gate, min=0.0) * up) @ w[p + "down"].T)


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    positions = list(range(len(tokens)))
    x = w["embed"][list(tokens)].clone()
    kvs = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        q, m, kind = p + "mix.", layer["mixer"], layer["type"]
        h = stored(rms_norm(x, w[p + "norm1"], eps))
        if kind == "mamba2":
            y = mamba2(h, w, q, m, eps)
        elif kind == "latent_attention":
            y = latent_attention(h, w, q, m, eps, positions)
        elif kind == "attention":
            src = m.get("kv_from")
            kvs[i] = keys_and_values(h, w, q, m, eps, positions) if src is None else kvs[src]
            y = attention(h, w, q, m, eps, positions, kvs[i])
        else:
            raise ValueError(kind)
        x = x + y
        if layer.get("mlp") is not None:
            x = x + relu_ff(stored(rms_norm(x, w[p + "norm2"], eps)), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.clone())
    return (stored(rms_norm(x, w["final.norm"], eps)) @ w["head"].T) * cfg["logit_scale"]


# ---------------------------------------------------------------------------------------- files and weights

def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W = cfg["width"]
    out: Dict[str, tuple] = {"embed": (cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m, q = layer["mixer"], p + "mix."
        H = m["heads"]
        out[p + "norm1"] = (W,)
        if layer["type"] == "mamba2":
            inner, bc = H * m["vdim"], 2 * m["groups"] * m["state"]
            out[q + "in"] = (2 * inner + bc + H, W)
            out[q + "conv"], out[q + "conv.b"] = (inner + bc, m["conv"]), (inner + bc,)
            out[q + "dt_bias"] = out[q + "A_log"] = out[q + "D"] = (H,)
            out[q + "norm"], out[q + "o"] = (inner,), (W, inner)
        elif layer["type"] == "attention":
            nq, nk, nv = H * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            out[q + "q"], out[q + "q.b"], out[q + "q.norm"] = (nq, W), (nq,), (nq,)
            if m.get("kv_from") is None:
                out[q + "k"], out[q + "k.b"], out[q + "k.norm"] = (nk, W), (nk,), (nk,)
                out[q + "v"], out[q + "v.b"] = (nv, W), (nv,)
            out[q + "sink"], out[q + "o"] = (H,), (W, H * m["vdim"])
        else:
            out[q + "q"] = (H * (m["dim"] + m["rot_dim"]), W)
            out[q + "dkv"], out[q + "dkv.norm"] = (m["kv_rank"] + m["rot_dim"], W), (m["kv_rank"],)
            out[q + "uk"], out[q + "uv"] = (H * m["dim"], m["kv_rank"]), (H * m["vdim"], m["kv_rank"])
            out[q + "g"], out[q + "o"] = (H * m["vdim"], W), (W, H * m["vdim"])
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out[p + "norm2"] = (W,)
            out[p + "mlp.gate"] = out[p + "mlp.up"] = (ff, W)
            out[p + "mlp.down"] = (W, ff)
    out["final.norm"], out["head"] = (W,), (cfg["vocab"], W)
    return out


def random_weights(cfg: dict, seed: int, sharpen: float = 2.0) -> Dict[str, torch.Tensor]:
    """Seeded weights as the float32 values that bfloat16 holds.  Matrices N(0, 1/fan_in) (what the latent's scores
    are made of times ``sharpen``, and so the normed queries' weights, so that attention is not flat), the embedding
    N(0, 1), norm weights around 1, biases and sinks N(0, 1/4) and N(0, 1), steps and decays between fast and slow."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[1] if "." in name else name
        n = torch.randn(shape, generator=g)
        if name == "embed":
            t = n
        elif leaf in ("mix.q.b", "mix.k.b", "mix.v.b", "mix.conv.b"):
            t = 0.5 * n
        elif leaf == "mix.conv":
            t = n / math.sqrt(shape[1])
        elif leaf == "mix.dt_bias":
            t = -2.0 + n
        elif leaf == "mix.A_log":
            t = 0.5 + n
        elif leaf in ("mix.sink", "mix.D"):
            t = n
        elif len(shape) == 1:
            t = 1.0 + 0.1 * n
            if leaf == "mix.q.norm":
                t = t * sharpen
        else:
            t = n / math.sqrt(shape[1])
            if leaf in ("mix.dkv", "mix.uk"):
                t = t * sharpen
        out[name] = t.to(torch.bfloat16).float()
    return out


def write_model_dir(path: str, cfg: dict, weights: Dict[str, torch.Tensor], dtype=torch.bfloat16) -> None:
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, t in weights.items():
        t = t.to(dtype).contiguous()
        raw = t.view(torch.int16 if dtype == torch.bfloat16 else torch.int32).numpy().tobytes()
        header[name] = {"dtype": {torch.bfloat16: "BF16", torch.float32: "F32"}[dtype], "shape": list(t.shape),
                        "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        for b in blobs:
            f.write(b)


def read_model_dir(path: str):
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw = np.frombuffer(data[lo:hi], dtype={"BF16": np.uint16, "F32": np.float32, "I32": np.int32}[info["dtype"]])
        if info["dtype"] == "BF16":
            t = torch.from_numpy((raw.astype(np.uint32) << 16).view(np.float32).copy())
        else:
            t = torch.from_numpy(raw.copy())
        out[name] = t.view(info["shape"])
    return cfg, out
