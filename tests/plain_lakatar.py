"""A plain, slow implementation of the Lakatar decoder, one function per mechanism, in float64 on whole
sequences (every token sees the full score matrix, recurrences run token by token; no cache, no portions).  It
shares no code with the package: it reads the configuration dictionary itself, makes its own random weights and
writes and reads its own safetensors files.  The GPU tests hold the engine to it.

Notation.  A linear map W is stored [out, in] and applied as W x.  x_t is the residual stream at token t
(position t, counted from 0).  N(u; w) = u / sqrt(mean u^2 + eps) * (1 + w);  R(u) = u / sqrt(mean u^2 + eps).

    x_t = E[token_t]
    layer:  x <- N(a x + s1 * mixer(x); w1);   x <- N(a x + s2 * ff(x); w2)      (a: one constant, s1, s2: vectors)
    logits = W_head N(x; w_f)

    time mixing ("wkv", H heads of d):  with y the stream of the token before (zeros before the first), every
        one of r, k, v, g, w reads its own mix m_s = x + (y - x) * mu_s;  r = W_r m_r, k = W_k m_k, v = W_v m_v,
        gate = silu(W_g m_g);  decay = exp(-exp(W_2 tanh(W_1 m_w) + b)) per head and key channel.  Per head
            o_t = S^T r_t + v_t sum_i r_i u_i k_i;      S <- diag(decay_t) S + k_t v_t^T
        out = W_o (joined(R(o_h)) * n * gate).
    retention (H heads, keys of d, values of e):  q = W_q x, k = W_k x rotated (entry i with entry i + half of
        the first `dims`), k times d^(-1/2), v = W_v x;  S <- c_h S + k v^T, o = S^T q;  out =
        W_o (joined(R(o_h)) * silu(W_g x)).
    latent attention (H heads):  q = W_uq (R(W_dq x) * n_q), per head [n | r];  [c' | k_r] = W_dkv x,
        c = R(c') * n_c;  q_r and k_r rotated in neighbouring pairs with stretched frequencies (YaRN), k_r is one
        vector for all heads;  k_n = W_uk c, v = W_uv c;  s_ij = scale (q_n,i . k_n,j + q_r,i . k_r,j), j <= i;
        softmax;  head h's output times sigmoid(W_g x)_h;  W_o on the joined heads.  A layer may take c and k_r of
        an earlier layer instead of making its own.
    routed feed-forward:  z = W_r x, s = softmax(z);  choice scores s + correction;  a group of neighbouring
        experts is scored by its largest choice score, the best `keep` groups stay, the `top` largest choice
        scores within them are chosen with weights s * scale;  expert: W_d (silu(W_g x) * (W_u x));  the result is
        the weighted sum plus sigmoid(w_sg . x) times a shared expert of the same form.
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


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit(x, eps) * (1.0 + w)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


# ---------------------------------------------------------------------------------------- rotation

def plain_frequencies(base: float, dims: int) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def stretched_frequencies(base: float, dims: int, scaling: Optional[dict]) -> Tuple[List[float], float]:
    """-> (frequency per pair, factor on cos and sin)."""
    f = plain_frequencies(base, dims)
    if scaling is None:
        return f, 1.0

    def pair_at(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_at(scaling["fast"])), 0)
    hi = min(math.ceil(pair_at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def angles(freq: Sequence[float], positions: Sequence[int], like: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    a = torch.tensor(list(positions), dtype=torch.float64)[:, None] * torch.tensor(list(freq), dtype=torch.float64)[None, :]
    shape = [like.shape[0]] + [1] * (like.dim() - 2) + [len(freq)]
    return torch.cos(a).to(like.dtype).view(shape), torch.sin(a).to(like.dtype).view(shape)


def rotate_halves(x: torch.Tensor, rot: dict, positions: Sequence[int]) -> torch.Tensor:
    """x [T, ..., n]: the first rot.dims entries turned, entry i with entry i + dims/2; the rest unchanged."""
    dims = rot["dims"]
    half = dims // 2
    c, s = angles(plain_frequencies(rot["base"], dims), positions, x)
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def rotate_pairs(x: torch.Tensor, rot: dict, positions: Sequence[int]) -> torch.Tensor:
    """x [T, ..., n]: entries 2i and 2i + 1 of the first rot.dims turned."""
    dims = rot["dims"]
    freq, mag = stretched_frequencies(rot["base"], dims, rot.get("scaling"))
    c, s = angles(freq, positions, x)
    c, s = c * mag, s * mag
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ---------------------------------------------------------------------------------------- mixers

def shifted(x: torch.Tensor) -> torch.Tensor:
    return torch.cat([torch.zeros_like(x[:1]), x[:-1]])


def channel_decay_recurrence(r, k, v, w, u) -> torch.Tensor:
    """One head: r, k, w [T, d], v [T, e], u [d] -> o [T, e]."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = []
    for t in range(r.shape[0]):
        kv = torch.outer(k[t], v[t])
        out.append((S + u[:, None] * kv).T @ r[t])
        S = w[t][:, None] * S + kv
    return torch.stack(out)


def wkv(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = x.shape[0]
    H, d = m["heads"], m["dim"]
    before = shifted(x)
    mix = {s: stored(x + (before - x) * w[p + "mu." + s]) for s in "rkvgw"}
    r = stored(mix["r"] @ w[p + "r"].T).view(T, H, d)
    k = stored(mix["k"] @ w[p + "k"].T).view(T, H, d)
    v = stored(mix["v"] @ w[p + "v"].T).view(T, H, d)
    gate = silu(stored(mix["g"] @ w[p + "g"].T))
    inner = stored(torch.tanh(mix["w"] @ w[p + "w1"].T))
    decay = torch.exp(-torch.exp(inner @ w[p + "w2"].T + w[p + "w0"])).view(T, H, d)
    heads = [unit(channel_decay_recurrence(r[:, h], k[:, h], v[:, h], decay[:, h], w[p + "u"][h]), eps) for h in range(H)]
    y = stored(torch.cat(heads, dim=1) * w[p + "norm"] * gate)
    return stored(y @ w[p + "o"].T)


def scalar_decay_recurrence(q, k, v, c: float) -> torch.Tensor:
    """One head: q, k [T, d], v [T, e] -> o [T, e]; the read-out sees the token's own write."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = []
    for t in range(q.shape[0]):
        S = c * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def retention(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float,
              positions: Sequence[int]) -> torch.Tensor:
    T = x.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q = rotate_halves(stored(x @ w[p + "q"].T).view(T, H, d), m["rot"], positions)
    k = rotate_halves(stored(x @ w[p + "k"].T).view(T, H, d), m["rot"], positions) * d ** -0.5
    v = stored(x @ w[p + "v"].T).view(T, H, e)
    gate = silu(stored(x @ w[p + "g"].T))
    heads = [unit(scalar_decay_recurrence(q[:, h], k[:, h], v[:, h], m["decay"][h]), eps) for h in range(H)]
    return stored(stored(torch.cat(heads, dim=1) * gate) @ w[p + "o"].T)


def causal_softmax(s: torch.Tensor) -> torch.Tensor:
    """s [T, T]: row i over j <= i."""
    seen = torch.ones(s.shape, dtype=torch.bool).tril()
    s = s.masked_fill(~seen, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_of(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float,
              positions: Sequence[int]) -> Tuple[torch.Tensor, torch.Tensor]:
    """-> (latent c [T, kv_rank], rotated key part [T, rot_dim])."""
    raw = stored(x @ w[p + "dkv"].T)
    c = stored(unit(raw[:, :m["kv_rank"]], eps) * w[p + "dkv.norm"])
    return c, stored(rotate_pairs(raw[:, m["kv_rank"]:], m["rot"], positions))


def latent_attention(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float,
                     positions: Sequence[int], latent: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    T = x.shape[0]
    H, dn, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = latent
    cq = stored(unit(stored(x @ w[p + "dq"].T), eps) * w[p + "dq.norm"])
    q = stored(cq @ w[p + "uq"].T).view(T, H, dn + dr)
    qn, qr = q[:, :, :dn], stored(rotate_pairs(q[:, :, dn:], m["rot"], positions))
    kn = stored(c @ w[p + "uk"].T).view(T, H, dn)
    v = stored(c @ w[p + "uv"].T).view(T, H, dv)
    gate = sigmoid(stored(x @ w[p + "g"].T))
    out = torch.zeros(T, H, dv, dtype=x.dtype)
    for h in range(H):
        s = (qn[:, h] @ kn[:, h].T + qr[:, h] @ kr.T) * m["scale"]
        out[:, h] = (causal_softmax(s) @ v[:, h]) * gate[:, h:h + 1]
    return stored(stored(out.reshape(T, H * dv)) @ w[p + "o"].T)


# ---------------------------------------------------------------------------------------- feed-forward

def expert(x: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return stored(stored(silu(stored(x @ gate.T)) * stored(x @ up.T)) @ down.T)


def choose(s: torch.Tensor, correction: torch.Tensor, router: dict) -> torch.Tensor:
    """s [T, n] scores -> chosen experts [T, top]."""
    choice = s + correction
    T, n = choice.shape
    g = router.get("groups")
    if g is not None:
        per = n // g["count"]
        best = choice.view(T, g["count"], per).max(-1).values
        kept = torch.topk(best, g["keep"], dim=-1).indices
        allowed = torch.zeros(T, g["count"], dtype=torch.bool).scatter_(1, kept, True)
        choice = choice.masked_fill(~allowed.repeat_interleave(per, dim=1), -math.inf)
    return torch.topk(choice, router["top"], dim=-1).indices


def routed_ff(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str, f: dict) -> torch.Tensor:
    r = f["router"]
    s = torch.softmax(x @ w[p + "router"].T, dim=-1)
    pick = choose(s, w[p + "correction"], r)
    weight = torch.gather(s, 1, pick) * r["scale"]
    out = torch.zeros_like(x)
    for e in range(r["experts"]):
        hit = pick == e
        rows = hit.any(-1).nonzero().flatten()
        if rows.numel():
            y = expert(x[rows], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
            out[rows] += (weight[rows] * hit[rows]).sum(-1, keepdim=True) * y
    if f.get("shared") is not None:
        y = expert(x, w[p + "shared.gate"], w[p + "shared.up"], w[p + "shared.down"])
        out = out + sigmoid(x @ w[p + "shared.sg"].T) * y
    return stored(out)


def summed_norm(x, y, alpha: float, scale, norm, eps: float) -> torch.Tensor:
    return zero_centred_norm(alpha * x + scale * y, norm, eps)


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[list] = None,
            first_pos: int = 0) -> torch.Tensor:
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in w.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    positions = [first_pos + t for t in range(len(tokens))]
    x = w["embed"][list(tokens)].clone()
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m, kind = layer["mixer"], layer["type"]
        h = x if kind == "wkv" else stored(x)                # (the shift mixes the stream itself)
        if kind == "wkv":
            y = wkv(h, w, p + "mix.", m, eps)
        elif kind == "retention":
            y = retention(h, w, p + "mix.", m, eps, positions)
        elif kind == "latent_attention":
            src = m.get("kv_from")
            latents[i] = latent_of(h, w, p + "mix.", m, eps, positions) if src is None else latents[src]
            y = latent_attention(h, w, p + "mix.", m, eps, positions, latents[i])
        else:
            raise ValueError(kind)
        x = summed_norm(x, y, alpha, w[p + "ls1"], w[p + "norm1"], eps)
        f = layer.get("mlp")
        if f is not None:
            x = summed_norm(x, routed_ff(stored(x), w, p + "mlp.", f), alpha, w[p + "ls2"], w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return stored(zero_centred_norm(x, w["final.norm"], eps)) @ w["head"].T


# ---------------------------------------------------------------------------------------- files and weights

def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W = cfg["width"]
    out: Dict[str, tuple] = {"embed": (cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        H, q = m["heads"], p + "mix."
        out[p + "norm1"] = out[p + "ls1"] = (W,)
        if layer["type"] == "wkv":
            n, rank = H * m["dim"], m["decay_rank"]
            for s in "rkvgw":
                out[q + "mu." + s] = (W,)
            for s in "rkvg":
                out[q + s] = (n, W)
            out[q + "w1"], out[q + "w2"], out[q + "w0"] = (rank, W), (n, rank), (n,)
            out[q + "u"], out[q + "norm"], out[q + "o"] = (H, m["dim"]), (n,), (W, n)
        elif layer["type"] == "retention":
            out[q + "q"] = out[q + "k"] = (H * m["dim"], W)
            out[q + "v"] = out[q + "g"] = (H * m["vdim"], W)
            out[q + "o"] = (W, H * m["vdim"])
        else:
            out[q + "dq"], out[q + "dq.norm"] = (m["q_rank"], W), (m["q_rank"],)
            out[q + "uq"] = (H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            if m.get("kv_from") is None:
                out[q + "dkv"], out[q + "dkv.norm"] = (m["kv_rank"] + m["rot_dim"], W), (m["kv_rank"],)
            out[q + "uk"], out[q + "uv"] = (H * m["dim"], m["kv_rank"]), (H * m["vdim"], m["kv_rank"])
            out[q + "g"], out[q + "o"] = (H, W), (W, H * m["vdim"])
        f = layer.get("mlp")
        if f is None:
            continue
        out[p + "norm2"] = out[p + "ls2"] = (W,)
        experts = {f"e{e}": f["expert"]["ff"] for e in range(f["router"]["experts"])}
        if f.get("shared") is not None:
            experts["shared"] = f["shared"]["ff"]
            out[p + "mlp.shared.sg"] = (1, W)
        for name, ff in experts.items():
            out[f"{p}mlp.{name}.gate"] = out[f"{p}mlp.{name}.up"] = (ff, W)
            out[f"{p}mlp.{name}.down"] = (W, ff)
        out[p + "mlp.router"], out[p + "mlp.correction"] = (f["router"]["experts"], W), (f["router"]["experts"],)
    out["final.norm"], out["head"] = (W,), (cfg["vocab"], W)
    return out


def random_weights(cfg: dict, seed: int, sharpen: float = 2.0) -> Dict[str, torch.Tensor]:
    """Seeded weights as the float32 values that bfloat16 holds.  Matrices N(0, 1/fan_in) (what scores are made
    of times ``sharpen``, so that attention is not flat), the embedding N(0, 1), norm weights around their neutral
    value, decays between fast and slow, corrections small."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[1] if "." in name else name
        n = torch.randn(shape, generator=g)
        if name == "embed":
            t = n
        elif leaf.startswith("mix.mu."):
            t = 0.5 + 0.25 * n
        elif leaf == "mix.w0":
            t = -3.0 + 1.5 * n
        elif leaf == "mix.u":
            t = 0.5 * n
        elif leaf in ("ls1", "ls2"):
            t = 1.0 + 0.2 * n
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            t = 0.1 * n
        elif leaf == "mlp.correction":
            t = 0.05 * n
        elif len(shape) == 1:
            t = 1.0 + 0.1 * n
        else:
            t = n / math.sqrt(shape[1])
            if leaf in ("mix.uq", "mix.dkv", "mix.uk"):
                t = t * sharpen
            if leaf == "mlp.router":
                t = t * 2.0
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
