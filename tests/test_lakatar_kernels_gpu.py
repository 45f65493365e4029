"""The kernels added for Lakatar, one by one, against float64 restatements (tests/plain_lakatar.py and this file):
the recurrence with a decay per token and channel and with one decay per head (token by token and in blocks on
the tensor cores, cut into chunks, from a given state, heads finished by the kernel or behind it), the token
shift and its state, the norm after the sum, the latent's preparation with rotated neighbours and a latent of
the queries, groups of experts scored by their best choice score, the gated shared expert, and the fused forms
for a few rows (choice and grouping in one launch, gated experts, several products at once, the decays' second
product) and for the sum of terms that is normed."""

import math

import pytest
import torch

import plain_lakatar as P

pytestmark = pytest.mark.gpu

DEV = "cuda"


def rel(a, b):
    return float((a.double().cpu() - b.double().cpu()).abs().max() / (b.double().abs().max() + 1e-30))


def recurrence(q, k, v, S, decay=None, w=None, u=None):
    """q, k [T, H, D], v [T, H, DV], S [H, D, DV] in float64; one decay per head, or w [T, H, D] with u [H, D]."""
    S = S.clone()
    o = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=torch.float64)
    for t in range(q.shape[0]):
        kv = torch.einsum("hd,he->hde", k[t], v[t])
        if w is None:
            S = torch.tensor(decay, dtype=torch.float64)[:, None, None] * S + kv
            o[t] = torch.einsum("hde,hd->he", S, q[t])
        else:
            o[t] = torch.einsum("hde,hd->he", S + u[:, :, None] * kv, q[t])
            S = w[t][:, :, None] * S + kv
    return o, S


LENS, SLOTS = [200, 1, 77, 2, 16], [4, 0, 2, 5, 1]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,DV", [(3, 16, 32), (2, 64, 64), (1, 24, 40), (2, 10, 14), (1, 128, 144), (2, 32, 16), (1, 7, 5),
                                    (1, 256, 32)])
@pytest.mark.parametrize("channel", [False, True])
def test_recurrence(dtype, H, D, DV, channel):
    """Five sequences of unequal length in one launch, each from its own non-zero state in its own slot: serial and
    cut into chunks, token by token and in blocks; float32 sums and finished heads; other slots untouched."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(D * 7 + DV)
    T = sum(LENS)
    buf = (torch.randn(T, 2 * H * D + 2 * H * DV + 8, generator=g) * 0.5).to(dtype)
    state0 = torch.randn(7, H, D, DV, generator=g)
    z = torch.randn(T, H * D, generator=g) * 1.5 - 2.0
    bias, u = torch.randn(H * D, generator=g) * 0.5, torch.randn(H * D, generator=g)
    decay = torch.tensor([0.999, 0.6, 0.93][:H])
    nw = 1.0 + 0.2 * torch.randn(H * DV, generator=g)
    rot, base, scale, eps = (0 if channel else max(2, D // 4 * 2)), 50.0, 0.37, 1e-5
    if 2 * (rot // 2) > D:
        rot = 0
    pos = torch.cat([torch.arange(n) + 3 * i for i, n in enumerate(LENS)]).to(torch.int32)
    seq_of = torch.tensor(sum(([i] * n for i, n in enumerate(LENS)), []), dtype=torch.int32)
    q64, k64 = buf[:, :H * D].double().view(T, H, D), buf[:, H * D:2 * H * D].double().view(T, H, D)
    v64, g64 = buf[:, 2 * H * D:2 * H * D + H * DV].double().view(T, H, DV), buf[:, 2 * H * D + H * DV:2 * H * D + 2 * H * DV].double()
    if rot:
        spec = {"base": base, "dims": rot}
        q64, k64 = P.rotate_halves(q64, spec, pos.tolist()), P.rotate_halves(k64, spec, pos.tolist())
    k64 = k64 * scale
    w64 = torch.exp(-torch.exp(z.double() + bias.double())).view(T, H, D)
    want_o, want_S, at = [], {}, 0
    for n, s in zip(LENS, SLOTS):
        sl = slice(at, at + n)
        kw = dict(w=w64[sl], u=u.double().view(H, D)) if channel else dict(decay=decay.tolist())
        o, S = recurrence(q64[sl], k64[sl], v64[sl], state0[s].double(), **kw)
        want_o.append(o)
        want_S[s] = S
        at += n
    want_o = torch.cat(want_o)
    want_y = (P.unit(want_o, eps).reshape(T, H * DV) * nw.double() * P.silu(g64))
    dev = buf.to(DEV)
    q, k = dev[:, :H * D], dev[:, H * D:2 * H * D]
    v, gate = dev[:, 2 * H * D:2 * H * D + H * DV], dev[:, 2 * H * D + H * DV:2 * H * D + 2 * H * DV]
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    kw = dict(k_scale=scale, status=status)
    if rot:
        ang = torch.arange(300, dtype=torch.float64)[:, None] * torch.tensor(P.plain_frequencies(base, rot), dtype=torch.float64)
        kw.update(cos=torch.cos(ang).float().to(DEV), sin=torch.sin(ang).float().to(DEV), positions=pos.to(DEV))
    if channel:
        kw.update(decay_bias=bias.to(DEV), bonus=u.to(DEV))
    dec = z.to(DEV) if channel else decay.to(DEV)
    for chunked in (False, True):
        for longest in (0, max(LENS)):
            chunk, max_chunks = (32, (max(LENS) + 31) // 32) if chunked else (0, 1)
            if chunked:
                kw.update(chunk_state=torch.full((5 * max_chunks * H * D * DV,), float("nan"), device=DEV),
                          chunk_decay=torch.full((5 * max_chunks * H * D,), float("nan"), device=DEV))
            common = dict(chunk=chunk, max_chunks=max_chunks, longest=longest, **kw)
            state = state0.clone().to(DEV)
            out = torch.zeros(T, H * DV, device=DEV)
            kernels.linear_attention(q, k, v, seq_of.to(DEV), torch.tensor(SLOTS, dtype=torch.int32, device=DEV), dec, state,
                                     out, T, 5, H, D, DV, **common)
            blocks = longest > 0 and dtype == torch.bfloat16          # (high and low parts: some 2^-16 of the terms)
            tol = 2e-4 if blocks else 3e-5
            assert rel(out, want_o.reshape(T, H * DV)) < tol, (chunked, longest)
            for s in range(7):
                if s in want_S:
                    assert rel(state[s], want_S[s]) < tol, (chunked, longest, s)
                else:
                    assert torch.equal(state[s].cpu(), state0[s])
            ytol = 2e-2 if dtype == torch.bfloat16 else 5e-4
            state = state0.clone().to(DEV)
            y = torch.empty(T, H * DV, dtype=dtype, device=DEV)
            kernels.linear_attention(q, k, v, seq_of.to(DEV), torch.tensor(SLOTS, dtype=torch.int32, device=DEV), dec, state, out,
                                     T, 5, H, D, DV, y=y, gate=gate, gate_mode=kernels.GATE_SILU, norm_w=nw.to(DEV), eps=eps,
                                     **common)
            assert rel(y, want_y) < ytol, (chunked, longest)
            for s in want_S:
                assert rel(state[s], want_S[s]) < tol, (chunked, longest, s)
    assert int(status.item()) == 0


@pytest.mark.parametrize("longest", [0, 64])
def test_recurrence_with_extreme_decays(longest):
    """Channels that forget everything at once beside channels that forget nothing: no overflow, no division."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(5)
    T, D = 64, 32
    q, k, v = ((torch.randn(T, D, generator=g) * 0.5).to(torch.bfloat16) for _ in range(3))
    z = torch.full((T, D), -30.0)
    z[:, :8] = 6.0                               # exp(-exp(6)) = 0
    z[::7, 8:16] = 3.0                           # now and then
    z[5::9, 16:20] = 120.0                       # exp(120) is no float32
    u = torch.randn(D, generator=g)
    w = torch.exp(-torch.exp(z.double())).view(T, 1, D)
    want, S = recurrence(q.double().view(T, 1, D), k.double().view(T, 1, D), v.double().view(T, 1, D),
                         torch.zeros(1, D, D, dtype=torch.float64), w=w, u=u.double().view(1, D))
    state = torch.zeros(1, D * D, device=DEV)
    out = torch.empty(T, D, device=DEV)
    zero = torch.zeros(T, dtype=torch.int32, device=DEV)
    kernels.linear_attention(q.to(DEV), k.to(DEV), v.to(DEV), zero, zero[:1].clone(), z.to(DEV), state, out, T, 1, 1, D, D,
                             decay_bias=torch.zeros(D, device=DEV), bonus=u.to(DEV), longest=longest,
                             status=torch.zeros(1, dtype=torch.int32, device=DEV))
    assert rel(out, want.view(T, D)) < 2e-4 and rel(state.view(D, D), S[0]) < 2e-4


def test_recurrence_reports_a_position_beyond_its_tables():
    from redline_b200.ops import kernels
    for longest in (0, 20):
        x = torch.randn(20, 32, device=DEV).to(torch.bfloat16)
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        tab = torch.ones(10, 8, device=DEV)
        zero = torch.zeros(20, dtype=torch.int32, device=DEV)
        kernels.linear_attention(x, x, x, zero, zero[:1].clone(), torch.ones(1, device=DEV), torch.zeros(1, 32 * 32, device=DEV),
                                 torch.empty(20, 32, device=DEV), 20, 1, 1, 32, 32, cos=tab, sin=tab,
                                 positions=torch.arange(20, dtype=torch.int32, device=DEV), status=status, longest=longest)
        assert int(status.item()) == 2


@pytest.mark.parametrize("x_dtype,y_dtype", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("width", [64, 100, 37, 1280])
def test_token_shift(x_dtype, y_dtype, width):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(width)
    lens, slots, G = [5, 1, 1, 40, 2], [3, 1, 0, 5, 2], 5
    T = sum(lens)
    x = torch.randn(T, width, generator=g).to(x_dtype)
    mu = torch.rand(G, width, generator=g)
    state0 = torch.randn(7, width, generator=g)
    seq_of = torch.tensor(sum(([i] * n for i, n in enumerate(lens)), []), dtype=torch.int32, device=DEV)
    y = torch.full((G, T + 3, width), float("nan"), dtype=y_dtype, device=DEV)
    state = state0.clone().to(DEV)
    kernels.token_shift(x.to(DEV), mu.to(DEV), y, seq_of, torch.tensor(slots, dtype=torch.int32, device=DEV), state, T)
    at = 0
    for n, s in zip(lens, slots):
        prev = torch.cat([state0[s:s + 1].double(), x[at:at + n - 1].double()])
        for i in range(G):
            want = x[at:at + n].double() + (prev - x[at:at + n].double()) * mu[i].double()
            assert rel(y[i, at:at + n], want) < (1e-6 if y_dtype == torch.float32 else 1e-2)
        assert torch.equal(state[s].cpu(), x[at + n - 1].float())
        at += n
    assert torch.isnan(y[:, T:].float()).all()
    for s in set(range(7)) - set(slots):
        assert torch.equal(state[s].cpu(), state0[s])


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("width", [48, 101, 2048, 2500, 4100, 9000])
@pytest.mark.parametrize("scaled", [True, False])
def test_norm_after_the_sum(dtype, tol, width, scaled):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(width)
    T, alpha, eps = 9, 1.9, 1e-4
    res, d = torch.randn(T, width, generator=g) * 2, (torch.randn(T, width, generator=g)).to(dtype)
    w, sc = 1.0 + 0.3 * torch.randn(width, generator=g), 1.0 + 0.3 * torch.randn(width, generator=g)
    want = P.unit(alpha * res.double() + (sc.double() if scaled else 1.0) * d.double(), eps) * w.double()
    r, out = res.clone().to(DEV), torch.empty(T, width, dtype=dtype, device=DEV)
    kernels.sum_norm(r, d.to(DEV), w.to(DEV), sc.to(DEV) if scaled else None, alpha, eps, out)
    assert rel(r, want) < 2e-6 and rel(out, want) < tol
    r = res.clone().to(DEV)
    kernels.sum_norm(r, d.to(DEV), w.to(DEV), sc.to(DEV) if scaled else None, alpha, eps, None)
    assert rel(r, want) < 2e-6
    r = res.clone().to(DEV)
    kernels.sum_norm(r, None, None, None, alpha, eps, out)                 # only the copy
    assert torch.equal(r.cpu(), res) and torch.equal(out.cpu(), res.to(dtype))


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("H,dn,dr,rank,rot,qr", [(3, 16, 8, 24, 8, 40), (2, 10, 6, 20, 2, 17), (4, 32, 16, 64, 16, 96)])
def test_latent_prep_with_neighbours_and_a_latent_of_the_queries(dtype, tol, H, dn, dr, rank, rot, qr):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(H * rank)
    T, ps, eps = 21, 16, 1e-5
    key = rank + dr
    scaling = {"factor": 5.0, "original": 40, "fast": 8.0, "slow": 1.0}
    spec = {"base": 300.0, "dims": rot, "scaling": scaling}
    freq, mag = P.stretched_frequencies(300.0, rot, scaling)
    ang = torch.arange(200, dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)
    cos, sin = (torch.cos(ang) * mag).float().to(DEV), (torch.sin(ang) * mag).float().to(DEV)
    proj = torch.randn(T, qr + key + 3, generator=g).to(dtype)
    q = torch.randn(T, H * (dn + dr), generator=g).to(dtype)
    nw, qw = (1.0 + 0.2 * torch.randn(rank, generator=g)).to(dtype), (1.0 + 0.2 * torch.randn(qr, generator=g)).to(dtype)
    pos = torch.randint(0, 200, (T,), generator=g).to(torch.int32)
    slots = torch.randperm(5 * ps, generator=g)[:T].to(torch.int32)
    slots[4] = -1
    cache = torch.full((5, 1, ps, key), float("nan"), dtype=dtype, device=DEV)
    qa = torch.full((T, H * key), float("nan"), dtype=dtype, device=DEV)
    cq = torch.empty(T, qr, dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    dev = proj.to(DEV)
    kernels.latent_prep(None, dev[:, qr:qr + key], pos.to(DEV), T, H, dn, dr, rank, rot, nw.to(DEV), eps, cos, sin, None,
                        slots.to(DEV), cache, ps, status, True, dq=dev[:, :qr], dq_w=qw.to(DEV), dq_out=cq)
    kernels.latent_prep(q.to(DEV), None, pos.to(DEV), T, H, dn, dr, rank, rot, None, eps, cos, sin, qa, None, None, ps, status, True)
    assert int(status.item()) == 0
    p64 = proj.double()
    assert rel(cq, P.unit(p64[:, :qr], eps) * qw.double()) < tol
    c = P.unit(p64[:, qr:qr + rank], eps) * nw.double()
    kr = P.rotate_pairs(p64[:, qr + rank:qr + key], spec, pos.tolist())
    flat = cache.view(5 * ps, key)
    rq = P.rotate_pairs(q.double().view(T, H, dn + dr)[:, :, dn:], spec, pos.tolist())
    for t in range(T):
        if int(slots[t]) >= 0:
            assert rel(flat[int(slots[t])], torch.cat([c[t], kr[t]])) < tol
    got = qa.view(T, H, key)
    assert rel(got[:, :, rank:], rq) < tol and torch.isnan(got[:, :, :rank].float()).all()
    # the same parts beside the per-head product that fills the rest, on both of its kernels
    w = torch.randn(H, rank, dn, generator=g).to(dtype)
    want = torch.einsum("hrd,thd->thr", w.double(), q.double().view(T, H, dn + dr)[:, :, :dn])
    for impl in (0, 1, 2):
        both = torch.full((T, H * key), float("nan"), dtype=dtype, device=DEV)
        kernels.head_linear(q.to(DEV), 0, dn + dr, w.to(DEV), both, 0, key, impl=impl,
                            turn=(dr, dn, rank, cos, sin, pos.to(DEV), True, status))
        assert rel(both.view(T, H, key)[:, :, :rank], want) < tol
        assert torch.equal(both.view(T, H, key)[:, :, rank:], got[:, :, rank:])
        few = torch.full((9, H * key), float("nan"), dtype=dtype, device=DEV)
        kernels.head_linear(q[:9].to(DEV), 0, dn + dr, w.to(DEV), few, 0, key, impl=impl,
                            turn=(dr, dn, rank, cos, sin, pos[:9].to(DEV), True, status))
        assert rel(few.view(9, H, key)[:, :, :rank], want[:9]) < tol
        assert torch.equal(few.view(9, H, key)[:, :, rank:], got[:9, :, rank:])
    assert int(status.item()) == 0
    # another layer's rows are attended over: only the queries' latent is normed, nothing is written
    before = cache.clone()
    cq.zero_()
    kernels.latent_prep(None, None, pos.to(DEV), T, H, dn, dr, rank, rot, None, eps, cos, sin, None, None, cache, ps, status, True,
                        dq=dev[:, :qr], dq_w=qw.to(DEV), dq_out=cq)
    assert rel(cq, P.unit(p64[:, :qr], eps) * qw.double()) < tol
    assert torch.equal(before.nan_to_num(7.0), cache.nan_to_num(7.0))


def test_groups_are_scored_by_their_best_choice_score():
    """The correction decides which groups stay; a group none of whose choice scores is positive may stay, and the
    weights are the scores without the correction."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(3)
    for n, count, keep, top, scale, shift in ((12, 3, 1, 2, 1.5, 0.0), (16, 4, 2, 5, 0.7, -1.0), (6, 6, 3, 3, 1.0, -2.0), (8, 1, 1, 4, 2.0, 0.0)):
        T = 64
        z = torch.randn(T, n, generator=g) * 2
        corr = 0.3 * torch.randn(n, generator=g) + shift
        router = {"top": top, "groups": {"count": count, "keep": keep}}
        s = torch.softmax(z.double(), dim=-1)
        pick = P.choose(s, corr.double(), router)
        # close calls aside
        ch = s + corr.double()
        srt = ch.sort(-1).values
        best = ch.view(T, count, n // count).max(-1).values.sort(-1).values
        calm = (srt[:, 1:] - srt[:, :-1]).min(-1).values > 1e-5
        calm &= (best[:, 1:] - best[:, :-1]).min(-1).values > 1e-5 if count > 1 else calm
        choice = torch.empty(T * top, dtype=torch.int32, device=DEV)
        weight = torch.empty(T * top, device=DEV)
        wide = torch.randn(T, n + 2, generator=g)
        wide[:, :n] = z
        kernels.moe_route(wide.to(DEV)[:, :n], None, choice, weight, T, count, keep, 1, top, softmax=True,
                          choice_bias=corr.to(DEV), weight_scale=scale)
        got = choice.view(T, top).cpu().long()
        assert calm.sum() > T // 2
        assert torch.equal(got[calm].sort(-1).values, pick[calm].sort(-1).values)
        assert rel(weight.view(T, top)[calm.to(DEV)], (torch.gather(s, 1, got) * scale)[calm]) < 1e-5


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-6), (torch.bfloat16, 1e-2)])
def test_a_gated_shared_expert_in_the_weighted_sum(dtype, tol):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(9)
    T, top, W = 7, 3, 300
    y, sh = torch.randn(T * top, W, generator=g).to(dtype), torch.randn(T, W, generator=g).to(dtype)
    weight, logits = torch.rand(T * top, generator=g), torch.randn(T, 5, generator=g) * 3
    out = torch.empty(T, W, dtype=dtype, device=DEV)
    kernels.moe_combine(y.to(DEV), weight.to(DEV), sh.to(DEV), out, T, top, shared_gate=logits.to(DEV)[:, 4])
    want = (weight.double().view(T, top, 1) * y.double().view(T, top, W)).sum(1) + P.sigmoid(logits[:, 4:].double()) * sh.double()
    assert rel(out, want) < tol


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("width,top,gated", [(96, 2, True), (101, 3, True), (2048, 4, False), (4100, 1, None)])
def test_norm_after_a_sum_of_terms(dtype, tol, width, top, gated):
    """The routed experts' weighted sum formed by the kernel that norms (gated None: no shared expert)."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(width + top)
    T, alpha, eps = 6, 1.3, 1e-5
    res = torch.randn(T, width, generator=g)
    y, sh = torch.randn(T * top, width, generator=g).to(dtype), torch.randn(T, width, generator=g).to(dtype)
    weight, logits = torch.rand(T * top, generator=g), torch.randn(T, 4, generator=g) * 2
    w, sc = 1.0 + 0.3 * torch.randn(width, generator=g), 1.0 + 0.3 * torch.randn(width, generator=g)
    d = (weight.double().view(T, top, 1) * y.double().view(T, top, width)).sum(1)
    if gated is not None:
        d = d + (P.sigmoid(logits[:, 2:3].double()) if gated else 1.0) * sh.double()
    want = P.unit(alpha * res.double() + sc.double() * d, eps) * w.double()
    r, out = res.clone().to(DEV), torch.empty(T, width, dtype=dtype, device=DEV)
    kernels.sum_norm(r, y.to(DEV), w.to(DEV), sc.to(DEV), alpha, eps, out, top=top, mix_weight=weight.to(DEV),
                     shared=sh.to(DEV) if gated is not None else None, shared_gate=logits.to(DEV)[:, 2] if gated else None)
    assert rel(r, want) < 3e-6 and rel(out, want) < tol


@pytest.mark.parametrize("tokens,experts,count,keep,top", [(1, 12, 3, 1, 2), (7, 32, 4, 2, 4), (16, 100, 1, 1, 16), (5, 6, 6, 3, 3), (3, 1, 1, 1, 1)])
def test_choice_and_grouping_in_one_launch(tokens, experts, count, keep, top):
    """The same choice, weights, order and tiles as the two kernels that do it one after the other."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(tokens * experts)
    z = (torch.randn(tokens, experts + 1, generator=g) * 2).to(DEV)[:, :experts]
    corr = (torch.randn(experts, generator=g) * 0.3).to(DEV)
    pairs, cap = tokens * top, kernels.moe_max_tiles(tokens * top, experts)
    for tiled in (experts, max(experts - 2, 0)):
        got = []
        for fused in (False, True):
            i32 = lambda n: torch.full((n,), -7, dtype=torch.int32, device=DEV)  # noqa: E731
            choice, weight, lists = i32(pairs), torch.zeros(pairs, device=DEV), (i32(pairs), i32(cap), i32(cap), i32(cap), i32(4))
            how = dict(softmax=True, choice_bias=corr, weight_scale=1.5)
            if fused:
                kernels.moe_route_group(z, choice, weight, tokens, count, keep, 1, top, *lists, tiled=tiled, **how)
            else:
                kernels.moe_route(z, None, choice, weight, tokens, count, keep, 1, top, **how)
                kernels.moe_group(choice, pairs, experts, *lists, tiled=tiled)
            n = int(lists[4][0])
            got.append((choice, weight, lists[0], lists[1][:n], lists[2][:n], lists[3][:n]))
        for a, b in zip(*got):
            assert torch.equal(a, b)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("ff,width", [(24, 64), (17, 33), (704, 256)])
@pytest.mark.parametrize("act", ["silu", "clamped_swish"])
def test_gated_experts_of_a_few_pairs(dtype, tol, ff, width, act):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(ff)
    experts, tokens, top, limit, slope = 5, 6, 2, 1.2, 1.702
    x = torch.randn(tokens, width, generator=g).to(dtype)
    w = (torch.randn(experts, 2 * ff, width, generator=g) / math.sqrt(width)).to(dtype)
    choice = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).to(torch.int32).reshape(-1).to(DEV)
    pairs, cap = tokens * top, kernels.moe_max_tiles(tokens * top, experts)
    i32 = lambda n: torch.zeros(n, dtype=torch.int32, device=DEV)  # noqa: E731
    lists = (i32(pairs), i32(cap), i32(cap), i32(cap), i32(4))
    kernels.moe_group(choice, pairs, experts, *lists)
    out = torch.empty(pairs, ff, dtype=dtype, device=DEV)
    mode = kernels.ACT_CLAMPED_SWISH if act == "clamped_swish" else kernels.ACT_SILU
    kernels.moe_gemm(x.to(DEV), top, w.to(DEV).view(experts * 2 * ff, width), out, *lists, cap, act=mode, gated=True, limit=limit, slope=slope)
    for p in range(pairs):
        z = w[int(choice[p])].double() @ x[p // top].double()
        gate, up = z[:ff], z[ff:]
        if act == "silu":
            want = P.silu(gate) * up
        else:
            c = gate.clamp(max=limit)
            want = c * P.sigmoid(slope * c) * (up.clamp(-limit, limit) + 1.0)
        assert rel(out[p], want) < tol


@pytest.mark.parametrize("rows,n,groups,k", [(1, 64, 4, 96), (8, 48, 3, 256), (3, 2048, 4, 2048), (5, 16, 5, 136)])
def test_several_products_of_a_few_rows_in_one_launch(rows, n, groups, k):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(rows + n)
    x = torch.randn(groups, rows + 2, k, generator=g).to(torch.bfloat16).to(DEV)
    w = (torch.randn(groups * n, k, generator=g) / math.sqrt(k)).to(torch.bfloat16).to(DEV)
    y = torch.empty(rows, groups * n, dtype=torch.bfloat16, device=DEV)
    assert kernels.gemm_skinny_grouped_ok(rows, x, w, n)
    kernels.gemm_skinny_grouped(x, w, y, rows, n)
    for i in range(groups):
        want = x[i, :rows].double().cpu() @ w[i * n:(i + 1) * n].double().cpu().T
        assert rel(y[:, i * n:(i + 1) * n], want) < 1e-2
    assert not kernels.gemm_skinny_grouped_ok(9, x, w, n) and not kernels.gemm_skinny_grouped_ok(rows, x, w, n + 8)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,n,rank", [(1, 100, 5), (16, 257, 64), (9, 64, 24)])
def test_low_rank_second_product(dtype, rows, n, rank):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(n)
    x = torch.randn(rows, rank, generator=g)
    w = torch.randn(n, rank, generator=g).to(dtype)
    z = torch.empty(rows, n, device=DEV)
    kernels.low_rank(x.to(DEV), w.to(DEV), z, kernels.ACT_TANH)
    assert rel(z, torch.tanh(x.double()) @ w.double().T) < (2e-6 if dtype == torch.float32 else 5e-3)
    y = torch.empty(rows, rank, dtype=dtype, device=DEV)
    kernels.act_cast(x.to(DEV), y, kernels.ACT_TANH)
    assert rel(z, y.double().cpu() @ w.double().T) < 2e-6


@pytest.mark.parametrize("pairs,experts,tiled", [(5, 3, 3), (64, 12, 10), (1000, 7, 7), (4097, 130, 128), (20000, 256, 256), (9000, 2000, 2000)])
def test_grouping_of_many_pairs(pairs, experts, tiled):
    """Every expert's pairs in ascending order, one expert after another, in tiles of up to 64 (few experts chosen
    often, many never)."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(pairs)
    choice = (torch.rand(pairs, generator=g) ** 3 * experts).to(torch.int32).clamp(max=experts - 1)
    cap = kernels.moe_max_tiles(pairs, experts)
    i32 = lambda n: torch.full((n,), -7, dtype=torch.int32, device=DEV)  # noqa: E731
    order, te, tb, tr, meta = i32(pairs), i32(cap), i32(cap), i32(cap), i32(4)
    kernels.moe_group(choice.to(DEV), pairs, experts, order, te, tb, tr, meta, tiled=tiled)
    want = torch.sort(choice, stable=True).indices
    assert torch.equal(order.cpu().long(), want)
    tiles, at = [], 0
    for e, n in enumerate(torch.bincount(choice.long(), minlength=experts).tolist()):
        if e < tiled:
            tiles += [(e, at + r, min(64, n - r)) for r in range(0, n, 64)]
        at += n
    n = int(meta[0])
    assert n == len(tiles)
    assert [tuple(t) for t in torch.stack([te[:n], tb[:n], tr[:n]], 1).tolist()] == tiles
