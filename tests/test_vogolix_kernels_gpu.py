"""The kernels added for Vogolix, one by one, against the float64 functions of tests/plain_vogolix.py: the
state-space recurrence (token by token and in blocks on the tensor cores, cut into chunks, from given states), the
norm in parts behind the gate, chunked and windowed attention with a sink over shuffled pages, biases, whole norms
and pair rotations of queries with and without keys, the convolution with a bias of its sums, per-head products with
a gate per entry, and the ReLU-gated products."""

import pytest
import torch

import plain_vogolix as P

pytestmark = pytest.mark.gpu

DEV = "cuda"


def rel(a, b):
    return float((a.double().cpu() - b.double().cpu()).abs().max() / (b.double().abs().max() + 1e-30))


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------------------- the state space

LENS, SLOTS = [200, 1, 77, 2, 64, 129], [4, 0, 2, 5, 1, 6]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,N,DV", [(4, 2, 16, 32), (2, 1, 64, 64), (3, 3, 24, 40), (2, 2, 10, 14), (2, 1, 128, 144),
                                      (6, 2, 48, 16), (1, 1, 7, 5), (1, 1, 256, 48), (8, 1, 80, 80)])
def test_recurrence(dtype, H, G, N, DV):
    """Six sequences of unequal length in one launch, each from its own non-zero state in its own slot, steps and
    decays between almost nothing and almost everything: serial and cut into chunks, token by token and in blocks;
    the other slots untouched."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(N * 7 + DV)
    T = sum(LENS)
    width = 2 * G * N + H * DV + H
    buf = torch.randn(T, width + 8, generator=g) * 0.5
    buf[:, 2 * G * N + H * DV:width] *= 4.0
    buf = buf.to(dtype)
    bias, a_log, skip = torch.randn(H, generator=g) - 1.5, torch.randn(H, generator=g), torch.randn(H, generator=g)
    a_log[0] = -4.0                                           # one head that hardly forgets
    state0 = torch.randn(8, H, N, DV, generator=g)
    seq_of = torch.tensor(sum(([i] * n for i, n in enumerate(LENS)), []), dtype=torch.int32, device=DEV)
    q64, k64 = buf[:, :G * N].double().view(T, G, N), buf[:, G * N:2 * G * N].double().view(T, G, N)
    v64 = buf[:, 2 * G * N:2 * G * N + H * DV].double().view(T, H, DV)
    dt = P.softplus(buf[:, 2 * G * N + H * DV:width].double() + bias.double())
    want_o, want_S, at = torch.zeros(T, H, DV, dtype=torch.float64), {}, 0
    for n, s in zip(LENS, SLOTS):
        sl = slice(at, at + n)
        want_S[s] = torch.zeros(H, N, DV, dtype=torch.float64)
        for h in range(H):
            want_o[sl, h], want_S[s][h] = P.state_space_recurrence(
                v64[sl, h], k64[sl, h // (H // G)], q64[sl, h // (H // G)], dt[sl, h], a_log[h].double(), skip[h].double(),
                state0[s, h].double())
        at += n
    want_o = want_o.reshape(T, H * DV)
    dev = buf.to(DEV)
    q, k, v = dev[:, :G * N], dev[:, G * N:2 * G * N], dev[:, 2 * G * N:2 * G * N + H * DV]
    z = dev[:, 2 * G * N + H * DV:width]
    for chunk in (0, 64, 96):
        for longest in (0, max(LENS)):
            chunks = (max(LENS) + chunk - 1) // chunk if chunk else 1
            kw = {}
            if chunk:
                kw = dict(chunk_state=torch.full((6 * chunks * H * N * DV,), float("nan"), device=DEV),
                          chunk_decay=torch.full((6 * chunks * H,), float("nan"), device=DEV))
            state = state0.clone().to(DEV)
            out = torch.full((T, H * DV), float("nan"), device=DEV)
            kernels.state_space(q, k, G, v, z, bias.to(DEV), a_log.to(DEV), skip.to(DEV), seq_of, i32(SLOTS), state, out, T, 6,
                                H, N, DV, chunk=chunk, max_chunks=chunks, longest=longest, **kw)
            blocks = longest > 0 and dtype == torch.bfloat16          # (high and low parts: some 2^-16 of the terms)
            tol = 2e-4 if blocks else 3e-5
            assert rel(out, want_o) < tol, (chunk, longest)
            for s in range(8):
                if s in want_S:
                    assert rel(state[s], want_S[s]) < tol, (chunk, longest, s)
                else:
                    assert torch.equal(state[s].cpu(), state0[s])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_recurrence_with_extreme_steps(dtype):
    """Steps that forget everything at once beside steps of nearly zero, in one sequence: nothing overflows, nothing of
    what was forgotten comes back, what was kept stays."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(5)
    T, H, N, DV = 300, 2, 32, 32
    q, k, v = (torch.randn(T, n, generator=g).to(dtype) for n in (N, N, H * DV))
    z = torch.where(torch.rand(T, H, generator=g) < 0.1, 60.0, -9.0).to(dtype)
    bias, a_log, skip = torch.zeros(H), torch.tensor([4.0, 0.0]), torch.zeros(H)
    dt = P.softplus(z.double())
    want = torch.stack([P.state_space_recurrence(v[:, h * DV:(h + 1) * DV].double(), k.double(), q.double(), dt[:, h],
                                                 a_log[h].double(), skip[h].double())[0] for h in range(H)], 1).reshape(T, -1)
    for longest in (0, T):
        for chunk in (0, 64):
            chunks = (T + 63) // 64 if chunk else 1
            kw = dict(chunk_state=torch.empty(chunks * H * N * DV, device=DEV), chunk_decay=torch.empty(chunks * H, device=DEV)) if chunk else {}
            out, state = torch.empty(T, H * DV, device=DEV), torch.zeros(1, H * N * DV, device=DEV)
            kernels.state_space(q.to(DEV), k.to(DEV), 1, v.to(DEV), z.to(DEV), bias.to(DEV), a_log.to(DEV), skip.to(DEV),
                                torch.zeros(T, dtype=torch.int32, device=DEV), i32([0]), state, out, T, 1, H, N, DV, chunk=chunk,
                                max_chunks=chunks, longest=longest, **kw)
            assert torch.isfinite(out).all() and rel(out, want) < 2e-4, (longest, chunk)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("n,groups", [(96, 3), (256, 1), (100, 4), (7, 7), (65, 5), (4096, 2), (6000, 1), (9000, 2)])
def test_norm_in_parts_behind_the_gate(dtype, tol, n, groups):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(n + groups)
    T = 11
    o = torch.randn(T, n, generator=g) * torch.linspace(0.1, 5.0, n)          # parts of different sizes
    z = (2 * torch.randn(T, n + 6, generator=g)).to(dtype)
    w = (1 + 0.2 * torch.randn(n, generator=g)).to(dtype)
    wide = torch.full((T, n + 4), float("nan"), dtype=dtype, device=DEV)
    for shift in (0, 3):                                                      # aligned rows and not
        kernels.group_gated_norm(o.to(DEV), z.to(DEV)[:, shift:shift + n], w.to(DEV), wide[:, shift:shift + n], groups, 1e-5)
        want = P.grouped_gated_norm(o.double(), z[:, shift:shift + n].double(), w.double(), groups, 1e-5)
        assert rel(wide[:, shift:shift + n], want) < tol
        wide.fill_(float("nan"))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,channels", [(1, 40), (3, 130), (4, 512), (8, 33)])
def test_convolution_with_a_bias_of_its_sums(taps, channels, dtype):
    """Portions of every length, single tokens between them; the slots keep the inputs as they came, without the bias."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(taps + channels)
    T = 70
    u = torch.randn(T, channels, generator=g).to(dtype)
    w, b = (0.5 * torch.randn(channels, taps, generator=g)).to(dtype), torch.randn(channels, generator=g)
    want = P.silu(P.causal_conv(u.double(), w.double(), b.double()))
    state = torch.zeros(3, max(taps - 1, 1) * channels, device=DEV)
    got, at = [], 0
    for n in [2, 1, 1, 9, 1, 2, 30, 1, 23]:
        x = u[at:at + n].to(DEV)
        y = torch.empty_like(x)
        kernels.short_conv(x, 0, w.to(DEV), None, y, 0, kernels.ACT_SILU, i32([0] * n), i32([1]), state, n, single=n == 1,
                           out_bias=b.to(DEV))
        got.append(y)
        at += n
    assert at == T and rel(torch.cat(got), want) < (1e-5 if dtype == torch.float32 else 1e-2)
    if taps > 1:
        assert torch.equal(state[1, :(taps - 1) * channels].view(taps - 1, channels).cpu(), u[T - taps + 1:].float())
    assert float(state[0].abs().max()) == 0.0 and float(state[2].abs().max()) == 0.0


# ---------------------------------------------------------------------------- attention

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,DV,kind,size,sink", [
    (4, 2, 16, 48, "chunk", 24, True), (4, 1, 80, 32, "chunk", 56, True), (2, 2, 96, 64, "chunk", 100, True),
    (3, 3, 20, 12, "chunk", 9, True), (2, 1, 7, 5, "chunk", 64, False), (2, 2, 32, 16, "chunk", 1, True),
    (2, 1, 48, 32, "chunk", 500, True), (2, 1, 32, 32, "chunk", 128, False), (4, 1, 48, 32, "window", 40, False),
    (3, 1, 26, 20, "window", 17, False), (2, 1, 64, 48, "window", 129, False)])
def test_chunks_and_windows_over_shuffled_pages(dtype, H, G, D, DV, kind, size, sink):
    """A portion of 150 tokens after 70 cached ones and, in the same cache, single tokens at contexts on both sides of
    page, chunk and partition borders; cache rows that no query may read hold NaN."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(H * D + DV + size)
    ps, L, p0, scale = 16, 220, 70, 0.3
    n = L - p0
    latent = kind == "window"                                # (values are the leading entries of the one key row)
    vs = D if latent else DV
    q, k = torch.randn(L, H, D, generator=g).to(dtype), torch.randn(L, G, D, generator=g).to(dtype)
    v = k[:, :, :DV] if latent else torch.randn(L, G, DV, generator=g).to(dtype)
    sk = torch.randn(H, generator=g)
    sk[0], sk[-1] = 6.0, -30.0
    seen = (P.chunk_mask if kind == "chunk" else P.window_mask)(L, size)
    pages = (L + ps - 1) // ps
    perm = (torch.randperm(pages + 3, generator=g) + 1)[:pages].to(torch.int32)
    kc = torch.full((pages + 4, G, ps, D), float("nan"), dtype=dtype)
    vc = torch.full((pages + 4, G, ps, DV), float("nan"), dtype=dtype)
    for j in range(L):
        if bool(seen[p0:, j].any()):
            kc[perm[j // ps], :, j % ps] = k[j]
            vc[perm[j // ps], :, j % ps] = v[j]
    kc = kc.to(DEV)
    vc = kc if latent else vc.to(DEV)
    table = torch.zeros(1, pages + 2, dtype=torch.int32)
    table[0, :pages] = perm
    table = table.to(DEV)
    want = torch.stack([P.masked_softmax((q[:, h].double() @ k[:, h // (H // G)].double().T) * scale, seen,
                                         sk[h].double() if sink else None) @ v[:, h // (H // G)].double()
                        for h in range(H)], 1)[p0:].reshape(n, H * DV)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    qd = q[p0:].reshape(n, -1).contiguous().to(DEV)
    mask = (size, 0) if kind == "window" else (0, 0)
    kw = dict(sink=sk.to(DEV) if sink else None, v_stride=vs if latent else 0, chunk=size if kind == "chunk" else 0)
    positions = torch.arange(p0, L, dtype=torch.int32, device=DEV)
    for impl in [1] + ([2] if dtype == torch.bfloat16 and D % 16 == 0 and DV % 16 == 0 else []):
        out = torch.full((n, H * DV), float("nan"), dtype=dtype, device=DEV)
        kernels.maps_attn_prefill(qd, H * D, kc, vc, table, i32([0, 0]), i32([0, 128]), i32([128, n - 128]), positions, out, 2,
                                  128, H, G, D, DV, 1, ps, *mask, scale, 0.0, 0.0, 1.0, 1e-5, False, impl=impl, **kw)
        assert rel(out, want) < tol, impl
    ends = sorted({p0 + 1, 112, 113, 127, 128, 129, 130, 192, 193, L} | {e for m in range(p0 + 2, L) if m % size == 0 for e in (m, m + 1)})
    rows = [e - 1 - p0 for e in ends]
    parts = (L + 127) // 128
    part_o = torch.full((len(ends) * H * parts * DV,), float("nan"), device=DEV)
    part_ml = torch.full((len(ends) * H * parts * 2,), float("nan"), device=DEV)
    out = torch.zeros((n, H * DV), dtype=dtype, device=DEV)
    kernels.maps_attn_decode(qd, H * D, kc, vc, table, i32([[r, 0, e, 0] for r, e in zip(rows, ends)]), part_o, part_ml, parts,
                             out, len(ends), H, G, D, DV, 1, ps, *mask, scale, 0.0, 0.0, 1.0, 1e-5, False, **kw)
    assert rel(out[rows], want[rows]) < tol


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("H,G,D,DV,rot,halves", [(4, 2, 16, 8, 8, False), (3, 1, 20, 12, 20, True), (8, 8, 64, 64, 2, False),
                                                 (2, 1, 7, 5, 6, False)])
def test_biases_whole_norms_and_rotations(dtype, tol, H, G, D, DV, rot, halves):
    """The kernel behind the projection with biases of queries, keys and values, keys and values into their caches; and
    the same over queries alone."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(H * D + rot)
    T, eps, base, ps, pages = 23, 1e-5, 300.0, 8, 9
    pos = torch.randperm(500, generator=g)[:T]
    qs, ks, vs = H * D, G * D, G * DV
    x = (2 * torch.randn(T, qs + ks + vs, generator=g)).to(dtype)
    b = torch.randn(qs + ks + vs, generator=g)
    wq, wk = (1 + 0.3 * torch.randn(qs, generator=g)).to(dtype), (1 + 0.3 * torch.randn(ks, generator=g)).to(dtype)
    spec = {"base": base, "dims": rot}
    turn = P.rotate_halves if halves else P.rotate_pairs
    xb = x.double() + b.double()
    want_q = turn(P.rms_norm(xb[:, :qs], wq.double(), eps).view(T, H, D), spec, pos.tolist()).reshape(T, -1)
    want_k = turn(P.rms_norm(xb[:, qs:qs + ks], wk.double(), eps).view(T, G, D), spec, pos.tolist()).reshape(T, -1)
    a = torch.arange(500, dtype=torch.float64)[:, None] * torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    cos, sin = torch.cos(a).float().to(DEV), torch.sin(a).float().to(DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    slots = torch.randperm(ps * pages, generator=g)[:T].to(torch.int32)
    slots[3] = -1
    kc = torch.full((pages, G, ps, D), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((pages, G, ps, DV), float("nan"), dtype=dtype, device=DEV)
    p32 = pos.to(torch.int32).to(DEV)
    xd = x.clone().to(DEV)
    kernels.head_prep(xd, p32, T, 0, H, qs, G, D, status, wq.to(DEV), wk.to(DEV), kernels.HEAD_NORM_WHOLE, eps, cos, sin, qs + ks,
                      vs, None, kernels.VALUE_MIX_NONE, 0.0, slots.to(DEV), kc, vc, ps, halves=halves, bias=b.to(DEV))
    assert rel(xd[:, :qs], want_q) < tol and rel(xd[:, qs:qs + ks], want_k) < tol
    for t in range(T):
        s = int(slots[t])
        if s >= 0:
            assert torch.equal(kc[s // ps, :, s % ps].reshape(-1), xd[t, qs:qs + ks])
            assert rel(vc[s // ps, :, s % ps].reshape(-1), xb[t, qs + ks:]) < tol
    # queries alone, in a buffer of their own: a gate's columns behind them stay as they are
    extra = torch.randn(T, 5, generator=g).to(dtype)
    xq = torch.cat([x[:, :qs], extra], 1).contiguous().to(DEV)
    kernels.head_prep(xq, p32, T, 0, H, qs, 0, D, status, wq.to(DEV), None, kernels.HEAD_NORM_WHOLE, eps, cos, sin, qs, 0, None,
                      kernels.VALUE_MIX_NONE, 0.0, None, kc, vc, ps, halves=halves, bias=b[:qs].contiguous().to(DEV))
    assert rel(xq[:, :qs], want_q) < tol and torch.equal(xq[:, qs:].cpu(), extra)
    assert int(status.item()) == 0


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("T,H,N,K", [(3, 4, 64, 96), (70, 3, 24, 40), (19, 2, 9, 20), (200, 1, 72, 64), (9, 5, 8, 16)])
def test_per_head_products_with_a_gate_per_entry(dtype, tol, T, H, N, K):
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(T + N)
    x = torch.randn(T, H * K, generator=g).to(dtype)
    w = (torch.randn(H, N, K, generator=g) / K ** 0.5).to(dtype)
    wide = (2 * torch.randn(T, H * N + 7, generator=g)).to(dtype)
    want = torch.einsum("thk,hnk->thn", x.double().view(T, H, K), w.double()).reshape(T, -1) * P.sigmoid(wide[:, 7:].double())
    for impl in (0, 1, 2):
        y = torch.full((T, H * N), float("nan"), dtype=dtype, device=DEV)
        kernels.head_linear(x.to(DEV), 0, K, w.to(DEV), y, 0, N, impl=impl, gate=wide.to(DEV)[:, 7:])
        assert rel(y, want) < tol, impl


# ---------------------------------------------------------------------------- the feed-forward

def test_relu_gated_products():
    """The activation kernel, the weight-streaming product and the tcgen05 product of every tiling."""
    from redline_b200.ops import kernels
    g = torch.Generator().manual_seed(2)
    for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 1e-2)):
        gu = (3 * torch.randn(9, 2 * 52, generator=g)).to(dtype).to(DEV)
        out = torch.empty(9, 52, dtype=dtype, device=DEV)
        kernels.gated_act(gu, out, kernels.ACTIVATIONS["relu"])
        assert rel(out, torch.relu(gu[:, :52].double()) * gu[:, 52:].double()) < tol
    for M, N, K in ((1, 48, 64), (8, 136, 256), (16, 72, 512), (130, 200, 128), (300, 512, 264)):
        x, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(2 * N, K, generator=g) / K ** 0.5).bfloat16()
        gu = (x.double() @ w.double().T).bfloat16().double()
        want = torch.relu(gu[:, :N]) * gu[:, N:]
        xd, wd = x.to(DEV), w.to(DEV)
        y = torch.full((M, N), float("nan"), dtype=torch.bfloat16, device=DEV)
        if M <= 16:
            kernels.gemm_skinny(wd, y, kernels.EPI_REGLU, M, x=xd)
            assert rel(y, want) < 2e-2
        else:
            for tile in (0, 128, 256, 512):
                y.fill_(float("nan"))
                kernels.gemm_tc(xd, wd, y, kernels.EPI_REGLU, tile_n=tile)
                assert rel(y, want) < 2e-2, tile
            assert int(kernels.tc_status(xd.device).item()) == 0
