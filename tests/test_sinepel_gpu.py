"""Sinepel on the GPU against the plain restatement (sinepel_plain.py): every kernel alone, prompts,
decoding, portions, batches, reuse of slots, chunk edges and far keys, long decoding, and generation
through the session, the command line and the server. Small random models; 32-bit sessions are held
to rounding error, bf16 sessions to bf16 rounding."""
import json
import subprocess
import threading
import urllib.request

import numpy as np
import pytest
import torch

import sinepel_plain as P

pytestmark = pytest.mark.gpu
TOL = {"f32": 2e-5, "b16": 3e-2}


@pytest.fixture(scope="module")
def dev():
    from ainfer_b200 import cuda_abi
    d = cuda_abi.Device(0)
    yield d
    d.close()


@pytest.fixture(scope="module")
def rt():
    from ainfer_b200 import runtime
    return runtime


def bf16(x):
    return torch.as_tensor(x).to(torch.bfloat16)


def bits(x):
    return bf16(x).contiguous().view(torch.int16).numpy()


def from_bits(a, shape):
    return torch.from_numpy(a.view(np.int16).copy()).view(torch.bfloat16).float().reshape(shape).numpy()


def f32(x):
    return np.ascontiguousarray(torch.as_tensor(x).float().numpy())


def ctrl(positions, tokens=None):
    c = np.zeros((len(positions), 4), np.int32)
    c[:, 1], c[:, 2] = positions, np.asarray(positions) + 1
    if tokens is not None:
        c[:, 0] = tokens
    return c


def close(got, want, tol):
    """Every element within tol of its own size plus the array's."""
    want = np.asarray(want, np.float64)
    err = (np.abs(np.asarray(got, np.float64) - want) / (np.abs(want) + np.sqrt((want ** 2).mean()) + 1e-30)).max()
    assert err < tol, err


# ------------------------------------------------------------------- kernels ---
@pytest.mark.parametrize("W,S", [(64, 4), (50, 3), (37, 1), (128, 2), (40, 5)])
def test_embedding_with_positions(dev, W, S):
    g = torch.Generator().manual_seed(W)
    V, Pn, tok, pos = 11, 9, [3, 0, 10, 7], [0, 8, 2, 5]
    e, p = bf16(torch.randn(V, W, generator=g)), bf16(torch.randn(Pn, W, generator=g))
    x = dev.zeros(4 * S * W * 4)
    dev.kernel("EmbedPosRows")(4, x, dev.upload(bits(e)), dev.upload(bits(p)), dev.upload(ctrl(pos, tok)), W, V, Pn, S, 2.5)
    want = (e[tok].float() * 2.5 + p[pos].float())[:, None, :].repeat(1, S, 1)
    assert np.array_equal(dev.download(x, (4, S, W), np.float32), want.numpy())


@pytest.mark.parametrize("out", ["f32", "b16"])
@pytest.mark.parametrize("W,S,per", [(64, 4, 1), (196, 4, 3), (50, 3, 2), (37, 1, 4), (36, 2, 8), (40, 5, 3)])
def test_stream_update_read_norm_and_shift(dev, W, S, per, out):
    """Three sequences in one pass: rows 0..4 start at position 0, 5..6 continue (even and odd position),
    7 is alone."""
    g = torch.Generator().manual_seed(W * S)
    pos, seq, first = [0, 1, 2, 3, 4, 7, 8, 6], [2, 2, 2, 2, 2, 0, 0, 1], [0, 0, 0, 0, 0, 5, 5, 7]
    R, eps = 8, 1e-3
    rn = lambda *s: torch.randn(*s, generator=g)   # noqa: E731
    x, y, mix, o, i, nw, sh, st = rn(R, S, W), rn(R, W), rn(S, S), rn(S), rn(S), rn(W), torch.rand(W, generator=g), rn(3, 2, W)
    xn = P.streams_write(x.double(), mix.double(), o.double(), y.double())
    h = P.rms(P.streams_read(xn, i.double()), eps, nw.double())
    want = h.clone()
    for r in range(R):
        prev = h[r - 1] if first[r] != r else (st[seq[r], (pos[r] - 1) & 1].double() if pos[r] else torch.zeros(W, dtype=torch.float64))
        want[r] = h[r] + (prev - h[r]) * sh.double()
    xo, pend, ho, ld = dev.zeros(R * S * W * 4), dev.zeros(3 * W * 4), dev.zeros(R * (W + 3) * 4), W + 3
    up = lambda t: dev.upload(f32(t))   # noqa: E731
    dx = up(x)
    k = dev.kernel("HyperNormRowsF32" if out == "f32" else "HyperNormRowsB16")
    ctl = [dev.upload(ctrl(pos)), dev.upload(np.int32(seq)), dev.upload(np.int32(first))]
    k(-(-R // per), dx, up(y), up(mix), up(o), xo, up(i), up(nw), up(sh), up(st), pend, *ctl, 0, ho, W, S, R, per, ld, eps)
    dev.sync()
    close(dev.download(xo, (R, S, W), np.float32), xn, 1e-5)
    raw = dev.download(ho, (R, ld), np.float32 if out == "f32" else np.uint16)
    got = raw[:, :W] if out == "f32" else from_bits(np.ascontiguousarray(raw[:, :W]), (R, W))
    close(got, want, 1e-5 if out == "f32" else 1e-2)
    pd = dev.download(pend, (3, W), np.float32)
    for r in (4, 6, 7):
        close(pd[seq[r]], h[r], 1e-5)
    # no pending update, chosen rows, plain sum of the streams
    idx = np.int32([6, 1])
    k(2, dx, 0, 0, 0, 0, 0, up(nw), 0, 0, 0, *ctl, dev.upload(idx), ho, W, S, 2, 1, ld, eps)
    dev.sync()
    raw = dev.download(ho, (2, ld), np.float32 if out == "f32" else np.uint16)
    got = raw[:, :W] if out == "f32" else from_bits(np.ascontiguousarray(raw[:, :W]), (2, W))
    close(got, P.rms(x.double().sum(1), eps, nw.double())[idx.tolist()], 1e-5 if out == "f32" else 1e-2)


@pytest.mark.parametrize("kind", ["f32", "b16"])
@pytest.mark.parametrize("taps,Qc,Kn,per", [(4, 24, 8, 1), (1, 300, 20, 3), (2, 16, 16, 2), (7, 20, 12, 5), (3, 1000, 40, 4), (4, 30, 5, 4)])
def test_short_convolution_over_rows(dev, taps, Qc, Kn, per, kind):
    """Two sequences in a pass, one from position 0 and one continuing; the pending rows are committed."""
    C, cap = Qc + Kn, 16
    g = torch.Generator().manual_seed(taps)
    full = [torch.randn(9, C, generator=g), torch.randn(21, C, generator=g)]
    cw = torch.randn(C, taps, generator=g)
    start, n = [0, 13], [9, 8]
    U = torch.cat([full[0], full[1][13:]])
    pos = list(range(9)) + list(range(13, 21))
    seq, first = [0] * 9 + [1] * 8, [0] * 9 + [9] * 8
    st = torch.zeros(2, taps, C)
    for p in range(max(0, 13 - taps), 13):
        st[1, p % taps] = full[1][p]
    dst, pend = dev.upload(f32(st)), dev.zeros(2 * taps * C * 4)
    q, kc = dev.zeros(17 * Qc * 4), dev.zeros(2 * cap * Kn * 4)
    ctl = [dev.upload(ctrl(pos)), dev.upload(np.int32(seq)), dev.upload(np.int32(first))]
    dev.kernel("ShortConvRowsF32" if kind == "f32" else "ShortConvRowsB16")(
        -(-17 // per) * (-(-C // (1024 if C % 4 == 0 and Qc % 4 == 0 and 2 <= taps <= 4 else 256))), dev.upload(f32(U)), dev.upload(f32(cw.T)), dst, pend, *ctl, q, kc, cap * Kn, 17, C, Qc, taps, cap, C, per)
    dev.sync()
    dt, tol = (np.float32, 1e-5) if kind == "f32" else (np.uint16, 1e-2)
    val = lambda a: a if kind == "f32" else from_bits(a, a.shape)   # noqa: E731
    gq, gk = val(dev.download(q, (17, Qc), dt)), val(dev.download(kc, (2, cap, Kn), dt))
    for s in range(2):
        y = P.short_conv(full[s].double(), cw.double())[start[s]:]
        rows = slice(9 * s, 9 * s + n[s])
        close(gq[rows], y[:, :Qc], tol)
        for i in range(n[s]):
            close(gk[s, (start[s] + i) % cap], y[i, Qc:], tol * 3)
    # commit: the ring then holds the last taps - 1 projections of each sequence
    rec = np.zeros(1, np.dtype([("a", "<u8"), ("b", "<u8"), ("c", "<u8"), ("d", "<u8"), ("C", "<i4"), ("taps", "<i4")]))
    W = 6
    psh, sh = dev.upload(np.arange(2 * W, dtype=np.float32)), dev.zeros(2 * 2 * W * 4)
    rec[0] = (psh, sh, pend, dst, C, taps)
    dev.kernel("SeqTailCommit")(17, dev.upload(rec.view(np.uint8)), *ctl, 1, 17, W, 0)
    dev.sync()
    ring, shift = dev.download(dst, (2, taps, C), np.float32), dev.download(sh, (2, 2, W), np.float32)
    for s, last in ((0, 8), (1, 20)):
        for i in range(taps - 1):
            assert np.array_equal(ring[s, (last - i) % taps], full[s][last - i].numpy())
        assert np.array_equal(shift[s, last & 1], np.arange(W) + W * s)


def _attn_case(T, H, G, D, chunk, seed, edge=None):
    """Queries, keys and head numbers; edge (i, j): row i's score for key j stands far out if it is seen."""
    g = torch.Generator().manual_seed(seed)
    q, k = torch.randn(T, H, D, generator=g), torch.randn(T, G, D, generator=g)
    if edge:
        for i, j in edge:
            k[j] *= 3.0
            for h in range(H):
                q[i, h] = k[j, h // (H // G)] * 2.0
    r1, r2, temp = torch.rand(H, generator=g), torch.rand(H, generator=g) * 3, 0.5 + torch.rand(H, generator=g)
    return bf16(q).float(), bf16(k).float(), r1, r2, temp


def _table(dev, r1, r2, n):
    lb = dev.zeros(len(r1) * n * 4)
    dev.kernel("LogDistanceTable")(4, lb, dev.upload(f32(r1)), dev.upload(f32(r2)), len(r1), n)
    return lb


def test_distance_table(dev):
    r1, r2 = torch.tensor([0.5, 2.0, 0.0]), torch.tensor([0.01, 3.0, 1.0])
    got = dev.download(_table(dev, r1, r2, 300), (3, 300), np.float32)
    want = P.log_distance(300, r1.double(), r2.double())[:, 299, :].flip(1)
    close(got, want, 1e-7)


ATTN = [(70, 4, 2, 16, 24, 128), (33, 3, 3, 20, 1, 64), (90, 8, 2, 64, 50, 128), (40, 5, 1, 33, 1000, 64), (150, 4, 4, 128, 64, 256),
        (140, 8, 1, 64, 37, 192), (200, 6, 2, 96, 130, 256), (300, 4, 2, 40, 64, 384), (260, 2, 1, 256, 200, 320), (129, 3, 1, 176, 128, 192),
        (130, 2, 2, 8, 65, 192)]


def _mma(base, D):
    return base + str(next(p for p in (32, 64, 96, 128, 192, 256) if D <= p))


@pytest.mark.parametrize("kind", ["f32", "b16", "mma"])
@pytest.mark.parametrize("T,H,G,D,chunk,cap", ATTN)
def test_chunk_attention_over_rows(dev, T, H, G, D, chunk, cap, kind):
    """Whole and from the middle (the first rows already in the cache)."""
    if kind == "mma" and D % 8:
        pytest.skip("head size for the CUDA-core form")
    edge = [(chunk - 1, 0), (chunk, chunk - 1), (2 * chunk, 2 * chunk - 1), (2 * chunk - 1, chunk)] if 2 * chunk < T else None
    q, k, r1, r2, temp = _attn_case(T, H, G, D, chunk, T, edge)
    want = P.shared_kv_attention(q.double(), k.double(), 0.25, temp.double(), r1.double(), r2.double(), chunk).reshape(T, H * D)
    conv = f32 if kind == "f32" else bits
    n = min(chunk, 512)
    lb = _table(dev, r1, r2, n)
    ring = torch.zeros(cap, G * D)
    assert T <= cap
    ring[:T] = k.reshape(T, G * D)
    dk = dev.upload(conv(ring))
    ldo = H * D + 8
    for start in (0, T // 3):
        R = T - start
        o = dev.zeros(R * ldo * 4)
        name, rows = {"f32": ("ChunkAttnRowsF32", 16), "b16": ("ChunkAttnRowsB16", 16), "mma": (_mma("ChunkAttnMma", D), 64)}[kind]
        dev.kernel(name)(
            -(-R // rows) * H, dev.upload(conv(q[start:].reshape(R, H * D))), dk, lb, dev.upload(f32(temp)), dev.upload(ctrl(range(start, T))), o, R, H,
            G, D, cap, chunk, n, ldo, 0.25)
        dev.sync()
        raw = dev.download(o, (R, ldo), np.float32 if kind == "f32" else np.uint16)[:, :H * D]
        got = raw if kind == "f32" else from_bits(np.ascontiguousarray(raw), (R, H * D))
        close(got, want[start:], 1e-5 if kind == "f32" else 3e-2)


@pytest.mark.parametrize("kind", ["f32", "b16", "mma"])
@pytest.mark.parametrize("H,G,D,chunk,taps,splits", [(16, 1, 96, 190, 3, 4), (4, 2, 192, 130, 4, 3), (4, 2, 256, 64, 2, 2), (4, 2, 16, 24, 3, 1), (6, 2, 20, 100, 1, 5), (8, 1, 64, 150, 4, 2), (3, 3, 33, 1, 2, 3),
                                                     (4, 4, 128, 90, 4, 8), (12, 2, 40, 200, 5, 16)])
def test_decode_attention_with_convolution(dev, H, G, D, chunk, taps, splits, kind):
    """Three sequences decode side by side from position 0, at different times, over several chunks; their
    key rings are shorter than the run."""
    if kind == "mma" and D % 8:
        pytest.skip("head size for the CUDA-core form")
    T, Q, K, C = 230, H * D, G * D, (H + G) * D
    cap, n = 256 if chunk > 100 else 128, min(chunk, 512)
    g = torch.Generator().manual_seed(D)
    u = torch.randn(3, T, C, generator=g)
    cw = torch.randn(C, taps, generator=g) * 0.6
    r1, r2, temp = torch.rand(H, generator=g), torch.rand(H, generator=g) * 3, 0.5 + torch.rand(H, generator=g)
    lag = [0, 17, 60]
    want = []
    for s in range(3):
        y = P.short_conv(u[s].double(), cw.double())
        if kind == "mma":       # this form's products take bf16 queries
            y[:, :Q] = bf16(y[:, :Q]).double()
        if kind != "f32":
            y[:, Q:] = bf16(y[:, Q:]).double()
        want.append(P.shared_kv_attention(y[:, :Q].reshape(T, H, D), y[:, Q:].reshape(T, G, D), 0.3, temp.double(), r1.double(), r2.double(),
                                          chunk).reshape(T, Q))
    lb = _table(dev, r1, r2, n)
    dcw, dtemp = dev.upload(f32(cw.T)), dev.upload(f32(temp))
    rng = np.random.default_rng(0)
    # slots hold leftovers of earlier sequences
    st = dev.upload(rng.standard_normal((3, taps, C)).astype(np.float32))
    kc = dev.upload(f32(torch.randn(3, cap, K, generator=g)) if kind == "f32" else bits(torch.randn(3, cap, K, generator=g)))
    part, cnt = dev.zeros(3 * splits * H * (D + 4) * 4), dev.zeros(3 * G * 4)
    o, du, dc = dev.zeros(3 * Q * 4), dev.zeros(3 * C * 4), dev.zeros(48)
    k = dev.kernel({"f32": "ChunkAttnStepF32", "b16": "ChunkAttnStepB16", "mma": _mma("ChunkAttnStepMma", D)}[kind])
    got = np.zeros((3, T, Q), np.float32)
    for t in range(T + 60):
        pos = [min(max(t - lag[s], 0), T - 1) for s in range(3)]
        dev.write(du, f32(torch.stack([u[s, pos[s]] for s in range(3)])))
        dev.write(dc, ctrl(pos))
        k(3 * G * splits, du, dcw, st, dc, kc, cap * K, lb, dtemp, part, cnt, o, 3, H, G, D, taps, cap, chunk, n, splits, C, Q, 0, 0.3)
        r = dev.download(o, (3, Q), np.float32)
        for s in range(3):
            got[s, pos[s]] = r[s]
    for s in range(3):
        close(got[s], want[s], 2e-5 if kind == "f32" else 2e-2)


ACTS = {0: lambda v, cap: v, 1: lambda v, cap: torch.relu(v) ** 2, 2: lambda v, cap: P.softcap(v, cap)}


@pytest.mark.parametrize("R,N,K,act", [(1, 5, 7, 0), (70, 130, 50, 1), (3, 64, 16, 2), (65, 1, 200, 0)])
def test_linear_rows_32bit(dev, R, N, K, act):
    g = torch.Generator().manual_seed(N)
    x, w, b = torch.randn(R, K, generator=g), bf16(torch.randn(N, K, generator=g)), torch.randn(N, generator=g)
    ldw = -(-K // 8) * 8
    wp = torch.zeros(N, ldw)
    wp[:, :K] = w.float()
    y = dev.zeros(R * (N + 2) * 4)
    dev.kernel("LinearRows")(-(-N // 64) * (-(-R // 64)), dev.upload(f32(x)), dev.upload(bits(wp)), dev.upload(f32(b)), y, R, N, K, K, ldw, N + 2,
                             act, 3.0)
    close(dev.download(y, (R, N + 2), np.float32)[:, :N], ACTS[act](x.double() @ w.double().T + b.double(), 3.0), 1e-5)


@pytest.mark.parametrize("R,N,K,nt,splits,act,out16", [
    (1, 5, 40, 16, 1, 0, 0), (17, 130, 200, 32, 1, 2, 0), (64, 256, 1024, 64, 4, 0, 0), (300, 384, 136, 128, 1, 1, 1), (520, 640, 512, 256, 1, 0, 0),
    (30, 100, 4096, 16, 8, 1, 1), (1000, 1536, 320, 256, 1, 1, 1), (129, 128, 64, 128, 1, 0, 0), (5, 300, 520, 16, 2, 0, 0), (100, 260, 2048, 128, 8, 2, 0),
    (33, 128, 72, 64, 2, 0, 1), (401, 200, 264, 176, 1, 1, 0), (97, 128, 64, 96, 1, 2, 1)])
def test_linear_tensor_cores(dev, R, N, K, nt, splits, act, out16):
    g = torch.Generator().manual_seed(R)
    x, w, b = bf16(torch.randn(R, K, generator=g)), bf16(torch.randn(N, K, generator=g)), torch.randn(N, generator=g)
    dx, dw = dev.upload(bits(x)), dev.upload(bits(w))
    tiles = -(-N // 128) * (-(-R // nt))
    y = dev.zeros(R * N * 4)
    k = dev.kernel("LinearTc" + (f"Split{splits}" if splits > 1 else ""))
    want = ACTS[act](x.double() @ w.double().T + b.double(), 3.0)
    for _ in range(2):
        k(tiles * splits if splits > 1 else min(tiles, 3), dev.tensor_map_bf16(dw, N, K, K, 128), dev.tensor_map_bf16(dx, R, K, K, nt), dev.upload(f32(b)), y,
          R, N, K, nt, N, act, out16, 3.0)
        dev.sync()
        raw = dev.download(y, (R, N), np.uint16 if out16 else np.float32)
        close(from_bits(raw, (R, N)) if out16 else raw, want, 2e-2 if out16 else 1e-5)


@pytest.mark.parametrize("N,K,rows_pb,act", [(7, 50, 3, 0), (64, 1000, 22, 1), (601, 256, 201, 2), (33, 4096, 11, 0), (9, 20000, 5, 0), (500, 2560, 250, 0),
                                             (3, 8, 1, 0)])
def test_decode_gemv(dev, N, K, rows_pb, act):
    g = torch.Generator().manual_seed(N)
    x, w, b = torch.randn(K, generator=g), bf16(torch.randn(N, K, generator=g)), torch.randn(N, generator=g)
    ldw = -(-K // 8) * 8
    wp = torch.zeros(N, ldw)
    wp[:, :K] = w.float()
    y = dev.zeros(N * 4)
    dev.kernel("StreamGemv")(-(-N // rows_pb), dev.upload(f32(x)), dev.upload(bits(wp)), dev.upload(f32(b)), y, N, K, ldw, rows_pb, act, 3.0)
    close(dev.download(y, N, np.float32), ACTS[act](w.double() @ x.double() + b.double(), 3.0), 1e-5)


@pytest.mark.parametrize("S,K,N,pos,shift", [(4, 64, 40, 0, True), (4, 200, 77, 5, True), (3, 50, 20, 6, True), (1, 37, 9, 3, True), (2, 96, 30, 4, False),
                                             (6, 48, 16, 1, True)])
def test_decode_gemv_from_streams(dev, S, K, N, pos, shift):
    g = torch.Generator().manual_seed(K)
    rn = lambda *s: torch.randn(*s, generator=g)   # noqa: E731
    x, y, mix, o, i, nw, sh, st, w, b = rn(S, K), rn(K), rn(S, S), rn(S), rn(S), rn(K), torch.rand(K, generator=g), rn(2, K), bf16(rn(N, K)), rn(N)
    ldw = -(-K // 8) * 8
    wp = torch.zeros(N, ldw)
    wp[:, :K] = w.float()
    d = lambda t: t.double()   # noqa: E731
    xn = P.streams_write(d(x)[None], d(mix), d(o), d(y)[None])
    h = P.rms(P.streams_read(xn, d(i)), 1e-3, d(nw))[0]
    hs = h + ((d(st)[(pos - 1) & 1] if pos else 0 * h) - h) * d(sh) if shift else h
    up = lambda t: dev.upload(f32(t))   # noqa: E731
    xo, out, dst = dev.zeros(S * K * 4), dev.zeros(N * 4), up(st)
    dev.kernel("HyperStreamGemv")(-(-N // 7), up(x), up(y), up(mix), up(o), xo, up(i), up(nw), up(sh) if shift else 0, dst, dev.upload(ctrl([pos])),
                                  dev.upload(bits(wp)), up(b), out, S, N, K, ldw, 7, 0, 1e-3, 0.0)
    close(dev.download(out, N, np.float32), hs @ d(w).T + d(b), 1e-5)
    close(dev.download(xo, (S, K), np.float32), xn[0], 1e-5)
    if shift:
        got = dev.download(dst, (2, K), np.float32)
        close(got[pos & 1], h, 1e-5)
        assert np.array_equal(got[(pos - 1) & 1], f32(st)[(pos - 1) & 1])


# -------------------------------------------------------------------- models ---
L = P.make_layer
MODELS = {
    "mixed": P.make_config(layers=[L(), L(heads=6, kv_heads=3, dim=20, conv=1, chunk=7, ff=None), L(heads=2, kv_heads=2, dim=48, conv=5, chunk=40, ff=33)]),
    "odd": P.make_config(width=50, vocab=77, streams=1, layers=[L(heads=3, kv_heads=1, dim=10, chunk=16, ff=21), L(heads=1, kv_heads=1, dim=9, ff=None)]),
    "many": P.make_config(width=72, vocab=130, streams=2, layers=[L(heads=20, kv_heads=1, dim=16, conv=3, chunk=30, ff=100),
                                                                  L(heads=34, kv_heads=2, dim=12, conv=6, chunk=55, ff=40)]),
    "wide": P.make_config(width=128, vocab=320, streams=4, eps=1e-3, embed_scale=0.5, cap=4.0,
                          layers=[L(heads=8, kv_heads=2, dim=32, conv=4, chunk=96, ff=512), L(heads=4, kv_heads=4, dim=64, conv=2, chunk=33, ff=256)]),
    "pairs": P.make_config(width=40, vocab=90, streams=6, layers=[L(heads=4, kv_heads=1, dim=24, conv=4, chunk=1000, ff=64),
                                                                   L(heads=4, kv_heads=2, dim=8, conv=3, chunk=1, ff=8)]),
}


@pytest.fixture(scope="module", params=sorted(MODELS))
def bundle(request, dev, rt, tmp_path_factory):
    c = MODELS[request.param]
    w = P.make_weights(c, sum(map(ord, request.param)))
    folder = str(tmp_path_factory.mktemp(request.param))
    P.write_model(folder, c, w)
    model = rt.Model(dev, folder)
    toks = [int(t) for t in np.random.default_rng(5).integers(0, c["vocab"], 130)]
    yield c, P.Plain(c, w), model, toks, P.Plain(c, w).forward(toks).numpy(), folder
    model.close()


def logit_err(got, want):
    d = got - want
    return np.sqrt((d * d).mean(-1)).max() / want.std()


@pytest.mark.parametrize("kind", ["f32", "b16"])
def test_prompt_decoding_and_portions(rt, bundle, kind):
    c, _, model, toks, want, _ = bundle
    T = len(toks)
    s = rt.Session(model, 200, rt.Session.F32 if kind == "f32" else 0)
    assert logit_err(s.prefill_logits(toks, range(T)), want) < TOL[kind]
    assert logit_err(s.prefill_logits(toks, [0, 3, 64, T - 1]), want[[0, 3, 64, T - 1]]) < TOL[kind]    # state from before is not read at position 0
    s.reset()
    got = []
    for i, t in enumerate(toks):
        s.step(t, i)
        got.append(s.logits())
    assert logit_err(np.stack(got), want) < TOL[kind]
    for sizes in ([2], [3, 2, 7], [17, 2, 1, 40, 5], [96, 2], [33]):
        s.reset()
        got, i, j = [], 0, 0
        while i < T:
            n = min(sizes[j % len(sizes)], T - i)
            if n == 1:
                s.step(toks[i], i)
                got.append(s.logits()[None])
            else:
                got.append(s.prefill_logits(toks[i:i + n], range(n), i))
            i, j = i + n, j + 1
        assert logit_err(np.concatenate(got), want) < TOL[kind], sizes
    # passes of few rows inside one call, then decoding
    s.prefill_rows(5)
    s.reset()
    s.prefill(toks[:77])
    got = []
    for i in range(77, T):
        s.step(toks[i], i)
        got.append(s.logits())
    assert logit_err(np.stack(got), want[77:]) < TOL[kind]
    s.close()


@pytest.mark.parametrize("kind", ["f32", "b16"])
def test_batch_of_unequal_sequences_and_reused_slots(rt, bundle, kind):
    """Three slots; sequences start at different steps, one slot is given to another sequence in the
    middle. Every sequence against the plain model alone."""
    c, plain, model, toks, _, _ = bundle
    seqs = [toks[:100], toks[30:], [(7 * t + 3) % c["vocab"] for t in toks[:60]], toks[50:90]]
    plan = [(0, 0, 0), (1, 1, 9), (2, 2, 0), (3, 2, 61)]        # (sequence, slot, first step)
    refs = [plain.forward(q).numpy() for q in seqs]
    bd = rt.BatchDecode(model, 3, 160, flags=rt.BatchDecode.F32 if kind == "f32" else 0)
    err = 0.0
    for step in range(110):
        tok, pos, who = [0, 1, 2], [0, 0, 0], [None] * 3
        for q, slot, s0 in plan:
            if s0 <= step < s0 + len(seqs[q]):
                tok[slot], pos[slot], who[slot] = seqs[q][step - s0], step - s0, q
        bd.set_inputs(tok, pos)
        bd.step()
        bd.dev.sync()
        lg = bd.read("logits", np.float32).reshape(3, -1)
        for slot in range(3):
            if who[slot] is not None:
                err = max(err, logit_err(lg[slot][None], refs[who[slot]][pos[slot]][None]) * refs[who[slot]][pos[slot]].std() / refs[who[slot]].std())
    assert err < TOL[kind]
    bd.close()


def test_sessions_do_not_leak_into_the_next_request(rt, bundle):
    c, _, model, toks, want, _ = bundle
    s = rt.Session(model, 200, rt.Session.F32)
    other = [(5 * t + 1) % c["vocab"] for t in toks]
    s.prefill(other)
    for i in range(3):
        s.step(other[i], 130 + i)
    a = s.prefill_logits(toks[:90], range(90))             # no reset: position 0 starts anew
    assert logit_err(a, want[:90]) < TOL["f32"]
    s.reset()
    b = s.prefill_logits(toks[:90], range(90))
    assert np.array_equal(a, b)
    s.close()


def test_greedy_generation_everywhere(rt, bundle):
    """Session loop (32-bit: the plain model's tokens), recorded per-layer lists, the command line, the
    server's worker, batched decode, and the folder converted to a container."""
    from ainfer_b200 import server
    c, plain, model, toks, _, folder = bundle
    prompt, n = toks[:21], 24
    want = plain.greedy(prompt, n)
    s = rt.Session(model, 96, rt.Session.F32)
    assert s.generate(prompt, n).tolist() == want
    s.reset()
    s.prefill(prompt[:-1])
    assert s.generate(prompt[-1:], n, start_pos=len(prompt) - 1).tolist() == want
    tok, _ = s.sample(0.7, top_k=1, rng=3)
    assert tok == int(s.logits().argmax())
    s.close()
    s = rt.Session(model, 96, rt.Session.F32 | rt.Session.PER_LAYER_LISTS)
    assert s.generate(prompt, n).tolist() == want
    s.close()
    eng = server.Engine(folder, 512, f32=True)
    assert eng.generate(prompt, n, {})[0] == want
    srv = server.serve(eng, server.IdTokenizer(eng.vocab), port=0)
    threading.Thread(target=srv.serve_forever, daemon=True).start()
    req = urllib.request.Request(f"http://127.0.0.1:{srv.server_address[1]}/v1/completions",
                                 data=json.dumps({"prompt": prompt, "max_tokens": n}).encode(), headers={"Content-Type": "application/json"})
    assert json.loads(urllib.request.urlopen(req, timeout=60).read())["choices"][0]["token_ids"] == want
    srv.shutdown()
    eng.close()
    for spec in (folder, folder + "/m.binfer"):
        if spec != folder:
            rt.from_safetensors(folder, json.dumps(c), spec)
        r = subprocess.run([rt.DECODE_EXE, spec, "0", str(n - 1), "--ids=" + ",".join(map(str, prompt)), "--dtype=float32", "--eos=-1"],
                           capture_output=True, text=True, timeout=120)
        assert r.returncode == 0, r.stderr
        line = [x for x in r.stdout.splitlines() if x.startswith("generated:")][0]
        assert [int(x) for x in line.split()[1:]] == want, spec


def test_residual_after_every_layer(rt, bundle):
    c, plain, model, toks, _, _ = bundle
    _, layers = plain.forward(toks[:60], want_layers=True)
    s = rt.Session(model, 96, rt.Session.F32 | rt.Session.DIAG)
    s.prefill(toks[:50])
    for i in range(50, 60):
        s.step(toks[i], i)
        got = s.read("layer_out", np.float32).reshape(len(c["layers"]), -1)
        for L in range(len(c["layers"])):
            close(got[L], layers[L, i], 3e-5)
    s.close()


def test_bf16_generation_follows_the_plain_logits(rt, bundle):
    c, plain, model, toks, _, _ = bundle
    s = rt.Session(model, 96)
    got = s.generate(toks[:21], 24).tolist()
    s.close()
    ref = plain.forward(toks[:21] + got[:-1]).numpy()[20:]
    lost = [ref[i].max() - ref[i][g] for i, g in enumerate(got)]
    assert max(lost) < 6 * TOL["b16"] * ref.std()


def _trained_like(c, seed, far):
    """Weights in which attention dominates: one head's queries and keys follow a few embedding
    directions strongly, so that single keys stand out among hundreds."""
    w = P.make_weights(c, seed)
    for i, ly in enumerate(c["layers"]):
        w[f"l{i}.mix.temp"] = bf16(torch.full((ly["mixer"]["heads"],), far))
        w[f"l{i}.hc1.out"] = bf16(torch.full((c["streams"],), 1.0))
    return w


@pytest.mark.parametrize("kind", ["f32", "b16"])
def test_long_context_over_ring_ends(dev, rt, tmp_path, kind):
    """A context longer than the key ring holds (the ring takes one chunk and one pass of rows), peaked
    scores, chunk edges inside passes, in prompts and in decoding."""
    c = P.make_config(width=32, vocab=64, streams=2, max_positions=4096, layers=[L(heads=2, kv_heads=1, dim=16, conv=4, chunk=150, ff=48),
                                                                               L(heads=2, kv_heads=2, dim=8, conv=2, chunk=500, ff=None)])
    w = _trained_like(c, 9, 4.0)
    P.write_model(str(tmp_path), c, w)
    T = 2900
    toks = [int(t) for t in np.random.default_rng(1).integers(0, 64, T)]
    want = P.Plain(c, w, torch.float32 if kind == "b16" else torch.float64).forward(toks).numpy()
    model = rt.Model(dev, str(tmp_path))
    s = rt.Session(model, 4096, rt.Session.F32 if kind == "f32" else 0)
    edges = sorted({p for k in (150, 500) for m in range(1, T // k + 1) for p in (m * k - 1, m * k, m * k + 1) if p < T} | set(range(0, 6)) | {T - 1})
    tol = TOL[kind] * (1 if kind == "f32" else 2)
    assert logit_err(s.prefill_logits(toks, edges), want[edges]) < tol
    s.reset()
    s.prefill(toks[:2430])
    got = []
    for i in range(2430, 2730):
        s.step(toks[i], i)
        got.append(s.logits())
    assert logit_err(np.stack(got), want[2430:2730]) < tol
    assert logit_err(s.prefill_logits(toks[2730:], range(T - 2730), 2730), want[2730:]) < tol
    s.close()
    # batched decode keeps a ring of one chunk: 600 steps go round it
    bd = rt.BatchDecode(model, 2, 4096, flags=rt.BatchDecode.F32 if kind == "f32" else 0)
    err = []
    for i in range(700):
        bd.set_inputs([toks[i], toks[max(0, i - 40)]], [i, max(0, i - 40)])
        bd.step()
        bd.dev.sync()
        lg = bd.read("logits", np.float32).reshape(2, -1)
        err += [logit_err(lg[:1], want[i:i + 1]), logit_err(lg[1:], want[max(0, i - 40)][None])]
    assert np.sqrt(np.mean(np.square(err))) < tol
    bd.close()
    model.close()


def test_limits_are_refused(dev, rt, tmp_path):
    c = P.make_config(max_positions=20, layers=[L()])
    P.write_model(str(tmp_path), c, P.make_weights(c, 0))
    model = rt.Model(dev, str(tmp_path))
    s = rt.Session(model, 64)                       # positions end before the context asked for
    with pytest.raises(rt.RuntimeError_, match="context overflow"):
        s.prefill(list(range(21)))
    s.prefill(list(range(20)))
    with pytest.raises(rt.RuntimeError_, match="context overflow"):
        s.step(1, 20)
    with pytest.raises(rt.RuntimeError_, match="ascending"):
        s.prefill_logits([1, 2, 3], [1, 1])
    with pytest.raises(rt.RuntimeError_, match="no MTP head"):
        s.mtp_draft(1, 1)
    s.close()
    model.close()
    named = rt.Model(dev, "synth:sinepel-tiny:seed=3")
    s = rt.Session(named, 4096, rt.Session.PERSISTENT)      # no persistent step: a recorded list
    assert s.launches_per_token() > 1 and len(s.generate([1, 2, 3], 5)) == 5
    s.close()
    named.close()
    tiny = rt.Model(dev, "synth:tiny")
    with pytest.raises(rt.RuntimeError_, match="32-bit"):
        rt.Session(tiny, 32, rt.Session.F32)
    # the INT4 model's logits of chosen rows, by the same call
    s = rt.Session(tiny, 64)
    p = [5, 17, 200, 9, 33, 7]
    a = s.prefill_logits(p, [2, 5])
    s.reset()
    for i, t in enumerate(p):
        s.step(t, i)
        if i in (2, 5):
            assert np.array_equal(s.logits(), a[0 if i == 2 else 1])
    s.close()
    tiny.close()


def test_trace_replay(rt, bundle, tmp_path):
    """bin/trace_run: two requests that alternate, wanted places in any order, a request that ends and
    whose session serves another."""
    import os
    c, plain, _, toks, want, folder = bundle
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    other = [(3 * t + 2) % c["vocab"] for t in toks[:50]]
    ref = plain.forward(other).numpy()
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": toks[:40], "want": [0, 39]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": other[:7], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": toks[40:41], "want": [0]}, {"id": "b", "tokens": other[7:50], "want": [42, 1]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "c", "tokens": other[:1], "want": [0]}], "end": []},
    ]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "160"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
    rd = lambda i: np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, c["vocab"])   # noqa: E731
    assert not (tmp_path / "1.f32").exists()
    for got, exp in ((rd(0), want[[0, 39]]), (rd(2), np.stack([want[40], ref[49], ref[8]])), (rd(3), ref[:1])):
        assert np.sqrt(((got - exp) ** 2).mean()) / want.std() < TOL["f32"]
