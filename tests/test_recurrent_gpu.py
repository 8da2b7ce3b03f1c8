"""Kernels of the layers with a recurrent state and of grouped attention against plain float64 loops: scan in both forms,
short convolution, gated norm, head norms with rotation and cache write, attention over the cache, closing norms."""
import ctypes
import importlib

import numpy as np
import pytest
import torch

from conftest import PKG
from oracle import float_oracle as fo

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def K(float_libpath):
    torch.backends.cuda.matmul.allow_tf32 = False
    return importlib.import_module(PKG + ".float_kernel")


def rnd(shape, dtype, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * scale).to(getattr(torch, dtype)).cuda()


def i32(*x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def np64(t):
    return t.double().cpu().numpy()


# ---- linear attention with a decaying state ----------------------------------------------------------------------
def run_scan(K, dtype, starts, seq, heads, groups, n, p, stepped, skip, decay=None, seed=0, poke=None):
    """one call on random inputs -> (outputs, states after, wanted outputs, wanted states)"""
    B, dt = len(starts), getattr(torch, dtype)
    tok = heads * p + 2 * groups * n + 8
    x = rnd((B * seq, tok), dtype, seed)
    if poke:
        poke(x)
    slots = [(3 * b + 1) % (B + 2) for b in range(B)]
    S = rnd((B + 2, heads, n, p), "float32", seed + 1)
    before = np64(S)
    g = np.random.default_rng(seed)
    if decay is None:
        decay = np.exp(g.uniform(-4, 1.5, heads)) if stepped else 1 - 2.0 ** -g.uniform(2, 11, heads)
    dec = torch.tensor(decay, dtype=torch.float32, device="cuda")
    sh = 8 * ((heads + 7) // 8)
    step, bias = rnd((B * seq, sh), "float32", seed + 2), rnd((heads,), "float32", seed + 3) - 2.0
    D = rnd((heads,), "float32", seed + 4) if skip else None
    out = torch.full((B * seq, heads * p), 9.0, dtype=dt, device="cuda")
    st, sl = i32(*starts), i32(*slots)
    es, ks = x.element_size(), 0.7
    q, k, v = x[:, heads * p + groups * n:], x[:, heads * p:], x
    a = K.ScanArgs(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), dec.data_ptr(), step.data_ptr() if stepped else None,
                   bias.data_ptr() if stepped else None, D.data_ptr() if skip else None, S.data_ptr(), None, st.data_ptr(),
                   sl.data_ptr(), tok, tok, tok, heads * p, n, p, p, sh, B, seq, heads, B + 2, heads // groups, n, p, K.code(dt), ks)
    path = K.scan_path(ctypes.byref(a))
    K.scan(a, "cuda")
    K.device_status(sync=True)
    x64, want, states = np64(x), np.zeros((B * seq, heads, p)), before.copy()
    for b in range(B):
        r = slice(b * seq, (b + 1) * seq)
        for h in range(heads):
            gq = h // (heads // groups)
            kk = x64[r, heads * p + gq * n:heads * p + (gq + 1) * n]
            qq = x64[r, heads * p + (groups + gq) * n:heads * p + (groups + gq + 1) * n]
            vv = x64[r, h * p:(h + 1) * p]
            at, wt = np.full(seq, np64(dec)[h]), np.full(seq, ks)
            if stepped:
                d = fo.softplus(np64(step)[r, h] + np64(bias)[h])
                at, wt = np.exp(-np64(dec)[h] * d), ks * d
            s = before[slots[b], h] * (starts[b] != 0)
            for t in range(seq):
                s = at[t] * s + np.outer(wt[t] * kk[t], vv[t])
                want[b * seq + t, h] = qq[t] @ s + (np64(D)[h] * vv[t] if skip else 0)
            states[slots[b], h] = s
    return path, np64(out).reshape(B * seq, heads, p), np64(S), want, states


SCANS = [  # starts, seq, heads, groups, n, p, stepped, skip
    ([0], 1, 2, 1, 64, 64, True, True), ([7], 1, 3, 3, 16, 24, False, False), ([0, 5], 2, 4, 2, 40, 48, True, True),
    ([9], 16, 2, 2, 128, 128, False, False), ([0], 17, 2, 1, 64, 64, True, True), ([3], 17, 1, 1, 8, 8, False, False),
    ([0, 11], 127, 4, 2, 48, 56, True, True), ([50], 128, 2, 2, 64, 96, False, False), ([0], 129, 3, 1, 128, 64, True, True),
    ([6, 0, 2], 300, 2, 1, 80, 136, True, False), ([1000], 700, 2, 2, 128, 200, False, True), ([0], 513, 6, 3, 72, 64, True, True),
    ([0], 2050, 1, 1, 64, 64, False, False), ([4], 1500, 2, 1, 128, 72, True, True), ([2], 70, 2, 1, 160, 40, True, True),
    ([2], 40, 1, 1, 264, 40, False, True)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", SCANS)
def test_scan(K, dtype, case):
    path, got, state, want, want_state = run_scan(K, dtype, *case)
    assert path == (1 if dtype == "bfloat16" and case[1] > 16 and case[4] <= 128 else 0)
    s = np.abs(state - want_state).max() / want_state.std()
    # the state is 32-bit in either format: what is stored in it differs only by the order of additions, or by the
    # remainder of two bfloat16 numbers on the tensor cores
    assert s < (2e-4 if path else 3e-5)
    assert close(got, want, dtype)


def close(got, want, dtype):
    """bfloat16: the result's own rounding and that of the decayed scores, on each head's scale"""
    d, spread = np.abs(got - want), want.std(axis=(0, 2), keepdims=True)
    return bool((d < 4e-5 * want.std()).all() if dtype == "float32" else (d < 8e-3 * np.abs(want) + 2.5e-2 * spread).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay", [0.0, 1e-30, 0.5, 1.0])
def test_scan_with_extreme_decays(K, dtype, decay):
    path, got, state, want, ws = run_scan(K, dtype, [3], 200, 2, 1, 64, 64, False, False, decay=[decay, 0.99])
    assert np.isfinite(got).all() and close(got, want, dtype)
    # steps so large that everything before a token is forgotten, beside a head that forgets nothing
    path, got, state, want, ws = run_scan(K, dtype, [3], 200, 2, 1, 64, 64, True, False, decay=[decay * 100, 0.0])
    assert np.isfinite(got).all() and close(got, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("at", [0, 31, 32, 127, 128, 255, 600])
def test_scan_carries_a_far_token(K, dtype, at):
    """one key that only the last token asks for, from every place of a chunk"""
    n = 64

    def poke(x):
        x[:, 64:] = 0                              # keys and queries, then the one pair
        x[at, 64] = 4.0
        x[-1, 64 + n] = 2.0
    path, got, state, want, ws = run_scan(K, dtype, [0], 700, 1, 1, n, 64, False, False, decay=[0.9990234375], poke=poke)
    assert np.abs(want[-1]).max() > 0.5 and np.abs(got - want).max() < 1e-2 * np.abs(want[-1]).max()


# ---- short convolution --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 7])
@pytest.mark.parametrize("portions", [[70], [1] * 9, [2, 1, 3, 33, 2], [64, 1, 40]])
def test_short_conv_in_portions(K, dtype, taps, portions):
    dt, C, B, T = getattr(torch, dtype), 136, 2, sum(portions)
    x = rnd((B, T, C + 16), dtype, 1)
    w, b = rnd((taps, C), "float32", 2), rnd((C,), "float32", 3)
    state = rnd((4, max(taps - 1, 1), C), dtype, 4, 50.0)             # what an earlier request left
    slots, at = i32(3, 1), 0
    got = []
    for n in portions:
        part = x[:, at:at + n].reshape(B * n, -1).contiguous()
        out = torch.empty((B * n, C), dtype=dt, device="cuda")
        start = i32(at, at)
        K.short_conv(K.ConvArgs(part.data_ptr(), w.data_ptr(), b.data_ptr(), out.data_ptr(), state.data_ptr(), start.data_ptr(),
                                slots.data_ptr(), part.stride(0), C, B, n, 4, C, taps, K.code(dt)))
        got.append(np64(out).reshape(B, n, C))
        at += n
    got = np.concatenate(got, 1)
    for i in range(B):
        want = fo.silu(fo.short_conv(np64(x[i, :, :C]), np64(w).T, np64(b)))
        assert np.abs(got[i] - want).max() < (2e-5 if dtype == "float32" else 5e-2)
        if taps > 1 and T >= taps - 1:
            assert np.array_equal(np64(state)[[3, 1][i]], np64(x[i, T - taps + 1:, :C]))


# ---- gated norm -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,vdim,part", [(3, 24, 24), (4, 20, 20), (6, 40, 80), (10, 24, 120), (3, 20, 30), (2, 12, 4), (4, 64, 256),
                                             (1, 8, 8), (12, 128, 1536), (5, 100, 250), (10, 100, 1000)])
def test_gated_norm(K, dtype, heads, vdim, part):
    dt, p, rows = getattr(torch, dtype), (vdim + 7) // 8 * 8, 5
    def padded(t):
        out = torch.zeros((rows, heads, p), dtype=dt, device="cuda")
        out[:, :, :vdim] = t.view(rows, heads, vdim)
        return out.view(rows, heads * p)
    x, g = padded(rnd((rows, heads * vdim), dtype, 1, 3.0)), padded(rnd((rows, heads * vdim), dtype, 2, 2.0))
    w = torch.zeros((heads, p), device="cuda"); w[:, :vdim] = rnd((heads, vdim), "float32", 3)
    x64, g64 = (np64(t).reshape(rows, heads, p)[:, :, :vdim].reshape(rows, -1) for t in (x, g))
    for weighted in ([True, False] if part == vdim else [True]):
        out = torch.full((rows, heads * p), 5.0, dtype=dt, device="cuda")
        K.gated_norm(K.GatedNormArgs(x.data_ptr(), g.data_ptr(), w.data_ptr() if weighted else None, out.data_ptr(), heads * p,
                                     heads * p, heads * p, rows, heads, vdim, p, part, K.code(dt), 0.6, 0.3))
        if weighted:
            y = (x64 * fo.silu(g64)).reshape(rows, -1, part)
            want = fo.rms_norm(y, 1.0, 0.3).reshape(rows, -1) * np64(w)[:, :vdim].reshape(-1)
        else:
            want = 0.6 * fo.rms_norm(x64.reshape(rows, -1, part), 1.0, 0.3).reshape(rows, -1) * fo.silu(g64)
        got = np64(out).reshape(rows, heads, p)
        assert np.abs(got[:, :, :vdim].reshape(rows, -1) - want).max() < (3e-5 if dtype == "float32" else 8e-2)
        assert not got[:, :, vdim:].any()


# ---- heads: norm, rotation, cache -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,dims", [(4, 2, 64, 64), (3, 3, 20, 8), (8, 1, 96, 32), (2, 1, 128, 128), (2, 2, 256, 100), (1, 1, 300, 300)])
def test_heads_are_normed_turned_and_cached(K, dtype, H, G, dim, dims):
    fm, cm = (importlib.import_module(PKG + n) for n in (".float_model", ".float_config"))
    dt, d, seq, starts, slots, cap = getattr(torch, dtype), K.pad8(dim), 3, [4, 10], [2, 0], 12
    rows, tok = 2 * seq, 16 + (H + G) * d
    rot = cm.Rotary(70.0, dims, "half")
    order = fm._rotation_order(rot, dim)
    table = fm.rotary_table(rot, 40, "cuda")
    raw = rnd((rows, H + G, dim), dtype, 5, 2.0)
    y = torch.full((rows, tok), 7.0, dtype=dt, device="cuda")
    y[:, 8:8 + (H + G) * d] = 0
    y[:, 8:8 + (H + G) * d].view(rows, H + G, d)[:, :, :dim] = raw[:, :, order]
    wq, wk = rnd((dim,), "float32", 6), rnd((dim,), "float32", 7)
    pad = lambda w: fm._padded(w.cpu()[order], (d,), torch.float32, "cuda")
    wqp, wkp = pad(wq), pad(wk)
    q = torch.full((rows, H, d), 3.0, dtype=dt, device="cuda")
    cache = torch.full((3, cap, 2 * G * d), 5.0, dtype=dt, device="cuda")
    st, sl = i32(*starts), i32(*slots)
    K.heads_post(K.HeadsArgs(y.data_ptr(), wqp.data_ptr(), wkp.data_ptr(), q.data_ptr(), cache.data_ptr(), table.data_ptr(),
                             st.data_ptr(), sl.data_ptr(), tok, 8, 8 + H * d, rows, seq, cache.stride(0), cache.stride(1), cap, H, G, d,
                             dim, dims // 2, K.code(dt), 0.2))
    tol, r64 = 2e-5 if dtype == "float32" else 4e-2, np64(raw)
    pos = np.concatenate([np.arange(s, s + seq) for s in starts]).astype(np.float64)
    turned = lambda x, w: fo.rotate_half(fo.rms_norm(x, np64(w), 0.2), pos, dims, 70.0)[:, :, order.numpy()]
    qw, kw = turned(r64[:, :H], wq), turned(r64[:, H:], wk)
    got_q, got = np64(q), np64(cache).reshape(3, cap, 2, G, d)
    untouched = np.ones((3, cap), bool)
    for r in range(rows):
        b, p = r // seq, int(pos[r])
        if p >= cap:
            assert (got_q[r] == 3.0).all()
            continue
        untouched[slots[b], p] = False
        assert np.abs(got_q[r, :, :dim] - qw[r]).max() < tol and not got_q[r, :, dim:].any()
        assert np.abs(got[slots[b], p, 0, :, :dim] - kw[r]).max() < tol
        assert np.array_equal(got[slots[b], p, 1, :, :dim], r64[r, H:][:, order.numpy()])
    assert (got[untouched] == 5.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("starts,S,H,G,d,window", [
    ([0], 1, 4, 2, 64, 90), ([255], 1, 4, 4, 64, 64), ([256], 1, 4, 1, 64, 65), ([100], 2, 6, 2, 40, 90), ([77], 16, 16, 2, 64, 40),
    ([5, 130], 3, 24, 8, 128, 64), ([1000], 1, 32, 8, 128, 513), ([700], 5, 8, 2, 96, 0), ([0, 63, 64], 1, 5, 5, 72, 65),
    ([300], 1, 8, 8, 24, 1), ([130], 2, 2, 1, 264, 100), ([62], 3, 2, 1, 512, 64)])
def test_grouped_attention_over_the_cache(K, dtype, starts, S, H, G, d, window):
    dt, B, cap = getattr(torch, dtype), len(starts), max(starts) + S + 9
    cache, q, g = rnd((B + 2, cap, 2 * G * d), dtype), rnd((B * S, H, d), dtype, 1), rnd((B * S, H * d + 8), dtype, 2)
    slots = [(2 * b + 1) % (B + 2) for b in range(B)]
    for b, s in enumerate(starts):
        i = s + S - 1
        if window and i - window + 1 > 0:
            cache[slots[b], i - window + 1, :d] = q[b * S + S - 1, 0] * 0.5      # just inside
            cache[slots[b], i - window, :d] = q[b * S + S - 1, 0] * 2            # just outside
    out = torch.zeros((B * S, H * d + 16), dtype=dt, device="cuda")
    st, sl = i32(*starts), i32(*slots)
    bound = min(max(starts) + S, window + S - 1) if window else max(starts) + S
    for gate in (None, g):
        a = K.GroupedArgs(q.data_ptr(), cache.data_ptr(), out.data_ptr(), K.ptr(gate), st.data_ptr(), sl.data_ptr(), None,
                          cache.stride(0), cache.stride(1), cap, G * d, out.stride(0), g.stride(0), B, S, H, G, d, window, bound,
                          K.code(dt), d ** -0.5, 0.7)
        K.grouped_attention(a, "cuda")
        for b, s in enumerate(starts):
            kv = np64(cache[slots[b], :s + S]).reshape(s + S, 2, G, d)
            i, j = np.arange(S)[:, None] + s, np.arange(s + S)[None]
            seen = (j <= i) & ((i - j < window) if window else True)
            for h in range(H):
                r = slice(b * S, (b + 1) * S)
                w = fo.softmax_rows(np64(q)[r, h] @ kv[:, 0, h // (H // G)].T * d ** -0.5, seen) @ kv[:, 1, h // (H // G)]
                if gate is not None:
                    w = w * fo.sigmoid(np64(g)[r, h * d:(h + 1) * d]) * 0.7
                assert np.abs(np64(out)[r, h * d:(h + 1) * d] - w).max() < (2e-5 if dtype == "float32" else 3e-2)
    assert not np64(out)[:, H * d:].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,start,H,G,d,window", [(17, 0, 4, 2, 64, 90), (130, 0, 2, 1, 96, 0), (300, 50, 6, 3, 48, 130),
                                                  (257, 90, 4, 4, 128, 1), (513, 700, 8, 2, 128, 257), (150, 20, 2, 1, 168, 77)])
def test_grouped_prefill_attention(K, dtype, S, start, H, G, d, window):
    dt = getattr(torch, dtype)
    base = max(0, start - window + 1) if window else 0
    keys = start + S - base
    q, kv, g = rnd((S, H, d), dtype), rnd((keys, 2 * G * d), dtype, 1), rnd((S, H * d + 8), dtype, 2)
    if window and window < keys:
        kv[keys - window, :d] = q[-1, 0] * 2                       # just inside the last query's window
        kv[keys - window - 1, :d] = q[-1, 0] * 3                   # just outside
    out, st = torch.zeros((S, H * d + 16), dtype=dt, device="cuda"), i32(start)
    es, p = q.element_size(), kv.data_ptr()
    for gate in (None, g):
        a = K.AttentionArgs(q.data_ptr(), p, p, p + G * d * es, out.data_ptr(), st.data_ptr(), None, None, d, d, kv.stride(0), d,
                            kv.stride(0), kv.stride(0), d, 0, base, keys, 1, S, H, d, 0, d, window, 0, K.code(dt), d ** -0.5, keys,
                            H // G, K.ptr(gate), g.stride(0), d, out.stride(0), 0.7)
        assert K.attention_path(ctypes.byref(a)) == (1 if dtype == "bfloat16" and d <= 128 else 0)
        K.attention(a)
        k64 = np64(kv).reshape(keys, 2, G, d)
        i, j = np.arange(S)[:, None] + start, np.arange(keys)[None] + base
        seen = (j <= i) & ((i - j < window) if window else True)
        for h in range(H):
            w = fo.softmax_rows(np64(q)[:, h] @ k64[:, 0, h // (H // G)].T * d ** -0.5, seen) @ k64[:, 1, h // (H // G)]
            if gate is not None:
                w = w * fo.sigmoid(np64(g)[:, h * d:(h + 1) * d]) * 0.7
            assert np.abs(np64(out)[:, h * d:(h + 1) * d] - w).max() < (3e-5 if dtype == "float32" else 3e-2)
    K.device_status(sync=True)


# ---- epilogues and closing norms ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,Kd,split", [(1, 168, 72, 160), (2, 640, 328, 608), (5, 1032, 520, 1024), (130, 136, 96, 128), (300, 2120, 264, 2112),
                                          (7, 200, 4096, 192)])
def test_linear_with_bias_second_output_and_a_rotated_range(K, dtype, M, N, Kd, split):
    A, W, bias = rnd((M, Kd), dtype), rnd((N, Kd), dtype, 1, Kd ** -0.5), rnd((N,), "float32", 2)
    ref = np64(A) @ np64(W).T + np64(bias)
    out, out2 = torch.empty((M, split), dtype=A.dtype, device="cuda"), torch.empty((M, N - split), device="cuda")
    table, begin, end, period, pairs = rnd((M + 9, 5, 2), "float32", 3), 24, 24 + 3 * 32, 32, 5
    K.linear(A, W, out, K.ROTATE, table=table, start=i32(4), seq=M, pairs=pairs, period=period, rotated=(begin, end), bias=bias, out2=out2)
    want, tab = ref.copy(), np64(table)
    for n in range(begin, end, 2):
        i = (n - begin) % period // 2
        if i < pairs:
            c, s = tab[4:4 + M, i, 0], tab[4:4 + M, i, 1]
            want[:, n], want[:, n + 1] = ref[:, n] * c - ref[:, n + 1] * s, ref[:, n + 1] * c + ref[:, n] * s
    tol = 5e-5 if dtype == "float32" else 6e-2
    assert np.abs(np64(out) - want[:, :split]).max() < tol and np.abs(np64(out2) - want[:, split:]).max() < 5e-5
    n = N // 16 * 16
    glu = torch.empty((M, n // 2), dtype=A.dtype, device="cuda")
    K.linear(A, W[:n], glu, K.GLU, bias=bias)
    assert np.abs(np64(glu) - fo.silu(ref[:, 0:n:2]) * ref[:, 1:n:2]).max() < tol
    K.device_status(sync=True)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [52, 328, 9000])
def test_add_norm_makes_the_next_input(K, dtype, width):
    pitch = K.pad8(width)
    x, y = rnd((5, pitch), "float32", 1), rnd((5, pitch), "float32", 2, 3.0)
    w, w2 = (torch.zeros(pitch, device="cuda") for _ in range(2))
    w[:width], w2[:width] = rnd((width,), "float32", 3), rnd((width,), "float32", 4)
    x[:, width:] = 0; y[:, width:] = 0
    xs, ys, ws, w2s = (np64(t)[..., :width] for t in (x, y, w, w2))
    h = torch.empty((5, pitch), dtype=getattr(torch, dtype), device="cuda")
    K.add_norm(x, y, w, h, width, 0.5, w2)
    new = xs + fo.rms_norm(ys, ws, 0.5)
    assert np.abs(np64(x)[:, :width] - new).max() < 1e-5
    assert np.abs(np64(h)[:, :width] - fo.rms_norm(new, w2s, 0.5)).max() < (2e-5 if dtype == "float32" else 4e-2)
    table = rnd((7, pitch), dtype, 4)
    K.embed(torch.tensor([6, 0, 3, 7, -1], device="cuda"), table, 7, x, None, 3.25)
    assert torch.equal(x[:3], table[[6, 0, 3]].float() * 3.25) and not x[3:].any()
