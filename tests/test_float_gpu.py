"""The floating-point decoder designs on the GPU against the plain oracle: every kernel alone, whole prompts, decoding,
portions, batches, reused slots, window and tile edges, generation and the two command lines."""
import ctypes
import importlib
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import float_cases as fc
from conftest import PKG, ROOT
from oracle import float_oracle as fo

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
CASES = ["ODD", "PEAKED", "WIDE"] + list(fc.RECURRENT)


@pytest.fixture(scope="module")
def K(float_libpath):
    torch.backends.cuda.matmul.allow_tf32 = False
    return importlib.import_module(PKG + ".float_kernel")


@pytest.fixture(scope="module")
def models(float_libpath, tmp_path_factory):
    """models(case, dtype): (config, weights, loaded model), each loaded once"""
    registry = importlib.import_module(PKG + ".registry")
    made = {}

    def get(case, dtype):
        if (case, dtype) not in made:
            cfg = getattr(fc, case)
            W = fc.make_weights(cfg, 11)
            path = fc.write_checkpoint(str(tmp_path_factory.mktemp("m")), cfg, W)
            made[case, dtype] = (cfg, W, registry.load(path, dtype=dtype, max_seq_len=640, max_batch_size=4))
        return made[case, dtype]

    return get


def tokens_of(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def run(model, toks, portions=None, want=None):
    """logits of all (or the wanted) positions of one request, its tokens cut into portions"""
    slots, out, at = model.begin_batch(1), [], 0
    try:
        for n in (portions or []) + [len(toks)]:
            n = min(n, len(toks) - at)
            if n:
                w = [p - at for p in range(at, at + n) if want is None or p in want]
                out.append(model.step(torch.tensor([toks[at:at + n]]), at, slots, want=w)[0].cpu().numpy())
            at += n
    finally:
        model.end_batch(slots)
    return np.concatenate(out)


# ---- kernels alone ---------------------------------------------------------------------------------------------
def rnd(shape, dtype, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * scale).to(getattr(torch, dtype)).cuda()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,Kd", [(1, 640, 328), (3, 24, 8), (4, 1032, 1544), (5, 200, 96), (16, 104, 3000), (17, 64, 64),
                                    (129, 96, 80), (300, 1000, 72), (257, 2120, 520), (70, 48, 2056), (9, 2120, 7168), (600, 136, 4096)])
def test_linear_and_its_epilogues(K, dtype, M, N, Kd):
    A, W = rnd((M, Kd), dtype), rnd((N, Kd), dtype, 1, Kd ** -0.5)
    want = A.double() @ W.double().T
    out = torch.full((M, N), 7.0, device="cuda")
    K.linear(A, W, out)
    assert (out - want).abs().max() < 2e-5 * (1 + Kd / 2048)
    loose = 3e-5 * (1 + Kd / 2048) if dtype == "float32" else 5e-2
    aux, gated = rnd((M, N), dtype, 2), torch.empty((M, N), dtype=A.dtype, device="cuda")
    K.linear(A, W, gated, K.GATE, aux=aux)
    assert (gated - torch.sigmoid(want) * aux).abs().max() < loose
    n = N // 16 * 16
    glu = torch.empty((M, n // 2), dtype=A.dtype, device="cuda")
    K.linear(A, W[:n], glu, K.GLU)
    assert (glu - torch.nn.functional.silu(want[:, 0:n:2]) * want[:, 1:n:2]).abs().max() < loose
    # two sequences at different positions when the rows divide
    seq, period, offset, pairs = (M // 2 if M % 2 == 0 else M), 24, 16, 3
    start = torch.tensor([4, 9][: M // seq], dtype=torch.int32, device="cuda")
    table = rnd((seq + 10, pairs, 2), "float32", 3)
    rot = torch.empty((M, N), dtype=A.dtype, device="cuda")
    K.linear(A, W, rot, K.ROTATE, table=table, start=start, seq=seq, pairs=pairs, period=period, offset=offset)
    pos = torch.cat([torch.arange(seq) + s for s in start.tolist()])
    ref = want.clone()
    for n in range(0, N, 2):
        i = (n % period - offset) // 2
        if n % period >= offset and i < pairs:
            c, s = table[pos.cuda(), i, 0].double(), table[pos.cuda(), i, 1].double()
            ref[:, n], ref[:, n + 1] = want[:, n] * c - want[:, n + 1] * s, want[:, n + 1] * c + want[:, n] * s
    assert (rot - ref).abs().max() < loose
    K.device_status(sync=True)


def test_linear_takes_the_kernel_meant_for_the_shape(K):
    def path(M, dtype):
        a = K.LinearArgs()
        a.M, a.N, a.K, a.dtype = M, 64, 64, dtype
        return K.linear_path(ctypes.byref(a))
    assert path(1, K.BF16) == 2 and path(1, K.F32) == 2 and path(100, K.BF16) == 1 and path(100, K.F32) == 0


@pytest.mark.parametrize("width", [52, 328, 9000])
def test_norms_and_embedding(K, width):
    pitch = K.pad8(width)
    x, y = rnd((5, pitch), "float32", 1), rnd((5, pitch), "float32", 2, 3.0)
    w = torch.zeros(pitch, device="cuda"); w[:width] = rnd((width,), "float32", 3)
    x[:, width:] = 0; y[:, width:] = 0
    xs, ys, ws = (t.double().cpu().numpy()[..., :width] for t in (x, y, w))
    xb = torch.empty((5, pitch), dtype=torch.bfloat16, device="cuda")
    index = torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda")
    out = torch.empty((3, pitch), device="cuda")
    K.norm_rows(x, index, w, out, width, 1e-3)
    assert np.abs(out.cpu().numpy()[:, :width] - fo.rms_norm(xs, ws, 1e-3)[[4, 0, 4]]).max() < 1e-5
    K.add_norm(x, y, w, xb, width, 0.5)
    want = xs + fo.rms_norm(ys, ws, 0.5)
    assert np.abs(x.cpu().numpy()[:, :width] - want).max() < 1e-5 and torch.equal(xb, x.to(torch.bfloat16))
    table = rnd((7, pitch), "bfloat16", 4)
    K.embed(torch.tensor([6, 0, 3, 7, -1], device="cuda"), table, 7, x, xb)
    assert torch.equal(x[:3], table[[6, 0, 3]].float()) and torch.equal(xb[0], table[6]) and not x[3:].any()


def attention_args(K, q, k1, k2, v, out, start, **kw):
    a = K.AttentionArgs()
    a.q, a.k1, a.k2, a.v, a.out, a.start = q.data_ptr(), k1, k2, v, out.data_ptr(), start.data_ptr()
    for n, x in kw.items():
        setattr(a, n, x)
    return a


def plain_attention(q, k, v, start, base, window, scale):
    """q [S, H, D], k [keys, H, D], v [keys, H, V] float64"""
    i, j = np.arange(q.shape[0])[:, None] + start, np.arange(k.shape[0])[None] + base
    seen = (j <= i) & ((i - j < window) if window else True)
    return np.stack([fo.softmax_rows(q[:, h] @ k[:, h].T * scale, seen) @ v[:, h] for h in range(q.shape[1])], 1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,start,H,D,R,V,window", [
    (17, 0, 2, 64, 32, 64, 90), (130, 0, 1, 64, 32, 64, 0), (300, 50, 3, 48, 16, 80, 130), (300, 0, 2, 64, 32, 64, 7),
    (257, 90, 2, 40, 24, 56, 1), (513, 700, 1, 128, 64, 128, 257), (260, 5, 2, 128, 64, 120, 100000), (385, 128, 1, 16, 8, 16, 129),
    (150, 20, 2, 64, 32, 168, 77), (90, 0, 1, 456, 64, 64, 50)])
def test_expanded_attention(K, dtype, S, start, H, D, R, V, window):
    dt = getattr(torch, dtype)
    base = max(0, start - window + 1) if window else 0
    keys = start + S - base
    q, kv, kr = rnd((S, H, D + R), dtype), rnd((keys, H * (D + V)), dtype, 1), rnd((keys, R + 8), dtype, 2)
    out, st = torch.zeros((S, H, V), dtype=dt, device="cuda"), torch.tensor([start], dtype=torch.int32, device="cuda")
    # one key far above the rest just inside and just outside the last query's window
    if window and window < keys:
        kv[keys - window, :H * D] = q[-1, :, :D].reshape(-1) * 2
        if keys > window:
            kv[keys - window - 1, :H * D] = q[-1, :, :D].reshape(-1) * 3
    es = kv.element_size()
    a = attention_args(K, q, kv.data_ptr(), kr.data_ptr(), kv.data_ptr() + H * D * es, out, st, q_head=D + R, o_head=V,
                       k1_tok=kv.stride(0), k1_head=D, k2_tok=kr.stride(0), v_tok=kv.stride(0), v_head=V, base=base,
                       keys=keys, batch=1, seq=S, heads=H, d1=D, d2=R, dv=V, window=window, shared=0, dtype=K.code(dt),
                       scale=(D + R) ** -0.5, max_keys=keys)
    fits = V <= 128 and D <= 320                  # wider heads run on the CUDA cores
    assert K.attention_path(ctypes.byref(a)) == (1 if dtype == "bfloat16" and fits else 0)
    K.attention(a)
    q64, kv64, kr64 = (t.double().cpu().numpy() for t in (q, kv, kr))
    k = np.concatenate([kv64[:, :H * D].reshape(keys, H, D), np.repeat(kr64[:, None, :R], H, 1)], 2)
    want = plain_attention(q64, k, kv64[:, H * D:].reshape(keys, H, V), start, base, window, (D + R) ** -0.5)
    got = out.double().cpu().numpy()
    assert np.abs(got - want).max() < (2e-5 if dtype == "float32" else 3e-2)
    K.device_status(sync=True)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("starts,S,H,C,R,window", [
    ([0], 1, 4, 64, 32, 90), ([255], 1, 4, 64, 32, 64), ([256], 1, 4, 64, 32, 65), ([100], 2, 5, 64, 32, 90),
    ([77], 16, 16, 64, 32, 40), ([5, 130], 3, 24, 128, 64, 64), ([1000], 1, 128, 512, 64, 513), ([700], 5, 48, 512, 64, 0),
    ([0, 63, 64], 1, 5, 72, 40, 65), ([300], 1, 8, 24, 8, 1), ([130], 2, 3, 520, 64, 100)])
def test_latent_attention(K, dtype, starts, S, H, C, R, window):
    dt, B, P, cap = getattr(torch, dtype), len(starts), C + R, max(starts) + S + 9
    cache, q = rnd((B + 2, cap, P), dtype), rnd((B * S, H, P), dtype, 1)
    slots = [(2 * b + 1) % (B + 2) for b in range(B)]
    for b, s in enumerate(starts):
        i = s + S - 1
        if window and i - window + 1 > 0:
            cache[slots[b], i - window + 1, :C] = q[b * S + S - 1, 0, :C] * 0.5      # just inside
            cache[slots[b], i - window, :C] = q[b * S + S - 1, 0, :C] * 2            # just outside
    out = torch.zeros((B * S, H, C), dtype=dt, device="cuda")
    st, sl = (torch.tensor(x, dtype=torch.int32, device="cuda") for x in (starts, slots))
    es = cache.element_size()
    a = attention_args(K, q, cache.data_ptr(), cache.data_ptr() + C * es, cache.data_ptr(), out, st, slots=sl.data_ptr(),
                       q_head=P, o_head=C, k1_tok=P, k2_tok=P, v_tok=P, slot_stride=cache.stride(0), keys=cap, batch=B, seq=S,
                       heads=H, d1=C, d2=R, dv=C, window=window, shared=1, dtype=K.code(dt), scale=P ** -0.5,
                       max_keys=min(max(starts) + S, window + S - 1) if window else max(starts) + S)
    assert K.attention_path(ctypes.byref(a)) == (1 if dtype == "bfloat16" and C <= 512 else 0)
    n = K.attention_scratch(a)
    scratch = torch.full((max(n, 1),), float("nan"), device="cuda")      # nothing may be read before it is written
    a.scratch = scratch.data_ptr()
    K.attention(a)
    for b, s in enumerate(starts):
        kc = cache[slots[b], :s + S].double().cpu().numpy()
        k = np.repeat(kc[:, None], H, 1)
        want = plain_attention(q[b * S:(b + 1) * S].double().cpu().numpy(), k, k[:, :, :C], s, 0, window, P ** -0.5)
        assert np.abs(out[b * S:(b + 1) * S].double().cpu().numpy() - want).max() < (2e-5 if dtype == "float32" else 3e-2)
    K.device_status(sync=True)


@pytest.mark.parametrize("dtype", DTYPES)
def test_latents_reach_the_cache_normed_and_rotated(K, dtype):
    dt, q_rank, C, R, seq, B = getattr(torch, dtype), 28, 36, 6, 3, 2
    qp, cp, pitch = K.pad8(q_rank), K.pad8(C), K.pad8(C) + K.pad8(R)
    y = torch.zeros((B * seq, qp + pitch), device="cuda")
    raw = rnd((B * seq, q_rank + C + R), "float32", 5, 2.0)
    y[:, :q_rank], y[:, qp:qp + C], y[:, qp + cp:qp + cp + R] = raw[:, :q_rank], raw[:, q_rank:q_rank + C], raw[:, q_rank + C:]
    wq, wc = torch.zeros(qp, device="cuda"), torch.zeros(cp, device="cuda")
    wq[:q_rank], wc[:C] = rnd((q_rank,), "float32", 6), rnd((C,), "float32", 7)
    fm = importlib.import_module(PKG + ".float_model")
    table = fm.rotary_table(importlib.import_module(PKG + ".float_config").Rotary(70.0, R), 40, "cuda")
    cache = torch.full((3, 12, pitch), 5.0, dtype=dt, device="cuda")
    cq = torch.empty((B * seq, qp), dtype=dt, device="cuda")
    start, slots = (torch.tensor(x, dtype=torch.int32, device="cuda") for x in ([4, 10], [2, 0]))
    a = K.LatentArgs(y.data_ptr(), wq.data_ptr(), wc.data_ptr(), cq.data_ptr(), cache.data_ptr(), table.data_ptr(),
                     start.data_ptr(), slots.data_ptr(), y.stride(0), cq.stride(0), B * seq, seq, cache.stride(0),
                     cache.stride(1), 12, q_rank, qp, C, cp, R // 2, 1, K.code(dt), 1e-2)
    K.latent_post(a)
    r = raw.double().cpu().numpy()
    tol = 1e-5 if dtype == "float32" else 3e-2
    assert np.abs(cq.double().cpu().numpy()[:, :q_rank] - fo.rms_norm(r[:, :q_rank], wq[:q_rank].double().cpu().numpy(), 1e-2)).max() < tol
    c = fo.rms_norm(r[:, q_rank:q_rank + C], wc[:C].double().cpu().numpy(), 1e-2)
    got = cache.double().cpu().numpy()
    for b, (s, slot) in enumerate(((4, 2), (10, 0))):
        kr = fo.rotate_pairs(r[b * seq:(b + 1) * seq, q_rank + C:], np.arange(s, s + seq, dtype=np.float64), 70.0)
        for t in range(seq):
            if s + t >= 12:
                continue                          # beyond the capacity: not written anywhere
            assert np.abs(got[slot, s + t, :C] - c[b * seq + t]).max() < tol
            assert np.abs(got[slot, s + t, cp:cp + R] - kr[t]).max() < tol
    untouched = np.ones((3, 12), bool)
    untouched[2, 4:7] = untouched[0, 10:12] = False
    assert (got[untouched] == 5).all()


# ---- whole models ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", CASES)
@pytest.mark.parametrize("n", [1, 2, 16, 17, 64, 65, 128, 129, 300])
def test_prompt_against_the_oracle(models, case, dtype, n):
    cfg, W, model = models(case, dtype)
    toks = tokens_of(cfg, n, n)
    assert fc.Expected(cfg, W, toks).ok(run(model, toks), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["ODD", "V_ODD", "V_WIDE"])
def test_residual_after_every_layer(models, case, dtype):
    cfg, W, model = models(case, dtype)
    toks, got = tokens_of(cfg, 70), []
    want = fc.Expected(cfg, W, toks)
    s = model.begin_batch(1)
    model.step(torch.tensor([toks]), 0, s, want=[], layers_out=got)
    model.end_batch(s)
    assert len(got) == len(cfg["layers"])
    for i, g in enumerate(got):
        assert g.dtype == torch.float32 and want.layer_ok(i, g.cpu().numpy(), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", CASES)
def test_portions_and_decoding_give_the_prompt_s_logits(models, case, dtype):
    cfg, W, model = models(case, dtype)
    toks = tokens_of(cfg, 280, 7)
    want = fc.Expected(cfg, W, toks)
    for portions in ([1] * 280, [2] * 140, [3, 17, 2, 64, 65, 2, 127], [100, 2, 2, 16, 160], [33] * 9, [200] + [1] * 80,
                     [63, 1, 1, 1, 62, 1, 1, 150]):
        assert want.ok(run(model, toks, portions), dtype), portions[:8]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["PEAKED", "V_PEAKED"])
def test_long_decoding_past_every_window(models, case, dtype):
    cfg, W, model = models(case, dtype)
    toks = tokens_of(cfg, 600, 8)
    want = set(range(0, 600, 37)) | {63, 64, 65, 127, 128, 129, 192, 599}
    got = run(model, toks, [5] + [1] * 595, want)
    assert fc.Expected(cfg, W, toks).ok(got, dtype, sorted(want))


def edge_model(window):
    """One layer whose attention score between a query and the token `marker` stands out: queries and the marker's key
    agree in one latent direction that no other token has."""
    cfg = fc.config(40, 48, 1e-6, [fc.layer(2, 16, 8, 16, 24, 32, window, None, scale=4.0)])
    W = fc.make_weights(cfg, 21)
    W["l0.mix.dkv"][0] = 0
    W["l0.mix.dkv"][0, 0] = 6.0                     # latent 0 <- activation 0
    W["embed"][:, 0] = 0
    W["embed"][39, 0] = 8.0                         # only the marker token has activation 0
    W["embed"][:, 1] = 2.0
    W["l0.mix.dq"][0] = 0
    W["l0.mix.dq"][0, 1] = 4.0                      # every query carries query latent 0
    W["l0.mix.uq"][0] = 0
    W["l0.mix.uq"][0, 0] = 3.0
    W["l0.mix.uk"][0] = 0
    W["l0.mix.uk"][0, 0] = 3.0
    return cfg, {k: fc.bf16_round(v) for k, v in W.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 63, 64, 65, 127, 128, 129, 200])
def test_key_just_inside_and_just_outside_the_window(float_libpath, tmp_path, dtype, window):
    registry = importlib.import_module(PKG + ".registry")
    cfg, W = edge_model(window)
    model = registry.load(fc.write_checkpoint(str(tmp_path), cfg, W), dtype=dtype, max_seq_len=512, max_batch_size=1)
    for at in (0, 1, 60, 127, 128):
        toks = np.random.default_rng(at).integers(0, 39, at + window + 3)
        toks[at] = 39
        want = fc.Expected(cfg, W, toks)
        inside, outside = at + window - 1, at + window
        other = toks.copy(); other[at] = 3
        base = fc.oracle_logits(cfg, W, other)
        assert not want.ok(base[inside:inside + 1], "bfloat16", [inside])      # the key matters inside
        assert np.allclose(base[outside], want.logits[outside])                # and not outside
        for portions in (None, [inside] + [1] * 4, [inside - 1, 2, 2]):
            assert want.ok(run(model, toks.tolist(), portions), dtype)


def key_valued_edge_model(window):
    """One layer whose attention score between any query and the token `marker` stands out: in an unrotated direction of the
    head every query points one way, the marker's key the same way and every other key the opposite one."""
    cfg = fc.vifelix(40, 48, 1e-6, 2.0, [fc.parallel(4, 2, 16, 8, window, 1, 8, 8, 8, [0.9], None, scale=1.0, right_scale=0.0)])
    W = fc.make_weights(cfg, 21)
    W["embed"][:, 0] = 0
    W["embed"][39, 0] = 8.0                         # only the marker has activation 0
    for name, heads, bias in (("q", 4, 6.0), ("k", 2, -2.0)):
        for h in range(heads):
            W["l0.mix.left." + name][h * 16 + 15] = 0
            W["l0.mix.left." + name + ".b"][h * 16 + 15] = bias
    for h in range(2):
        W["l0.mix.left.k"][h * 16 + 15, 0] = 4.0
    W["l0.mix.left.q.norm"][15] = W["l0.mix.left.k.norm"][15] = 1.5
    return cfg, {k: fc.bf16_round(v) for k, v in W.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 63, 64, 65, 127, 128, 129, 200])
def test_key_inside_and_outside_the_window_of_key_valued_attention(float_libpath, tmp_path, dtype, window):
    registry = importlib.import_module(PKG + ".registry")
    cfg, W = key_valued_edge_model(window)
    model = registry.load(fc.write_checkpoint(str(tmp_path), cfg, W), dtype=dtype, max_seq_len=512, max_batch_size=1)
    for at in (0, 1, 60, 127, 128):
        toks = np.random.default_rng(at).integers(0, 39, at + window + 3)
        toks[at] = 39
        want = fc.Expected(cfg, W, toks)
        inside, outside = at + window - 1, at + window
        other = toks.copy(); other[at] = 3
        base = fc.oracle_logits(cfg, W, other)
        assert not want.ok(base[inside:inside + 1], "bfloat16", [inside])      # the key matters inside
        assert np.allclose(base[outside], want.logits[outside])                # and not outside
        for portions in (None, [inside] + [1] * 4, [inside - 1, 2, 2]):
            assert want.ok(run(model, toks.tolist(), portions), dtype)


def memory_model(kind):
    """One layer that writes the token `marker` into its state, hardly anything else, and reads it at every later token"""
    if kind == "retention":
        layer = fc.parallel(2, 1, 8, 8, 4, 2, 24, 16, 8, [0.998, 0.9995], None, left_scale=0.0)
    else:
        layer = fc.mamba2(2, 16, 24, 1, 4, 2)
    cfg = fc.vifelix(40, 48, 1e-6, 2.0, [layer])
    W = fc.make_weights(cfg, 22)
    W["embed"][:, 0], W["embed"][:, 1] = 0, 1.0
    W["embed"][39, 0] = 4.0                         # activation 0 is the marker's, activation 1 is everyone's
    if kind == "retention":
        for h in range(2):
            for name, source in (("q", 1), ("k", 0)):
                W["l0.mix.right." + name][h * 24:(h + 1) * 24] *= 0.05
                W["l0.mix.right." + name][h * 24 + 20, source] = 4.0
    else:
        i, n = 32, 24
        W["l0.mix.in"][2 * i:2 * i + 2 * n] *= 0.05
        W["l0.mix.in"][2 * i + 5, 0] = 6.0          # B
        W["l0.mix.in"][2 * i + n + 5, 1] = 6.0      # C
        W["l0.mix.conv.b"][i:] = 0
        W["l0.mix.conv"][i:] = np.array([0, 0, 0, 1.0])
        W["l0.mix.A_log"][:] = (-7.0, -6.0)
        W["l0.mix.D"][:] = 0.1
        W["l0.mix.in"][2 * i + 2 * n:] *= 0.1
    return cfg, {k: fc.bf16_round(v) for k, v in W.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["retention", "mamba2"])
def test_a_token_far_back_is_remembered(float_libpath, tmp_path, kind, dtype):
    registry = importlib.import_module(PKG + ".registry")
    cfg, W = memory_model(kind)
    model = registry.load(fc.write_checkpoint(str(tmp_path), cfg, W), dtype=dtype, max_seq_len=640, max_batch_size=2)
    for at in (0, 1, 2, 127, 128, 255):
        toks = np.random.default_rng(at).integers(0, 39, at + 330)
        toks[at] = 39
        want, other = fc.Expected(cfg, W, toks), toks.copy()
        other[at] = 3
        last = len(toks) - 1
        assert not want.ok(fc.oracle_logits(cfg, W, other)[last:], "bfloat16", [last])     # the token matters to the end
        for portions in (None, [at + 1, 2], [max(at, 1), 1, 16, 17, 200], [128, 128], [at + 300] + [1] * 30, [2] * 20):
            assert want.ok(run(model, toks.tolist(), portions), dtype), portions


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["WIDE", "V_WIDE", "V_ODD"])
def test_batch_equals_each_request_alone(models, case, dtype):
    cfg, W, model = models(case, dtype)
    rows = [tokens_of(cfg, 150, 30 + b) for b in range(3)]
    slots = model.begin_batch(3)
    got = [[] for _ in rows]
    at = 0
    for n in (100, 17, 2, 16, 1, 1, 13):
        lg = model.step(torch.tensor([r[at:at + n] for r in rows]), at, slots, want=list(range(3 * n)))[0]
        for b in range(3):
            got[b].append(lg[b * n:(b + 1) * n].cpu().numpy())
        at += n
    model.end_batch(slots)
    for b, r in enumerate(rows):
        assert fc.Expected(cfg, W, r).ok(np.concatenate(got[b]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["PEAKED", "V_PEAKED", "V_ODD"])
def test_a_used_slot_leaves_nothing_behind(models, case, dtype):
    cfg, W, model = models(case, dtype)
    short = tokens_of(cfg, 40, 50)
    first = run(model, short, [20, 2] + [1] * 18)
    for seed in range(3):                            # longer requests fill the slot with other latents
        run(model, tokens_of(cfg, 500, 60 + seed), [300] + [1] * 200, {499})
    again = run(model, short, [20, 2] + [1] * 18)
    assert np.array_equal(first, again)
    assert model.cache.free_slots() == model.cache.slots


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_take_turns(models, dtype):
    """two requests of different lengths, their portions interleaved, slots side by side"""
    cfg, W, model = models("V_WIDE", dtype)
    rows = [tokens_of(cfg, n, 40 + n) for n in (260, 90)]
    slots, at, got = [model.begin_batch(1) for _ in rows], [0, 0], [[], []]
    for r, n in ((0, 130), (1, 3), (0, 1), (1, 40), (0, 20), (1, 1), (0, 2), (1, 46), (0, 107)):
        part = torch.tensor([rows[r][at[r]:at[r] + n]])
        got[r].append(model.step(part, at[r], slots[r], want=list(range(n)))[0].cpu().numpy())
        at[r] += n
    for r in range(2):
        assert at[r] == len(rows[r]) and fc.Expected(cfg, W, rows[r]).ok(np.concatenate(got[r]), dtype)
        model.end_batch(slots[r])


@pytest.mark.parametrize("case", ["WIDE", "V_WIDE"])
def test_large_steps_run_in_portions(models, case, monkeypatch):
    cfg, W, model = models(case, "float32")
    fm = importlib.import_module(PKG + ".float_model")
    monkeypatch.setattr(fm, "MAX_STEP_TOKENS", 100)
    rows = [tokens_of(cfg, 130, 70 + b) for b in range(2)]
    slots = model.begin_batch(2)
    want = [5, 129, 130 + 49, 130 + 50, 3]
    got = model.step(torch.tensor(rows), 0, slots, want=want)[0].cpu().numpy()
    model.end_batch(slots)
    ref = [fc.Expected(cfg, W, r) for r in rows]
    for g, w in zip(got, want):
        assert ref[w // 130].ok(g[None], "float32", [w % 130])
    slots = model.begin_batch(1)
    got = model.step(torch.tensor(rows[:1]), 0, slots)[0].cpu().numpy()
    model.end_batch(slots)
    assert ref[0].ok(got, "float32", [129])


def test_a_step_must_follow_what_the_slot_holds(models):
    cfg, W, model = models("WIDE", "bfloat16")
    cache = importlib.import_module(PKG + ".sequence_cache")
    slots = model.begin_batch(1)
    with pytest.raises(ValueError):
        model.step(torch.tensor([[1]]), 3, slots)
    with pytest.raises(cache.CacheFull):
        model.step(torch.tensor([[1] * 641]), 0, slots)
    model.end_batch(slots)
    with pytest.raises(RuntimeError):
        model.begin_batch(5)


# ---- generation and command lines -----------------------------------------------------------------------------------
def oracle_greedy(cfg, W, prompt, n):
    """greedy tokens and the smallest margin by which one was chosen"""
    toks, margin = list(prompt), np.inf
    for _ in range(n):
        l = np.sort(fc.oracle_logits(cfg, W, toks)[-1])
        margin = min(margin, (l[-1] - l[-2]) / l.std())
        toks.append(int(fc.oracle_logits(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):], margin


@pytest.mark.parametrize("case", ["ODD", "PEAKED", "V_ODD", "V_PEAKED"])
def test_greedy_generation_of_unequal_prompts(models, case):
    G = importlib.import_module(PKG + ".generate")
    cfg, W, model = models(case, "float32")
    prompts = [tokens_of(cfg, n, 80 + n) for n in (30, 1, 45)]
    trace = []
    out = G.generate(model, prompts, 12, eos_id=-5, trace=trace)
    assert trace[0]["pos"] == 1 and model.cache.free_slots() == model.cache.slots
    for p, got in zip(prompts, out):
        want, margin = oracle_greedy(cfg, W, p, 12)
        assert margin > 1e-4 and got == want
        assert G.generate(model, [p], 12, eos_id=-5) == [want]
    eos = out[0][4]
    stop = out[0].index(eos)
    assert G.generate(model, [prompts[0]], 12, eos_id=eos) == [out[0][:stop]]
    probe = []
    assert G.generate(model, [prompts[0]], 3, eos_id=-5, layer_probe=True, trace=probe) == [out[0][:3]]
    assert len(probe[0]["layer_tokens"]) == len(cfg["layers"])


@pytest.mark.parametrize("case", ["WIDE", "V_WIDE"])
def test_bfloat16_generation_follows_its_own_logits(models, case):
    G = importlib.import_module(PKG + ".generate")
    cfg, W, model = models(case, "bfloat16")
    prompt = tokens_of(cfg, 140, 90)
    out = G.generate(model, [prompt], 40, eos_id=-5)[0]
    logits = run(model, prompt + out)
    ref = fc.Expected(cfg, W, prompt + out)
    assert ref.ok(logits, "bfloat16")
    for i, t in enumerate(out):
        l = ref.logits[len(prompt) - 1 + i]
        assert l[t] > l.max() - 10 * ref.rounding.max() * l.std()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["ODD", "V_ODD"])
def test_trace_and_generate_programs(float_libpath, tmp_path, case, dtype):
    cfg = getattr(fc, case)
    W = fc.make_weights(cfg, 12)
    path = fc.write_checkpoint(str(tmp_path / "m"), cfg, W)
    out = tmp_path / "out"
    out.mkdir()
    reqs = {"a": tokens_of(cfg, 90, 1), "b": tokens_of(cfg, 70, 2)}
    lines, where, n = [], [], 0
    for rid, toks in reqs.items():
        at = 0
        for k in (50, 2, 17, 1, 1, 1, 30):
            k = min(k, len(toks) - at)
            if not k:
                break
            want = [0, k - 1] if n % 3 else []
            lines.append({"step": n, "entries": [{"id": rid, "tokens": toks[at:at + k], "want": want}],
                          "end": [rid] if at + k == len(toks) else []})
            where.append((rid, [at + w for w in want]))
            at += k
            n += 1
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "100"], input="\n".join(json.dumps(x) for x in lines) + "\n", text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done %d" % i for i in range(n)]
    ref = {k: fc.Expected(cfg, W, v) for k, v in reqs.items()}
    for i, (rid, pos) in enumerate(where):
        f = out / ("%d.f32" % i)
        assert f.exists() == bool(pos)
        if pos:
            assert ref[rid].ok(np.fromfile(f, dtype="<f4").reshape(len(pos), -1), dtype, pos)
    if dtype == "float32":
        prompt = reqs["a"][:20]
        r = subprocess.run([os.path.join(ROOT, "bin", "generate"), "--model", path, "--dtype", dtype, "--max-new-tokens", "6",
                            "--tokens", ",".join(map(str, prompt)), "--max-seq-len", "64"], text=True, capture_output=True,
                           timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert json.loads(r.stdout.strip().split("\n")[-1]) == oracle_greedy(cfg, W, prompt, 6)[0]
