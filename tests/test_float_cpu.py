"""Host side of the floating-point decoder designs: oracle mechanisms, configuration, checkpoint reading, cache slots,
the generation loop and the trace protocol.  No GPU, no CUDA library."""
import copy
import importlib
import io
import json

import numpy as np
import pytest
import torch

import float_cases as fc
from conftest import PKG
from oracle import float_oracle as fo

cfgmod = importlib.import_module(PKG + ".float_config")
registry = importlib.import_module(PKG + ".registry")
cachemod = importlib.import_module(PKG + ".sequence_cache")


# ---- the oracle against hand-made cases ---------------------------------------------------------------------
def test_oracle_norm_rotation_and_window():
    x = np.array([[3.0, -4.0]])
    assert np.allclose(fo.rms_norm(x, np.array([2.0, 0.5]), 0.0), [[6 / np.sqrt(12.5), -2 / np.sqrt(12.5)]])
    assert np.allclose(fo.rms_norm(np.zeros((1, 2)), np.ones(2), 1e-6), 0)
    v = np.zeros((3, 4)); v[:, 0] = 1; v[:, 3] = 1
    r = fo.rotate_pairs(v, np.array([0.0, 1.0, 2.0]), 100.0)
    assert np.allclose(r[1], [np.cos(1), np.sin(1), -np.sin(0.1), np.cos(0.1)])
    assert np.allclose(r[0], v[0]) and np.allclose(r[2][:2], [np.cos(2), np.sin(2)])
    m = fo.window_mask(5, 2)
    assert m.sum(1).tolist() == [1, 2, 2, 2, 2] and m[4].tolist() == [False, False, False, True, True]


def test_oracle_score_depends_on_distance_only():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 6)), rng.standard_normal((1, 6))
    def dot(i, j):
        return (fo.rotate_pairs(q, np.array([float(i)]), 50.0) @ fo.rotate_pairs(k, np.array([float(j)]), 50.0).T).item()
    assert np.isclose(dot(9, 4), dot(105, 100)) and not np.isclose(dot(9, 4), dot(9, 5))


@pytest.mark.parametrize("case", ["ODD", "PEAKED", "WIDE"])
def test_oracle_is_causal_and_windowed(case):
    cfg = getattr(fc, case)
    W = fc.make_weights(cfg, 1)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 150)
    full = fc.oracle_logits(cfg, W, toks)
    assert np.allclose(full[:60], fc.oracle_logits(cfg, W, toks[:60]))
    reach = sum(L["mixer"]["mask"]["size"] - 1 for L in cfg["layers"])       # farthest token any layer stack sees
    if reach < 140:
        other = toks.copy(); other[0] = (other[0] + 1) % cfg["vocab"]
        got = fc.oracle_logits(cfg, W, other)
        assert np.allclose(got[reach + 1:], full[reach + 1:]) and not np.allclose(got[:40], full[:40])


@pytest.mark.parametrize("mistake", ["window", "rotation", "gate", "shared", "eps", "scale"])
def test_a_planted_mistake_is_beyond_the_limits(mistake, monkeypatch):
    """the weights of the cases are such that an error of one mechanism shows in the logits"""
    cfg = copy.deepcopy(fc.PEAKED)
    W = fc.make_weights(cfg, 3)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], 120)
    want = fc.Expected(cfg, W, toks)
    assert want.ok(want.logits, "float32") and want.ok(want.logits, "bfloat16")
    if mistake == "window":
        cfg["layers"][1]["mixer"]["mask"]["size"] += 1
    elif mistake == "rotation":
        cfg["layers"][0]["mixer"]["rot"]["base"] *= 1.5
        cfg["layers"][1]["mixer"]["rot"]["base"] *= 1.5
    elif mistake == "gate":
        monkeypatch.setattr(fo, "sigmoid", lambda z: np.ones_like(z) * 0.5 if z.shape[1] == 64 else 1 / (1 + np.exp(-z)))
    elif mistake == "shared":
        real = fo.latent_attention
        monkeypatch.setattr(fo, "latent_attention", lambda h, c, kr, *a: real(h, c, np.roll(kr, 1, 0), *a))
    elif mistake == "eps":
        cfg["norm"]["eps"] = 1.0
    else:
        cfg["layers"][0]["mixer"]["scale"] *= 1.3
    got = fc.oracle_logits(cfg, W, toks)
    assert not want.ok(got, "float32") and not want.ok(got, "bfloat16")


def test_oracle_half_rotation_and_its_order():
    rng = np.random.default_rng(1)
    x, pos = rng.standard_normal((4, 2, 10)), np.arange(4.0)
    r = fo.rotate_half(x, pos, 6, 50.0)
    assert np.array_equal(r[..., 6:], x[..., 6:]) and np.allclose(r[0], x[0])
    assert np.allclose(r[2, 0, 1], x[2, 0, 1] * np.cos(2 * 50 ** (-1 / 3)) - x[2, 0, 4] * np.sin(2 * 50 ** (-1 / 3)))
    # with the pairs side by side it is the other rotation
    order = [0, 3, 1, 4, 2, 5]
    assert np.allclose(fo.rotate_pairs(x[..., order], pos, 50.0), r[..., order])


def test_oracle_recurrences():
    rng = np.random.default_rng(2)
    q, k, v = (rng.standard_normal((6, n)) for n in (3, 3, 2))
    want = np.stack([sum(0.5 ** (t - j) * (q[t] @ k[j]) * v[j] for j in range(t + 1)) for t in range(6)])
    assert np.allclose(fo.decayed_sums(q, k, v, np.full(6, 0.5)), want)
    w, x = rng.standard_normal((2, 3)), rng.standard_normal((5, 2))
    y = fo.short_conv(x, w, [1.0, 2.0])
    assert np.allclose(y[0], [1, 2] + w[:, 2] * x[0]) and np.allclose(y[4], [1, 2] + (w * x[2:5].T).sum(1))
    assert np.allclose(fo.softplus(np.array([-800.0, 0.0, 800.0])), [0, np.log(2), 800])


@pytest.mark.parametrize("case", fc.RECURRENT)
def test_oracle_of_the_recurrent_design_is_causal(case):
    cfg = getattr(fc, case)
    W = fc.make_weights(cfg, 1)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 90)
    full = fc.oracle_logits(cfg, W, toks)
    assert np.allclose(full[:40], fc.oracle_logits(cfg, W, toks[:40]))


PLANTED = ["window", "rotation", "left_rotation_part", "key_groups", "gate", "values", "key_bias", "left_scale", "right_scale", "decay",
           "unit_norm", "state", "conv_order", "conv_bias", "conv_state", "groups", "gate_after_norm", "norm_groups", "skip", "step_bias",
           "offset", "outer_norm", "embedding", "ff_bias", "head"]


@pytest.mark.parametrize("mistake", PLANTED)
def test_a_planted_mistake_in_the_recurrent_design_is_beyond_the_limits(mistake, monkeypatch):
    cfg = copy.deepcopy(fc.V_PEAKED)
    cfg["layers"][1]["mixer"]["norm_groups"] = 2
    W = fc.make_weights(cfg, 3)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], 120)
    want = fc.Expected(cfg, W, toks)
    assert want.ok(want.logits, "float32") and want.ok(want.logits, "bfloat16")
    mx = [L["mixer"] for L in cfg["layers"]]
    attention, sums, conv, norm = fo.key_valued_attention, fo.decayed_sums, fo.short_conv, fo.rms_norm
    if mistake == "window": mx[0]["left"]["mask"]["size"] += 1
    elif mistake == "rotation": mx[0]["right"]["rot"]["base"] *= 1.5
    elif mistake == "left_rotation_part": mx[0]["left"]["rot"]["dims"] = 24
    elif mistake == "key_groups":
        def swapped(h, V, p, m, *a):
            V = dict(V)
            order = np.arange(m["heads"] * m["dim"]).reshape(-1, m["heads"] // m["kv_heads"], m["dim"]).transpose(1, 0, 2).ravel()
            V[p + "q"], V[p + "q.b"] = V[p + "q"][order], V[p + "q.b"][order]
            return attention(h, V, p, m, *a)
        monkeypatch.setattr(fo, "key_valued_attention", swapped)
    elif mistake == "gate": W["l0.mix.left.g"][:] = 0
    elif mistake == "values":
        def normed(h, V, p, m, eps, rnd=fo.exact):
            V = dict(V)
            v = (h @ V[p + "k"].T + V[p + "k.b"]).reshape(len(h), m["kv_heads"], m["dim"])
            scale = 1 / np.sqrt((v * v).mean(-1).mean())
            V[p + "k"], V[p + "k.b"] = V[p + "k"] * scale, V[p + "k.b"] * scale
            return attention(h, V, p, m, eps, rnd)
        monkeypatch.setattr(fo, "key_valued_attention", normed)
    elif mistake == "key_bias": W["l0.mix.left.k.b"][:] = 0
    elif mistake in ("left_scale", "right_scale"): mx[0][mistake] *= 1.2
    elif mistake == "decay": mx[0]["right"]["decay"] = mx[0]["right"]["decay"][::-1]
    elif mistake == "unit_norm":
        monkeypatch.setattr(fo, "rms_norm", lambda x, w, eps: x if x.shape[1:] == (2, 24) else norm(x, w, eps))
    elif mistake == "state":                       # forgotten at a chunk's edge
        monkeypatch.setattr(fo, "decayed_sums", lambda q, k, v, d: np.concatenate(
            [sums(q[:64], k[:64], v[:64], d[:64]), sums(q[64:], k[64:], v[64:], d[64:])]))
    elif mistake == "conv_order": W["l1.mix.conv"] = W["l1.mix.conv"][:, ::-1]
    elif mistake == "conv_bias": W["l1.mix.conv.b"][:] = 0
    elif mistake == "conv_state":
        monkeypatch.setattr(fo, "short_conv", lambda x, w, b: np.concatenate([conv(x[:64], w, b), conv(x[64:], w, b)]))
    elif mistake == "groups":                      # B and C of another group
        i = mx[1]["heads"] * mx[1]["vdim"]
        n = mx[1]["groups"] * mx[1]["state"]
        W["l1.mix.in"][2 * i:2 * i + n] = np.roll(W["l1.mix.in"][2 * i:2 * i + n], mx[1]["state"], 0)
    elif mistake == "gate_after_norm":
        monkeypatch.setattr(fo, "gated_norm", lambda o, z, w, g, eps:
                            norm(o.reshape(len(o), g, -1), 1.0, eps).reshape(o.shape) * w * fo.silu(z))
    elif mistake == "norm_groups": mx[1]["norm_groups"] = 1
    elif mistake == "skip": W["l1.mix.D"][:] = 0
    elif mistake == "step_bias": W["l1.mix.dt_bias"][:] = 0
    elif mistake == "offset":
        for n in W:
            if n.endswith(("norm1", "norm1b", "norm2", "norm2b")): W[n] = W[n] - 1
    elif mistake == "outer_norm": W["l1.norm1b"][:] = 0
    elif mistake == "embedding": cfg["embedding"]["scale"] *= 1.3
    elif mistake == "ff_bias": W["l0.mlp.up.b"][:] = 0
    else: W["head"] = W["embed"]
    got = fc.oracle_logits(cfg, W, toks)
    assert not want.ok(got, "float32") and not want.ok(got, "bfloat16")


# ---- configuration and checkpoint ------------------------------------------------------------------------------
def test_config_is_read_per_layer():
    args = cfgmod.parse_config(fc.ODD)
    assert args.n_layers == 4 and args.vocab_size == 101 and args.dim == 52 and args.eps == 1e-3
    m = [l.mixer for l in args.layers]
    assert [x.window for x in m] == [40, 1, 67, 1000] and [x.heads for x in m] == [3, 2, 5, 1]
    assert [x.kv_from for x in m] == [None, None, 0, 1] and m[2].scale == 0.9
    assert args.layers[1].mlp is None and args.layers[0].mlp.ff == 44


def test_sizes_left_out_come_from_the_tensors():
    cfg = copy.deepcopy(fc.ODD)
    shapes = fc.tensor_shapes(cfg)
    for k in ("vocab", "width"):
        del cfg[k]
    for L in cfg["layers"]:
        for k in ("dim", "vdim", "q_rank", "kv_rank", "rot_dim"):
            del L["mixer"][k]
        if L["mlp"]:
            del L["mlp"]["ff"]
    assert cfgmod.parse_config(cfg, shapes) == cfgmod.parse_config(fc.ODD)
    with pytest.raises(cfgmod.ConfigError):
        cfgmod.parse_config(cfg)


def test_recurrent_config_is_read_per_layer():
    args = cfgmod.parse_config(fc.V_ODD)
    d = args.design
    assert (d.norm_placement, d.norm_offset, d.ff_bias, d.tied_output) == ("both", 1.0, True, False)
    assert args.embed_scale == 3.5 and [l.mixer_kind for l in args.layers] == ["mamba2", "parallel", "parallel", "mamba2", "parallel"]
    p, m = args.layers[1].mixer, args.layers[3].mixer
    assert (p.left.heads, p.left.kv_heads, p.left.dim, p.left.window, p.left.rot.dims, p.left.rot.layout) == (6, 2, 20, 40, 12, "half")
    assert p.right.decay == (0.9, 1.0, 0.01) and (p.right.dim, p.right.vdim) == (12, 28) and (p.left_scale, p.right_scale) == (0.7, 1.1)
    assert (m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups) == (4, 10, 9, 2, 5, 10)
    assert args.layers[2].mlp is None and args.layers[3].mlp == cfgmod.DenseConfig(30, True)
    # sizes left out come from the tensors
    cfg = copy.deepcopy(fc.V_ODD)
    shapes = fc.tensor_shapes(cfg)
    for k in ("vocab", "width"):
        del cfg[k]
    for L in cfg["layers"]:
        mx = L["mixer"]
        for part, keys in ((mx, ("vdim", "state", "conv", "heads")), (mx.get("left", {}), ("dim", "vdim", "heads", "kv_heads")),
                           (mx.get("right", {}), ("dim", "vdim", "heads"))):
            for k in keys:
                part.pop(k, None)
        if L["mlp"]:
            del L["mlp"]["ff"]
    assert cfgmod.parse_config(cfg, shapes) == args


@pytest.mark.parametrize("edit", ["kv_heads", "vdim", "rotation", "no_rotation", "decay", "decays", "groups", "norm_groups", "side"])
def test_bad_recurrent_configurations_are_refused(edit):
    cfg = copy.deepcopy(fc.V_ODD)
    p, m = cfg["layers"][1]["mixer"], cfg["layers"][3]["mixer"]
    if edit == "kv_heads": p["left"]["kv_heads"] = 4
    if edit == "vdim": p["left"]["vdim"] = 24
    if edit == "rotation": p["left"]["rot"]["dims"] = 22
    if edit == "no_rotation": p["right"]["rot"] = None
    if edit == "decay": p["right"]["decay"][0] = 1.5
    if edit == "decays": p["right"]["decay"] = [0.9]
    if edit == "groups": m["groups"] = 3
    if edit == "norm_groups": m["norm_groups"] = 7
    if edit == "side": del p["left"]
    with pytest.raises((cfgmod.ConfigError, KeyError)):
        cfgmod.parse_config(cfg)


@pytest.mark.parametrize("edit", ["arch", "mixer", "mlp", "forward_ref", "borrowed_ref", "rank", "rotation"])
def test_bad_configurations_are_refused(edit):
    cfg = copy.deepcopy(fc.ODD)
    m = [L["mixer"] for L in cfg["layers"]]
    if edit == "arch": cfg["architecture"] = "Nothing"
    if edit == "mixer": cfg["layers"][0]["type"] = "other"
    if edit == "mlp": cfg["layers"][0]["mlp"]["kind"] = "other"
    if edit == "forward_ref": m[0]["kv_from"] = 2
    if edit == "borrowed_ref": m[3]["kv_from"] = 2
    if edit == "rank": m[2]["kv_rank"] = 30
    if edit == "rotation": m[0]["rot"]["dims"] = 4
    with pytest.raises(cfgmod.ConfigError):
        cfgmod.parse_config(cfg)


def test_registry_names_every_design():
    assert registry.architecture_of({"architecture": "Munalorn"}) == "Munalorn"
    assert registry.architecture_of({"dim": 7168, "n_layers": 2}) == registry.INTEGER_MODEL
    assert set(registry.architectures()) == {"Munalorn", "Vifelix", registry.INTEGER_MODEL}
    with pytest.raises(cfgmod.ConfigError):
        registry.architecture_of({"architecture": "Else"})


def test_tensor_files_round_trip(tmp_path):
    W = fc.make_weights(fc.ODD, 5)
    fc.write_checkpoint(str(tmp_path), fc.ODD, W)
    files = registry.TensorFiles(str(tmp_path))
    assert files.shapes() == fc.tensor_shapes(fc.ODD)
    for n in ("embed", "l2.mix.uv", "l3.mlp.down"):
        assert np.array_equal(files(n, W[n].shape).float().numpy(), W[n])
    with pytest.raises(ValueError):
        files("embed", (100, 52))
    with pytest.raises(KeyError):
        files("l1.mlp.up", (1, 1))


# ---- cache slots -----------------------------------------------------------------------------------------------
def test_cache_slots_are_handed_out_and_taken_back():
    c = cachemod.SequenceCache([16, None, 24], [0, 0, 2], 2, 10, torch.float32, "cpu")
    assert c.buffer(1) is c.buffer(0) and c.buffer(2).shape == (2, 10, 24) and c.bytes() == 2 * 10 * 40 * 4
    a, b = c.acquire(), c.acquire()
    assert a != b and c.free_slots() == 0
    with pytest.raises(cachemod.CacheFull):
        c.acquire()
    c.extend(a, 0, 7)
    with pytest.raises(ValueError):
        c.extend(a, 6, 1)
    with pytest.raises(cachemod.CacheFull):
        c.extend(a, 7, 4)
    c.truncate(a, 3)
    c.extend(a, 3, 7)
    c.release(a)
    with pytest.raises(ValueError):
        c.release(a)
    assert c.acquire() == a and c.lengths[a] == 0
    with pytest.raises(ValueError):
        cachemod.SequenceCache([None, 16], [0, 1], 1, 4, torch.float32, "cpu")


def test_recurrent_state_has_a_block_per_slot():
    states = [{"sums": ((2, 8, 16), torch.float32)}, {}, {"sums": ((1, 8, 8), torch.float32), "conv": ((3, 40), torch.bfloat16)}]
    c = cachemod.SequenceCache([None, 16, None], [None, 1, None], 3, 10, torch.bfloat16, "cpu", states)
    assert c.state(0, "sums").shape == (3, 2, 8, 16) and c.state(2, "conv").dtype == torch.bfloat16
    assert c.bytes() == 3 * (10 * 16 * 2 + 2 * 8 * 16 * 4 + 64 * 4 + 120 * 2)
    s = c.acquire()
    c.extend(s, 0, 7)
    with pytest.raises(ValueError):                 # a state cannot go back in part
        c.truncate(s, 3)
    c.truncate(s, 7)
    c.truncate(s, 0)
    c.extend(s, 0, 2)


# ---- the loops that drive a model --------------------------------------------------------------------------------
class FakeModel:
    """counts: the next token is the sum of everything a slot has seen, modulo the vocabulary"""

    class args:
        max_seq_len, vocab_size, n_layers = 64, 50, 0

    device = torch.device("cpu")

    def __init__(self, slots=4):
        self.free, self.seen, self.calls = list(range(slots)), {}, []

    def begin_batch(self, n):
        got = [self.free.pop() for _ in range(n)]
        for s in got:
            self.seen[s] = []
        return got

    def end_batch(self, slots):
        self.free += slots

    def step(self, tokens, start, slots, want=None, layer_probe=False):
        self.calls.append((tokens.shape[1], start))
        out = []
        for b, s in enumerate(slots):
            assert len(self.seen[s]) == start
            for t in tokens[b].tolist():
                self.seen[s].append(t)
                out.append(torch.nn.functional.one_hot(torch.tensor(sum(self.seen[s]) % 50), 50).float())
        S = tokens.shape[1]
        rows = [b * S + S - 1 for b in range(len(slots))] if want is None else want
        return torch.stack([out[r] for r in rows]) if rows else torch.empty(0, 50), {}


def test_generation_loop_on_a_counting_model():
    G = importlib.import_module(PKG + ".generate")
    m = FakeModel()
    out = G.generate(m, [[1, 2, 3], [5]], 3, eos_id=-7)
    assert out == [[6, 12, 24], [5, 10, 20]] and len(m.free) == 4
    assert m.calls[0] == (1, 0)
    assert G.generate(m, [[1, 2, 3]], 5, eos_id=24) == [[6, 12]] and len(m.free) == 4


def test_trace_protocol(tmp_path):
    T = importlib.import_module(PKG + ".trace")
    m, replies = FakeModel(2), []
    lines = [json.dumps(s) for s in (
        {"step": 0, "entries": [{"id": "a", "tokens": [5, 7], "want": [0, 1]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": [1], "want": []}], "end": ["a"]},
        {"step": 2, "entries": [{"id": "b", "tokens": [9, 9, 9], "want": [2]}], "end": ["b"]})]
    T.run(m, io.StringIO("\n".join(lines) + "\n"), str(tmp_path), replies.append)
    assert replies == ["done 0", "done 1", "done 2"] and len(m.free) == 2
    assert sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "2.f32"]
    a = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, 50)
    assert a.argmax(1).tolist() == [5, 12]
    assert np.fromfile(tmp_path / "2.f32", dtype="<f4").argmax() == 27
    with pytest.raises(ValueError):
        T.run(m, [json.dumps({"step": 3, "entries": [{"id": "c", "tokens": [50], "want": []}], "end": []})],
              str(tmp_path), replies.append)
