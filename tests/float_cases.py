"""Small seeded models of the floating-point decoder designs for the tests: configurations, weights, checkpoint
directories and comparisons.  Weights are rounded to bfloat16, so both number formats start from the same numbers."""
import json
import os

import numpy as np

from oracle import float_oracle as fo


def layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, ff, kv_from=None, base=5000.0, scale=None):
    mx = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
          "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "mask": {"size": window},
          "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mx, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, eps, layers):
    return {"architecture": "Munalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# sizes that are multiples of nothing, different heads / windows / value sizes per layer, latents read by layers that
# are not neighbours, a layer without a feed-forward, windows of one token and beyond the prompt
ODD = config(101, 52, 1e-3, [
    layer(3, 20, 6, 12, 28, 36, 40, 44),
    layer(2, 24, 10, 9, 17, 22, 1, None),
    layer(5, 12, 6, 20, 30, 36, 67, 30, kv_from=0, scale=0.9),
    layer(1, 33, 10, 7, 12, 22, 1000, 21, kv_from=1),
])
# peaked attention (large scale): a window that is one token off shows
PEAKED = config(130, 72, 1e-5, [
    layer(4, 16, 8, 24, 40, 48, 64, 80, scale=0.7, base=100.0),
    layer(4, 16, 8, 16, 40, 48, 33, 96, kv_from=0, scale=0.7, base=100.0),
])
# sizes the tensor-core kernels take without padding, windows on tile borders and one off them
WIDE = config(264, 192, 1e-6, [
    layer(6, 32, 16, 48, 96, 112, 128, 256, scale=0.6),
    layer(8, 48, 16, 32, 64, 112, 129, 160, kv_from=0, scale=0.6),
    layer(2, 64, 32, 128, 48, 80, 63, None, base=20000.0, scale=0.6),
])


def parallel(heads, kv_heads, dim, rot_dims, window, r_heads, r_dim, r_vdim, r_rot, decay, ff, scale=None, base=5000.0,
             r_base=9000.0, left_scale=0.7, right_scale=1.1):
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff}, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window},
                 "rot": {"base": base, "dims": rot_dims}, "scale": dim ** -0.5 if scale is None else scale},
        "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": decay, "rot": {"base": r_base, "dims": r_rot}},
        "left_scale": left_scale, "right_scale": right_scale}}


def mamba2(heads, vdim, state, groups, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def vifelix(vocab, width, eps, scale, layers):
    return {"architecture": "Vifelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


# sizes that are multiples of nothing, norm groups that cut through heads, decays of 1 and almost 0, windows of one token and
# beyond the prompt, rotations of a part of the head, every kind of layer with and without a feed-forward
V_ODD = vifelix(103, 52, 1e-3, 3.5, [
    mamba2(3, 20, 12, 1, 3, 2),
    parallel(6, 2, 20, 12, 40, 3, 12, 28, 6, [0.9, 1.0, 0.01], 44),
    parallel(3, 3, 12, 12, 1, 1, 20, 9, 20, [0.97], None, left_scale=1.3, right_scale=0.4),
    mamba2(4, 10, 9, 2, 5, 10, 30),
    parallel(2, 1, 33, 4, 1000, 5, 10, 12, 2, [0.5, 0.8, 0.99, 0.999, 0.95], 21),
])
# peaked attention and slow decays: a window that is one token off or a lost state shows
V_PEAKED = vifelix(130, 72, 1e-5, 6.0, [
    parallel(4, 2, 24, 16, 64, 2, 16, 24, 16, [0.998, 0.96], 80, scale=0.9, base=100.0, r_base=200.0),
    mamba2(4, 24, 16, 4, 4, 1),
    parallel(4, 4, 16, 8, 33, 3, 24, 16, 12, [0.999, 0.9, 0.99], 96, scale=0.9, base=100.0, r_base=300.0),
])
# sizes the tensor-core kernels take without padding, windows on tile borders and one off them, wide states
V_WIDE = vifelix(264, 192, 1e-6, 9.0, [
    mamba2(4, 64, 128, 2, 4, 4, 160),
    parallel(8, 2, 64, 32, 128, 2, 128, 64, 128, [0.96875, 0.998046875], 256, scale=0.4),
    parallel(4, 4, 96, 96, 129, 1, 72, 136, 40, [0.9921875], None, scale=0.4, base=20000.0),
    mamba2(3, 72, 80, 3, 2, 3),
])
RECURRENT = ("V_ODD", "V_PEAKED", "V_WIDE")


def bf16_round(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) >> 16 << 16
    return u.astype(np.uint32).view(np.float32)


def bf16_round_randomly(x, rng):
    """up or down with the probability that keeps the mean"""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + rng.integers(0, 1 << 16, u.shape, dtype=np.uint64)) >> 16 << 16
    return u.astype(np.uint32).view(np.float32)


def latent_shapes(p, m, w):
    H, D, R, V, C, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
    out = {p + "dq": (Q, w), p + "dq.norm": (Q,), p + "uq": (H * (D + R), Q), p + "uk": (H * D, C), p + "uv": (H * V, C),
           p + "g": (H * V, w), p + "o": (w, H * V)}
    if m.get("kv_from") is None:
        out.update({p + "dkv": (C + R, w), p + "dkv.norm": (C,)})
    return out


def parallel_shapes(p, m, w):
    l, r = m["left"], m["right"]
    H, G, D, N, P = l["heads"], l["kv_heads"], l["dim"], r["heads"] * r["dim"], r["heads"] * r["vdim"]
    return {p + "left.q": (H * D, w), p + "left.q.b": (H * D,), p + "left.k": (G * D, w), p + "left.k.b": (G * D,),
            p + "left.q.norm": (D,), p + "left.k.norm": (D,), p + "left.g": (H * D, w), p + "left.o": (w, H * D),
            p + "right.q": (N, w), p + "right.k": (N, w), p + "right.v": (P, w), p + "right.g": (P, w), p + "right.o": (w, P)}


def mamba2_shapes(p, m, w):
    H, i, n = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
    return {p + "in": (2 * i + 2 * n + H, w), p + "conv": (i + 2 * n, m["conv"]), p + "conv.b": (i + 2 * n,), p + "dt_bias": (H,),
            p + "A_log": (H,), p + "D": (H,), p + "norm": (i,), p + "o": (w, i)}


MIXER_SHAPES = {"latent_attention": latent_shapes, "parallel": parallel_shapes, "mamba2": mamba2_shapes}


def tensor_shapes(cfg):
    w, both = cfg["width"], cfg["architecture"] == "Vifelix"
    out = {"embed": (cfg["vocab"], w), "final.norm": (w,)}
    if both:
        out["head"] = (cfg["vocab"], w)
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        out.update(MIXER_SHAPES[L["type"]](p + "mix.", L["mixer"], w))
        norms = ["norm1"] + (["norm2"] if L["mlp"] is not None else [])
        out.update({p + n + e: (w,) for n in norms for e in (("", "b") if both else ("",))})
        if L["mlp"] is not None:
            F = L["mlp"]["ff"]
            out.update({p + "mlp.gate": (F, w), p + "mlp.up": (F, w), p + "mlp.down": (w, F)})
            if both:
                out.update({p + "mlp.gate.b": (F,), p + "mlp.up.b": (F,), p + "mlp.down.b": (w,)})
    return out


def make_weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    W, both = {}, cfg["architecture"] == "Vifelix"
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if both and last in ("norm1", "norm1b", "norm2", "norm2b") or both and name == "final.norm":
            W[name] = bf16_round(0.3 * rng.standard_normal(shape))               # stored around zero
        elif "norm" in name or last == "D":
            W[name] = bf16_round(1.0 + 0.3 * rng.standard_normal(shape))
        elif last in ("A_log", "dt_bias"):
            W[name] = bf16_round(rng.uniform(-4.0, 0.5, shape))
        elif last == "b":
            W[name] = bf16_round(0.5 * rng.standard_normal(shape))
        elif name == "embed":
            W[name] = bf16_round(rng.standard_normal(shape) / cfg.get("embedding", {"scale": 1.0})["scale"])
        else:
            W[name] = bf16_round(rng.standard_normal(shape) * shape[1] ** -0.5)
    return W


def write_checkpoint(path, cfg, W):
    """config.json and model.safetensors with every tensor in bfloat16"""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, w in W.items():
        b = (np.ascontiguousarray(w, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(w.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(header).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h + b"".join(blobs))
    return path


def oracle_logits(cfg, W, tokens, layers_out=None, rnd=fo.exact):
    return fo.forward(cfg, {k: v.astype(np.float64) for k, v in W.items()}, tokens, layers_out, rnd)


def row_errors(got, want, spread):
    """root-mean-square difference of every row, mean taken off, over the spread of the wanted values"""
    d = np.asarray(got, dtype=np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / spread


class Expected:
    """The oracle's logits of one request and the error that bfloat16 rounding of the stored activations causes in
    them: some positions react a hundred times more than others (an attention output that nearly cancels is blown
    up by the norm behind it), so the limits follow that error instead of being one number."""

    def __init__(self, cfg, W, tokens):
        self.layers = []
        self.logits = oracle_logits(cfg, W, tokens, self.layers)
        self.spread = self.logits.std()
        rng = np.random.default_rng(99)
        self.rounding, self.layer_rounding = 0.0, [0.0] * len(self.layers)
        for k in range(5):                       # to nearest, then four random roundings: the worst of them per row
            rnd = bf16_round if k == 0 else lambda x: bf16_round_randomly(x, rng)
            layers = []
            got = oracle_logits(cfg, W, tokens, layers, lambda x: rnd(x).astype(np.float64))
            self.rounding = np.maximum(self.rounding, row_errors(got, self.logits, self.spread))
            self.layer_rounding = [np.maximum(e, row_errors(r, w, w.std()))
                                   for e, r, w in zip(self.layer_rounding, layers, self.layers)]

    @staticmethod
    def _check(e, rounding, dtype):
        if dtype == "float32":
            return e.max() < 4e-5
        # a row may be four times as far off as rounding puts it or the rows around the median, and the whole half
        # as far again as rounding does
        limit = 4 * np.maximum(rounding, np.median(rounding))
        return bool((e < limit).all() and np.sqrt((e * e).mean()) < 2 * np.sqrt((rounding * rounding).mean()) + 1e-3)

    def ok(self, got, dtype, positions=None):
        at = slice(None) if positions is None else list(positions)
        return self._check(row_errors(got, self.logits[at], self.spread), self.rounding[at], dtype)

    def layer_ok(self, i, got, dtype):
        w = self.layers[i]
        return self._check(row_errors(got, w, w.std()), self.layer_rounding[i], dtype)
