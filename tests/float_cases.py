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


def bf16_round(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) >> 16 << 16
    return u.astype(np.uint32).view(np.float32)


def bf16_round_randomly(x, rng):
    """up or down with the probability that keeps the mean"""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + rng.integers(0, 1 << 16, u.shape, dtype=np.uint64)) >> 16 << 16
    return u.astype(np.uint32).view(np.float32)


def tensor_shapes(cfg):
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "final.norm": (w,)}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], "l%d." % i
        H, D, R, V, C, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
        out.update({p + "norm1": (w,), p + "mix.dq": (Q, w), p + "mix.dq.norm": (Q,), p + "mix.uq": (H * (D + R), Q),
                    p + "mix.uk": (H * D, C), p + "mix.uv": (H * V, C), p + "mix.g": (H * V, w), p + "mix.o": (w, H * V)})
        if m.get("kv_from") is None:
            out.update({p + "mix.dkv": (C + R, w), p + "mix.dkv.norm": (C,)})
        if L["mlp"] is not None:
            F = L["mlp"]["ff"]
            out.update({p + "norm2": (w,), p + "mlp.gate": (F, w), p + "mlp.up": (F, w), p + "mlp.down": (w, F)})
    return out


def make_weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        if "norm" in name:
            W[name] = bf16_round(1.0 + 0.3 * rng.standard_normal(shape))
        else:
            W[name] = bf16_round(rng.standard_normal(shape) * (1.0 if name == "embed" else shape[1] ** -0.5))
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
            return e.max() < 2e-5
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
