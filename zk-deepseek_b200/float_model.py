"""Floating-point decoder modules on the B200 kernels: the building blocks of the designs in `float_config.DESIGNS`
and the model that strings them together.

Number formats.  In bfloat16 mode weights, activations that enter a matrix product and the cache are bfloat16, every
product accumulates in 32-bit, and the residual stream, norms, rotations, attention scores and softmax are 32-bit.  In
float32 mode everything is, without reduced-precision products.

Layouts.  Every size is padded to a multiple of 8 when the weights are prepared, per head where a head has its own
size, and padding holds zeros, so kernels only see aligned rows:
    dq | dkv        one stacked product [q_rank | kv_rank | rot_dim]; a layer without a key/value projection has dq only
    uq              per head [dim | rot_dim]; the rotation is its epilogue
    uk | uv         stacked, so that the expanded keys and values of a context are one product
    gate | up       rows interleaved; silu(gate) * up is the epilogue

    mixers of several projections    one stacked product, see `StackedMixer`
    rotated heads whose pairs lie half a rotation apart    reordered to adjacent pairs in every tensor that meets them

Latent attention has two forms with the same result.  A step with few tokens works on the latents themselves: the queries go
through W_uk^T, attention reads the cache rows of the window once for all heads, and the result goes through W_uv.
A step with many tokens expands the latents of its context to per-head keys and values first.
"""
import math

import torch
from torch import nn

try:
    from . import float_kernel as K
    from .sequence_cache import SequenceCache
except ImportError:  # pragma: no cover - this directory first on sys.path
    import float_kernel as K
    from sequence_cache import SequenceCache

# a step with at most this many tokens per sequence takes the decode form of attention: over the latents themselves, or over
# chunks of the cached keys side by side; a longer one the prefill form
ABSORB_MAX_TOKENS = 16
# a step with more rows than this is run in portions (bounds the activations and the expanded keys and values)
MAX_STEP_TOKENS = 8192


def _padded(t, shape, dtype, device):
    """t in the corner of a zero tensor"""
    out = torch.zeros(shape, dtype=dtype, device=device)
    out[tuple(slice(0, n) for n in t.shape)] = t.to(device=device, dtype=dtype)
    return out


def rotary_table(rot, positions, device):
    """(cos, sin) of p * base^(-2i/dims) as float32 [positions, dims / 2, 2], computed in float64"""
    i = torch.arange(rot.dims // 2, dtype=torch.float64)
    ang = torch.outer(torch.arange(positions, dtype=torch.float64), float(rot.base) ** (-2.0 * i / rot.dims))
    return torch.stack((ang.cos(), ang.sin()), dim=-1).to(device=device, dtype=torch.float32).contiguous()


class Step:
    """What the layers need to know about the step that is running."""

    def __init__(self, batch, seq, start_pos, start, slots, host_slots, cache):
        self.batch, self.seq, self.rows = batch, seq, batch * seq
        self.start_pos = start_pos        # None in a recorded step
        self.start, self.slots = start, slots          # device int32 [batch]
        self.host_slots, self.cache = host_slots, cache
        # most keys any query of this step could see
        self.bound = start_pos + seq if start_pos is not None else cache.capacity


class RMSNorm(nn.Module):
    """x / rms(x) * (offset + stored weight)"""

    def __init__(self, dim, eps, offset=0.0):
        super().__init__()
        self.dim, self.eps, self.offset = dim, eps, offset
        self.register_buffer("weight", None)

    def load(self, w, device):
        self.weight = _padded(w.float() + self.offset, (K.pad8(self.dim),), torch.float32, device)

    def forward(self, x, out, index=None):
        K.norm_rows(x, index, self.weight, out, self.dim, self.eps)
        return out

    def add_to(self, x, y, h, then=None):
        """x += norm(y); h (if not None) = x in h's format, or then(x) for another norm `then`"""
        K.add_norm(x, y, self.weight, h, self.dim, self.eps, None if then is None else then.weight)


class LatentAttention(nn.Module):
    def __init__(self, layer_id, args, cfg):
        super().__init__()
        self.layer_id, self.cfg, self.dim = layer_id, cfg, args.dim
        self.eps = args.eps
        self.own_kv = cfg.kv_from is None
        self.d, self.r, self.v = K.pad8(cfg.dim), K.pad8(cfg.rot_dim), K.pad8(cfg.vdim)
        self.c, self.q = K.pad8(cfg.kv_rank), K.pad8(cfg.q_rank)
        self.pitch = self.c + self.r
        self.pairs = cfg.rot_dim // 2
        for n in ("w_down", "w_uq", "w_ukv", "w_g", "w_o", "q_norm", "kv_norm", "table"):
            self.register_buffer(n, None)

    @staticmethod
    def tensors(prefix, cfg):
        names = ["dq", "dq.norm", "uq", "uk", "uv", "g", "o"] + (["dkv", "dkv.norm"] if cfg.kv_from is None else [])
        return [prefix + "mix." + n for n in names]

    def load(self, W, prefix, dtype, device, tables):
        c, p = self.cfg, prefix + "mix."
        H, width = c.heads, K.pad8(self.dim)
        rows = self.q + (self.c + self.r if self.own_kv else 0)
        w = torch.zeros(rows, width, dtype=dtype, device=device)
        w[:c.q_rank, :self.dim] = W(p + "dq", (c.q_rank, self.dim))
        self.q_norm = _padded(W(p + "dq.norm", (c.q_rank,)), (self.q,), torch.float32, device)
        if self.own_kv:
            dkv = W(p + "dkv", (c.kv_rank + c.rot_dim, self.dim))
            w[self.q:self.q + c.kv_rank, :self.dim] = dkv[:c.kv_rank]
            w[self.q + self.c:self.q + self.c + c.rot_dim, :self.dim] = dkv[c.kv_rank:]
            self.kv_norm = _padded(W(p + "dkv.norm", (c.kv_rank,)), (self.c,), torch.float32, device)
        self.w_down = w
        uq = W(p + "uq", (H * (c.dim + c.rot_dim), c.q_rank)).view(H, c.dim + c.rot_dim, c.q_rank)
        w = torch.zeros(H, self.d + self.r, self.q, dtype=dtype, device=device)
        w[:, :c.dim, :c.q_rank] = uq[:, :c.dim]
        w[:, self.d:self.d + c.rot_dim, :c.q_rank] = uq[:, c.dim:]
        self.w_uq = w.view(H * (self.d + self.r), self.q)
        w = torch.zeros(H * (self.d + self.v), self.c, dtype=dtype, device=device)
        w[:H * self.d].view(H, self.d, self.c)[:, :c.dim, :c.kv_rank] = \
            W(p + "uk", (H * c.dim, c.kv_rank)).view(H, c.dim, c.kv_rank)
        w[H * self.d:].view(H, self.v, self.c)[:, :c.vdim, :c.kv_rank] = \
            W(p + "uv", (H * c.vdim, c.kv_rank)).view(H, c.vdim, c.kv_rank)
        self.w_ukv = w
        w = torch.zeros(H, self.v, width, dtype=dtype, device=device)
        w[:, :c.vdim, :self.dim] = W(p + "g", (H * c.vdim, self.dim)).view(H, c.vdim, self.dim)
        self.w_g = w.view(H * self.v, width)
        w = torch.zeros(width, H, self.v, dtype=dtype, device=device)
        w[:self.dim, :, :c.vdim] = W(p + "o", (self.dim, H * c.vdim)).view(self.dim, H, c.vdim)
        self.w_o = w.view(width, H * self.v)
        self.table = tables(c.rot)

    def cache_pitch(self):
        return self.pitch if self.own_kv else None

    def cache_owner(self):
        return self.layer_id if self.own_kv else self.cfg.kv_from

    def state_shapes(self, dtype):
        return {}

    def forward(self, h, st):
        """h [rows, width] activations -> [rows, width] float32"""
        c, dt, dev = self.cfg, h.dtype, h.device
        y = torch.empty(st.rows, self.w_down.shape[0], dtype=torch.float32, device=dev)
        K.linear(h, self.w_down, y)
        cq = torch.empty(st.rows, self.q, dtype=dt, device=dev)
        cache = st.cache.buffer(self.layer_id)
        a = K.LatentArgs(y.data_ptr(), self.q_norm.data_ptr(), K.ptr(self.kv_norm), cq.data_ptr(), cache.data_ptr(),
                         self.table.data_ptr(), st.start.data_ptr(), st.slots.data_ptr(), y.stride(0), cq.stride(0),
                         st.rows, st.seq, cache.stride(0), cache.stride(1), cache.shape[1], c.q_rank, self.q,
                         c.kv_rank, self.c, self.pairs, int(self.own_kv), K.code(dt), self.eps)
        K.latent_post(a, y, cq, cache, self.q_norm, self.kv_norm, self.table, st.start, st.slots)
        q = torch.empty(st.rows, c.heads, self.d + self.r, dtype=dt, device=dev)
        K.linear(cq, self.w_uq, q.view(st.rows, -1), K.ROTATE, table=self.table, start=st.start, seq=st.seq,
                 pairs=self.pairs, period=self.d + self.r, offset=self.d)
        o = self._absorbed(q, cache, st) if st.seq <= ABSORB_MAX_TOKENS else self._expanded(q, cache, st)
        o = o.view(st.rows, c.heads * self.v)
        og = torch.empty_like(o)
        K.linear(h, self.w_g, og, K.GATE, aux=o)
        out = torch.empty(st.rows, self.w_o.shape[0], dtype=torch.float32, device=dev)
        return K.linear(og, self.w_o, out)

    def _absorbed(self, q, cache, st):
        c, dt, dev, H = self.cfg, q.dtype, q.device, self.cfg.heads
        uk = self.w_ukv[:H * self.d].view(H, self.d, self.c)
        uv = self.w_ukv[H * self.d:].view(H, self.v, self.c)
        qa = torch.empty(st.rows, H, self.pitch, dtype=dt, device=dev)
        K.perhead(q, uk, qa, True, copy=(self.d, self.c, self.r))
        lat = torch.empty(st.rows, H, self.c, dtype=dt, device=dev)
        bound = min(st.bound, c.window + st.seq - 1) if c.window else st.bound
        base, es = cache.data_ptr(), cache.element_size()
        a = K.AttentionArgs(qa.data_ptr(), base, base + self.c * es, base, lat.data_ptr(), st.start.data_ptr(),
                            st.slots.data_ptr(), None, self.pitch, self.c, self.pitch, 0, self.pitch, self.pitch, 0,
                            cache.stride(0), 0, cache.shape[1], st.batch, st.seq, H, self.c, self.r, self.c, c.window,
                            1, K.code(dt), c.scale, bound)
        n = K.attention_scratch(a)
        scratch = torch.empty(n, dtype=torch.float32, device=dev) if n else None
        a.scratch = K.ptr(scratch)
        K.attention(a, qa, lat, cache, scratch, st.start, st.slots)
        o = torch.empty(st.rows, H, self.v, dtype=dt, device=dev)
        K.perhead(lat, uv, o, False)
        return o

    def _expanded(self, q, cache, st):
        c, dt, dev, H = self.cfg, q.dtype, q.device, self.cfg.heads
        o = torch.empty(st.rows, H, self.v, dtype=dt, device=dev)
        base = max(0, st.start_pos - c.window + 1) if c.window else 0
        keys = st.start_pos + st.seq - base
        kv = torch.empty(keys, H * (self.d + self.v), dtype=dt, device=dev)
        es = cache.element_size()
        for b in range(st.batch):
            rows = cache[st.host_slots[b], base:base + keys]
            K.linear(rows[:, :self.c], self.w_ukv, kv)
            qb, ob = q[b * st.seq:], o[b * st.seq:]
            a = K.AttentionArgs(qb.data_ptr(), kv.data_ptr(), rows.data_ptr() + self.c * es,
                                kv.data_ptr() + H * self.d * es, ob.data_ptr(), st.start.data_ptr() + 4 * b, None,
                                None, self.d + self.r, self.v, kv.stride(0), self.d, self.pitch, kv.stride(0), self.v,
                                0, base, keys, 1, st.seq, H, self.d, self.r, self.v, c.window, 0, K.code(dt), c.scale,
                                keys)
            K.attention(a)
        return o


def _rotation_order(rot, dim, device="cpu"):
    """positions of a head's elements with the rotated pairs adjacent"""
    order = torch.arange(dim, device=device)
    if rot.layout == "half":
        half = rot.dims // 2
        order[0:rot.dims:2] = torch.arange(half, device=device)
        order[1:rot.dims:2] = torch.arange(half, device=device) + half
    return order


class StackedMixer(nn.Module):
    """A mixer that is one product, a core and one product: every projection of the input is a row range of `w_in`, the
    core turns the projected rows y (and y32, its last columns in 32-bit) into gated activations, `w_o` projects them.

    Subclasses give `cols`, `cols32` and `out_cols` (all multiples of 8; y is padded to a multiple of 32 when there are
    32-bit columns), write their weights in `fill` and run the core in `mix`.  `rotation` names the columns of y that
    turn in the product's epilogue: (begin, end, period, Rotary)."""
    cols32 = 0
    rotation = None

    def __init__(self, layer_id, args, cfg):
        super().__init__()
        self.layer_id, self.cfg, self.dim, self.eps = layer_id, cfg, args.dim, args.eps
        for n in ("w_in", "bias", "w_o", "table"):
            self.register_buffer(n, None)

    def load(self, W, prefix, dtype, device, tables):
        width = K.pad8(self.dim)
        self.n = self.cols if not self.cols32 else (self.cols + 31) // 32 * 32
        self.w_in = torch.zeros(self.n + self.cols32, width, dtype=dtype, device=device)
        bias = torch.zeros(self.w_in.shape[0], dtype=torch.float32, device=device)
        self.w_o = torch.zeros(width, self.out_cols, dtype=dtype, device=device)
        self.fill(W, prefix + "mix.", self.w_in[:self.n], self.w_in[self.n:], bias[:self.n], self.w_o, tables)
        self.bias = bias if self.biased else None
        if self.rotation is not None:
            self.table = tables(self.rotation[3])

    biased = False

    def cache_pitch(self):
        return None

    def cache_owner(self):
        return self.layer_id if self.cache_pitch() is not None else None

    def state_shapes(self, dtype):
        return {}

    def _rows(self, t, heads, size, pad, order=None):
        """t [heads * size, ...] as [heads, pad, ...] zero-padded, elements of a head in `order`"""
        t = t.view((heads, size) + t.shape[1:])
        if order is not None:
            t = t[:, order]
        out = torch.zeros((heads, pad) + t.shape[2:], dtype=t.dtype, device=t.device)
        out[:, :size] = t
        return out.view((heads * pad,) + t.shape[2:])

    def _put(self, w, begin, t, heads, size, pad, order=None):
        """projection rows t [heads * size, dim] into w from row `begin`; returns the next free row"""
        end = begin + heads * pad
        w[begin:end, :self.dim] = self._rows(t, heads, size, pad, order).to(w.device, w.dtype)
        return end

    def _put_out(self, w_o, t, heads, size, pad, order=None):
        """output weights t [dim, heads * size] into w_o"""
        w_o[:self.dim] = self._rows(t.t().contiguous(), heads, size, pad, order).t().to(w_o.device, w_o.dtype)

    def forward(self, h, st):
        """h [rows, width] activations -> [rows, width] float32"""
        dt, dev = h.dtype, h.device
        y = torch.empty(st.rows, self.n, dtype=dt, device=dev)
        y32 = torch.empty(st.rows, self.cols32, dtype=torch.float32, device=dev) if self.cols32 else None
        kw = {}
        if self.rotation is not None:
            begin, end, period, rot = self.rotation
            kw = dict(epilogue=K.ROTATE, table=self.table, start=st.start, seq=st.seq, pairs=rot.dims // 2, period=period,
                      rotated=(begin, end))
        K.linear(h, self.w_in, y, bias=self.bias, out2=y32, **kw)
        act = torch.empty(st.rows, self.out_cols, dtype=dt, device=dev)
        self.mix(y, y32, act, st)
        out = torch.empty(st.rows, self.w_o.shape[0], dtype=torch.float32, device=dev)
        return K.linear(act, self.w_o, out)


class KeyValuedAttention(StackedMixer):
    """Grouped softmax attention over a window; the values are the projected keys before norm and rotation, queries and
    keys are normed per head, the output is gated.  y: [q | k | gate]; cache rows: keys of all key heads, then values."""
    biased = True
    out_scale = 1.0

    def __init__(self, layer_id, args, cfg):
        super().__init__(layer_id, args, cfg)
        self.d = K.pad8(cfg.dim)
        self.q_cols, self.k_cols = cfg.heads * self.d, cfg.kv_heads * self.d
        self.cols, self.out_cols = 2 * self.q_cols + self.k_cols, self.q_cols
        for n in ("q_norm", "k_norm", "rot_table"):
            self.register_buffer(n, None)

    @staticmethod
    def names(p, cfg):
        return [p + n for n in ("q", "q.b", "k", "k.b", "q.norm", "k.norm", "g", "o")]

    def fill(self, W, p, w, w32, bias, w_o, tables):
        c, d, dim = self.cfg, self.d, self.cfg.dim
        order = _rotation_order(c.rot, dim)
        H, G = c.heads, c.kv_heads
        for begin, name, heads in ((0, "q", H), (self.q_cols, "k", G)):
            end = self._put(w, begin, W(p + name, (heads * dim, self.dim)), heads, dim, d, order)
            bias[begin:end] = self._rows(W(p + name + ".b", (heads * dim,)), heads, dim, d, order).to(bias.device, bias.dtype)
        self._put(w, end, W(p + "g", (H * dim, self.dim)), H, dim, d, order)
        self._put_out(w_o, W(p + "o", (self.dim, H * dim)), H, dim, d, order)
        norm = lambda n: _padded(W(p + n, (dim,))[order], (d,), torch.float32, w.device)
        self.q_norm, self.k_norm = norm("q.norm"), norm("k.norm")
        self.rot_table = tables(c.rot)

    def cache_pitch(self):
        return 2 * self.k_cols

    def mix(self, y, y32, out, st):
        c, dt, d = self.cfg, y.dtype, self.d
        cache = st.cache.buffer(self.layer_id)
        q = torch.empty(st.rows, c.heads, d, dtype=dt, device=y.device)
        a = K.HeadsArgs(y.data_ptr(), self.q_norm.data_ptr(), self.k_norm.data_ptr(), q.data_ptr(), cache.data_ptr(),
                        self.rot_table.data_ptr(), st.start.data_ptr(), st.slots.data_ptr(), y.stride(0), 0, self.q_cols,
                        st.rows, st.seq, cache.stride(0), cache.stride(1), cache.shape[1], c.heads, c.kv_heads, d, c.dim,
                        c.rot.dims // 2, K.code(dt), self.eps)
        K.heads_post(a, y, q, cache, self.q_norm, self.k_norm, self.rot_table, st.start, st.slots)
        gate = y[:, self.q_cols + self.k_cols:]
        es = y.element_size()
        if st.seq <= ABSORB_MAX_TOKENS:
            bound = min(st.bound, c.window + st.seq - 1) if c.window else st.bound
            a = K.GroupedArgs(q.data_ptr(), cache.data_ptr(), out.data_ptr(), gate.data_ptr(), st.start.data_ptr(),
                              st.slots.data_ptr(), None, cache.stride(0), cache.stride(1), cache.shape[1], self.k_cols,
                              out.stride(0), y.stride(0), st.batch, st.seq, c.heads, c.kv_heads, d, c.window, bound,
                              K.code(dt), c.scale, self.out_scale)
            K.grouped_attention(a, y.device, q, cache, out, y, st.start, st.slots)
            return
        base = max(0, st.start_pos - c.window + 1) if c.window else 0
        keys = st.start_pos + st.seq - base
        for b in range(st.batch):
            rows = cache[st.host_slots[b], base:base + keys]
            k, v = rows.data_ptr(), rows.data_ptr() + self.k_cols * es
            a = K.AttentionArgs(q[b * st.seq:].data_ptr(), k, k, v, out[b * st.seq:].data_ptr(), st.start.data_ptr() + 4 * b,
                                None, None, d, d, rows.stride(0), d, rows.stride(0), rows.stride(0), d, 0, base, keys, 1,
                                st.seq, c.heads, d, 0, d, c.window, 0, K.code(dt), c.scale, keys, c.heads // c.kv_heads,
                                gate[b * st.seq:].data_ptr(), y.stride(0), d, out.stride(0), self.out_scale)
            K.attention(a)


class Retention(StackedMixer):
    """Linear attention with a fixed decay per head; heads at unit root mean square, silu gate.  y: [q | k | v | gate]"""
    out_scale = 1.0

    def __init__(self, layer_id, args, cfg):
        super().__init__(layer_id, args, cfg)
        self.nd, self.p = K.pad8(cfg.dim), K.pad8(cfg.vdim)
        self.qk_cols, self.v_cols = cfg.heads * self.nd, cfg.heads * self.p
        self.cols, self.out_cols = 2 * (self.qk_cols + self.v_cols), self.v_cols
        self.rotation = (0, 2 * self.qk_cols, self.nd, cfg.rot)
        self.register_buffer("decay", None)

    @staticmethod
    def names(p, cfg):
        return [p + n for n in ("q", "k", "v", "g", "o")]

    def fill(self, W, p, w, w32, bias, w_o, tables):
        c, order = self.cfg, _rotation_order(self.cfg.rot, self.cfg.dim)
        at = 0
        for name, size, pad, o in (("q", c.dim, self.nd, order), ("k", c.dim, self.nd, order), ("v", c.vdim, self.p, None),
                                   ("g", c.vdim, self.p, None)):
            at = self._put(w, at, W(p + name, (c.heads * size, self.dim)), c.heads, size, pad, o)
        self._put_out(w_o, W(p + "o", (self.dim, c.heads * c.vdim)), c.heads, c.vdim, self.p)
        self.decay = torch.tensor(c.decay, dtype=torch.float32, device=w.device)

    def state_shapes(self, dtype):
        return {"sums": ((self.cfg.heads, self.nd, self.p), torch.float32)}

    def mix(self, y, y32, out, st):
        c, dt = self.cfg, y.dtype
        S = st.cache.state(self.layer_id, "sums")
        o = torch.empty(st.rows, self.v_cols, dtype=dt, device=y.device)
        es, tok = y.element_size(), y.stride(0)
        a = K.ScanArgs(y.data_ptr(), y.data_ptr() + self.qk_cols * es, y.data_ptr() + 2 * self.qk_cols * es, o.data_ptr(),
                       self.decay.data_ptr(), None, None, None, S.data_ptr(), None, st.start.data_ptr(), st.slots.data_ptr(),
                       tok, tok, tok, o.stride(0), self.nd, self.p, self.p, 0, st.batch, st.seq, c.heads, S.shape[0], 1,
                       self.nd, self.p, K.code(dt), c.dim ** -0.5)
        K.scan(a, y.device, y, o, S, self.decay, st.start, st.slots)
        g = y[:, 2 * self.qk_cols + self.v_cols:]
        n = K.GatedNormArgs(o.data_ptr(), g.data_ptr(), None, out.data_ptr(), o.stride(0), tok, out.stride(0), st.rows,
                            c.heads, c.vdim, self.p, c.vdim, K.code(dt), self.out_scale, self.eps)
        K.gated_norm(n, o, y, out)


class Parallel(StackedMixer):
    """Two mixers on the same input, added with fixed weights: their projections are one product, their outputs lie side
    by side in the input of one output product, and the weights are applied where the parts are gated."""
    biased = True

    def __init__(self, layer_id, args, cfg):
        super().__init__(layer_id, args, cfg)
        self.left = KeyValuedAttention(layer_id, args, cfg.left)
        self.right = Retention(layer_id, args, cfg.right)
        self.left.out_scale, self.right.out_scale = cfg.left_scale, cfg.right_scale
        self.cols = self.left.cols + self.right.cols
        self.out_cols = self.left.out_cols + self.right.out_cols
        begin, end, period, rot = self.right.rotation
        self.rotation = (self.left.cols + begin, self.left.cols + end, period, rot)

    @staticmethod
    def tensors(prefix, cfg):
        return KeyValuedAttention.names(prefix + "mix.left.", cfg.left) + Retention.names(prefix + "mix.right.", cfg.right)

    def fill(self, W, p, w, w32, bias, w_o, tables):
        l, o = self.left.cols, self.left.out_cols
        self.left.fill(W, p + "left.", w[:l], None, bias[:l], w_o[:, :o], tables)
        self.right.fill(W, p + "right.", w[l:], None, bias[l:], w_o[:, o:], tables)

    def cache_pitch(self):
        return self.left.cache_pitch()

    def state_shapes(self, dtype):
        return self.right.state_shapes(dtype)

    def mix(self, y, y32, out, st):
        l, o = self.left.cols, self.left.out_cols
        self.left.mix(y[:, :l], None, out[:, :o], st)
        self.right.mix(y[:, l:], None, out[:, o:], st)


class Mamba2(StackedMixer):
    """State-space mixer: short convolution and silu on [x | B | C], a state per head that decays by the token's step
    size, gate and norm.  y: [z | x | B | C], y32: step sizes."""

    def __init__(self, layer_id, args, cfg):
        super().__init__(layer_id, args, cfg)
        self.p, self.nd = K.pad8(cfg.vdim), K.pad8(cfg.state)
        self.inner, self.bc = cfg.heads * self.p, cfg.groups * self.nd
        self.channels = self.inner + 2 * self.bc
        self.cols, self.cols32, self.out_cols = self.inner + self.channels, K.pad8(cfg.heads), self.inner
        for n in ("conv_w", "conv_b", "rate", "step_bias", "skip", "norm_w"):
            self.register_buffer(n, None)

    @staticmethod
    def tensors(prefix, cfg):
        return [prefix + "mix." + n for n in ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")]

    def _channels(self, t):
        """[x | B | C] rows of t, padded per head and group"""
        c = self.cfg
        i, n = c.heads * c.vdim, c.groups * c.state
        return torch.cat([self._rows(t[:i], c.heads, c.vdim, self.p), self._rows(t[i:i + n], c.groups, c.state, self.nd),
                          self._rows(t[i + n:i + 2 * n], c.groups, c.state, self.nd)])

    def fill(self, W, p, w, w32, bias, w_o, tables):
        c, dev = self.cfg, w.device
        i, n = c.heads * c.vdim, c.groups * c.state
        t = W(p + "in", (2 * i + 2 * n + c.heads, self.dim))
        at = self._put(w, 0, t[:i], c.heads, c.vdim, self.p)
        w[at:at + self.channels, :self.dim] = self._channels(t[i:2 * i + 2 * n]).to(dev, w.dtype)
        w32[:c.heads, :self.dim] = t[2 * i + 2 * n:].to(dev, w.dtype)
        f32 = lambda x: x.float().to(dev).contiguous()
        self.conv_w = f32(self._channels(W(p + "conv", (i + 2 * n, c.conv)))).t().contiguous()
        self.conv_b = f32(self._channels(W(p + "conv.b", (i + 2 * n,))))
        self.rate = f32(W(p + "A_log", (c.heads,)).double().exp())
        self.step_bias, self.skip = f32(W(p + "dt_bias", (c.heads,))), f32(W(p + "D", (c.heads,)))
        self.norm_w = f32(self._rows(W(p + "norm", (i,)), c.heads, c.vdim, self.p))
        self._put_out(w_o, W(p + "o", (self.dim, i)), c.heads, c.vdim, self.p)

    def state_shapes(self, dtype):
        return {"conv": ((self.cfg.conv - 1, self.channels), dtype),
                "sums": ((self.cfg.heads, self.nd, self.p), torch.float32)}

    def mix(self, y, y32, out, st):
        c, dt, es = self.cfg, y.dtype, y.element_size()
        conv, S = (st.cache.state(self.layer_id, n) for n in ("conv", "sums"))
        xbc = torch.empty(st.rows, self.channels, dtype=dt, device=y.device)
        a = K.ConvArgs(y.data_ptr() + self.inner * es, self.conv_w.data_ptr(), self.conv_b.data_ptr(), xbc.data_ptr(),
                       conv.data_ptr(), st.start.data_ptr(), st.slots.data_ptr(), y.stride(0), xbc.stride(0), st.batch,
                       st.seq, conv.shape[0], self.channels, c.conv, K.code(dt))
        K.short_conv(a, y, xbc, conv, self.conv_w, self.conv_b, st.start, st.slots)
        o = torch.empty(st.rows, self.inner, dtype=dt, device=y.device)
        x, tok = xbc.data_ptr(), xbc.stride(0)
        B = x + self.inner * es
        a = K.ScanArgs(B + self.bc * es, B, x, o.data_ptr(), self.rate.data_ptr(), y32.data_ptr(), self.step_bias.data_ptr(),
                       self.skip.data_ptr(), S.data_ptr(), None, st.start.data_ptr(), st.slots.data_ptr(), tok, tok, tok,
                       o.stride(0), self.nd, self.p, self.p, y32.stride(0), st.batch, st.seq, c.heads, S.shape[0],
                       c.heads // c.groups, self.nd, self.p, K.code(dt), 1.0)
        K.scan(a, y.device, xbc, o, y32, S, self.rate, self.step_bias, self.skip, st.start, st.slots)
        n = K.GatedNormArgs(o.data_ptr(), y.data_ptr(), self.norm_w.data_ptr(), out.data_ptr(), o.stride(0), y.stride(0),
                            out.stride(0), st.rows, c.heads, c.vdim, self.p, c.heads * c.vdim // c.norm_groups, K.code(dt),
                            1.0, self.eps)
        K.gated_norm(n, o, y, self.norm_w, out)


class DenseFF(nn.Module):
    """W_down (silu(W_gate h) * (W_up h)), each with a bias or none; gate and up rows are interleaved in one product"""

    def __init__(self, layer_id, args, cfg):
        super().__init__()
        self.dim, self.ff, self.biased = args.dim, cfg.ff, cfg.bias
        for n in ("w_gate_up", "w_down", "b_gate_up", "b_down"):
            self.register_buffer(n, None)

    @staticmethod
    def tensors(prefix, cfg):
        names = ["gate", "up", "down"]
        return [prefix + "mlp." + n for n in names + ([n + ".b" for n in names] if cfg.bias else [])]

    def load(self, W, prefix, dtype, device):
        p, width, ff = prefix + "mlp.", K.pad8(self.dim), K.pad8(self.ff)
        w = torch.zeros(ff, 2, width, dtype=dtype, device=device)
        w[:self.ff, 0, :self.dim] = W(p + "gate", (self.ff, self.dim))
        w[:self.ff, 1, :self.dim] = W(p + "up", (self.ff, self.dim))
        self.w_gate_up = w.view(2 * ff, width)
        self.w_down = _padded(W(p + "down", (self.dim, self.ff)), (width, ff), dtype, device)
        if self.biased:
            b = torch.zeros(ff, 2, dtype=torch.float32, device=device)
            b[:self.ff, 0], b[:self.ff, 1] = W(p + "gate.b", (self.ff,)), W(p + "up.b", (self.ff,))
            self.b_gate_up = b.view(2 * ff)
            self.b_down = _padded(W(p + "down.b", (self.dim,)), (width,), torch.float32, device)

    def forward(self, h, st=None):
        hid = torch.empty(h.shape[0], self.w_down.shape[1], dtype=h.dtype, device=h.device)
        K.linear(h, self.w_gate_up, hid, K.GLU, bias=self.b_gate_up)
        out = torch.empty(h.shape[0], self.w_down.shape[0], dtype=torch.float32, device=h.device)
        return K.linear(hid, self.w_down, out, bias=self.b_down)


MIXERS = {"latent_attention": LatentAttention, "parallel": Parallel, "mamba2": Mamba2}
FEEDFORWARDS = {"dense": DenseFF}


class DecoderLayer(nn.Module):
    """x <- x + N(f(x)) for the mixer and then the feed-forward, or x <- x + N(f(N'(x))) in designs with norms on both
    sides.  A sublayer's closing kernel also makes the next sublayer's input: x in the activations' format or N'(x)."""

    def __init__(self, layer_id, args, cfg):
        super().__init__()
        self.prefix = "l%d." % layer_id
        self.both = args.design.norm_placement == "both"
        self.mixer = MIXERS[cfg.mixer_kind](layer_id, args, cfg.mixer)
        self.ff = FEEDFORWARDS[cfg.mlp_kind](layer_id, args, cfg.mlp) if cfg.mlp_kind else None
        for n in self.norm_names():
            setattr(self, n, RMSNorm(args.dim, args.eps, args.design.norm_offset))
        self.following = []       # [the norm ahead of the next layer], not a submodule

    def norm_names(self):
        ends = ("", "b") if self.both else ("",)
        return ["norm%d%s" % (i, e) for i in ((1, 2) if self.ff is not None else (1,)) for e in ends]

    def load(self, W, dtype, device, tables):
        self.mixer.load(W, self.prefix, dtype, device, tables)
        if self.ff is not None:
            self.ff.load(W, self.prefix, dtype, device)
        for n in self.norm_names():
            norm = getattr(self, n)
            norm.load(W(self.prefix + n, (norm.dim,)), device)

    def forward(self, x, h, st):
        """x: residual stream, h: the input of the mixer (x itself where the formats agree and there is no norm)"""
        after = self.following[0] if self.following else None
        into = None if h is x or (self.both and after is None) else h
        if self.ff is None:
            (self.norm1b if self.both else self.norm1).add_to(x, self.mixer(h, st), into, after)
        elif self.both:
            self.norm1b.add_to(x, self.mixer(h, st), h, self.norm2)
            self.norm2b.add_to(x, self.ff(h, st), into, after)
        else:
            self.norm1.add_to(x, self.mixer(h, st), into)
            self.norm2.add_to(x, self.ff(h, st), into)


class FloatTransformer(nn.Module):
    """Embedding, layers, final norm and output projection of a floating-point decoder design.

    `step` runs the next tokens of a batch of sequences that stand at the same position; `begin_batch` /
    `end_batch` hand out and take back their cache slots.  The per-layer calls `prep_inference`,
    `layer_inference` and `finish_inference` have the shape of the integer model's.
    """

    def __init__(self, args, dtype=torch.bfloat16):
        super().__init__()
        if args.design.norm_placement not in ("output", "both") or args.design.activation != "silu":
            raise NotImplementedError("design %s" % args.design.name)
        self.args, self.dtype = args, dtype
        self.layers = nn.ModuleList([DecoderLayer(i, args, c) for i, c in enumerate(args.layers)])
        self.pre_norm = args.design.norm_placement == "both"
        if self.pre_norm:
            for layer, after in zip(self.layers, self.layers[1:]):
                layer.following.append(after.norm1)
        self.norm = RMSNorm(args.dim, args.eps, args.design.norm_offset)
        self.register_buffer("embed", None)
        self.register_buffer("head", None)
        self.cache = None
        self._tables = {}
        self._recorded = {}         # batch size -> recorded one-token step

    # -- weights and cache --------------------------------------------------------------------------
    def load_weights(self, W, device):
        """W(name, shape) returns a checked tensor"""
        args = self.args

        def tables(rot):
            key = rot.base, rot.dims
            if key not in self._tables:
                self._tables[key] = rotary_table(rot, args.max_seq_len, device)
            return self._tables[key]

        for layer in self.layers:
            layer.load(W, self.dtype, device, tables)
        self.norm.load(W("final.norm", (args.dim,)), device)
        shape, padded = (args.vocab_size, args.dim), (K.pad8(args.vocab_size), K.pad8(args.dim))
        self.embed = _padded(W("embed", shape), padded, self.dtype, device)
        self.head = self.embed if args.design.tied_output else _padded(W("head", shape), padded, self.dtype, device)
        mixers = [l.mixer for l in self.layers]
        self.cache = SequenceCache([m.cache_pitch() for m in mixers], [m.cache_owner() for m in mixers], args.max_batch_size,
                                   args.max_seq_len, self.dtype, device, [m.state_shapes(self.dtype) for m in mixers])
        return self

    def tensor_names(self):
        names = ["embed", "final.norm"] + ([] if self.args.design.tied_output else ["head"])
        for layer, cfg in zip(self.layers, self.args.layers):
            names += layer.mixer.tensors(layer.prefix, cfg.mixer) + [layer.prefix + n for n in layer.norm_names()]
            if layer.ff is not None:
                names += layer.ff.tensors(layer.prefix, cfg.mlp)
        return names

    @property
    def device(self):
        return self.embed.device

    def begin_batch(self, n):
        if n > self.cache.free_slots():
            raise RuntimeError("%d sequences, %d free cache slots" % (n, self.cache.free_slots()))
        return [self.cache.acquire() for _ in range(n)]

    def end_batch(self, slots):
        for s in slots:
            self.cache.release(s)

    # -- one step --------------------------------------------------------------------------------------
    def prep_inference(self, tokens, start_pos, slots):
        """(activations, step) of tokens [B, S] that follow position start_pos - 1 of the given slots"""
        B, S = tokens.shape
        for s in slots:
            self.cache.extend(s, start_pos, S)
        meta = torch.tensor([[start_pos] * B, list(slots)], dtype=torch.int32).to(self.device, non_blocking=True)
        st = Step(B, S, start_pos, meta[0], meta[1], list(slots), self.cache)
        return self._embed(tokens.to(self.device)), st

    def _embed(self, tokens):
        rows, pitch = tokens.numel(), self.embed.shape[1]
        x = torch.empty(rows, pitch, dtype=torch.float32, device=self.device)
        h = x if self.dtype == torch.float32 and not self.pre_norm else \
            torch.empty(rows, pitch, dtype=self.dtype, device=self.device)
        K.embed(tokens.contiguous().view(-1), self.embed, self.args.vocab_size, x, None if self.pre_norm or h is x else h,
                self.args.embed_scale)
        if self.pre_norm:
            self.layers[0].norm1(x, h)
        return x, h

    def layer_inference(self, layer_id, h, st):
        self.layers[layer_id](h[0], h[1], st)
        return h

    def finish_inference(self, h, st, want=None):
        """float32 logits [n, vocab] of the wanted rows (default: the last row of every sequence)"""
        if want is None:
            want = torch.arange(st.batch, dtype=torch.int32, device=self.device) * st.seq + (st.seq - 1)
        x = torch.empty(want.shape[0], self.embed.shape[1], dtype=self.dtype, device=self.device)
        self.norm(h[0], x, want)
        logits = torch.empty(want.shape[0], self.head.shape[0], dtype=torch.float32, device=self.device)
        return K.linear(x, self.head, logits)[:, :self.args.vocab_size]

    @torch.inference_mode()
    def step(self, tokens, start_pos, slots, want=None, layer_probe=False, layers_out=None):
        """Runs tokens [B, S] (int64) of the sequences in `slots`, all of which stand at start_pos.

        want: row numbers b * S + s whose logits are returned ([] for none); None takes the last of each sequence.
        Returns (logits, info): info["layer_tokens"] with `layer_probe`.  layers_out (a list) receives the residual
        stream after every layer.
        """
        B, S = tokens.shape
        info = {}
        if S == 1 and not layer_probe and layers_out is None and (want is None or len(want)):
            logits = self._decode(tokens, start_pos, slots)
            return (logits if want is None else logits[list(want)]), info
        limit = max(ABSORB_MAX_TOKENS + 1, MAX_STEP_TOKENS // B)
        if S > limit and layers_out is None and not layer_probe:
            out = []
            for s0 in range(0, S, limit):
                n = min(limit, S - s0)
                w = [] if s0 + n < S else None
                if want is not None:
                    w = [b * n + s - s0 for b, s in (divmod(r, S) for r in want) if s0 <= s < s0 + n]
                    out += [(r, s0) for r in want if s0 <= r % S < s0 + n]
                part = self.step(tokens[:, s0:s0 + n], start_pos + s0, slots, w)[0]
                if want is None:
                    logits = part
                else:
                    info.setdefault("parts", []).append(part)
            if want is None:
                return logits, {}
            parts = torch.cat(info.pop("parts"))
            order = [r for r, _ in out]
            return parts[[order.index(r) for r in want]], info
        h, st = self.prep_inference(tokens, start_pos, slots)
        for i in range(self.args.n_layers):
            h = self.layer_inference(i, h, st)
            if layers_out is not None:
                layers_out.append(h[0][:, :self.args.dim].clone())
            if layer_probe:
                info.setdefault("layer_tokens", []).append(self.finish_inference(h, st).argmax(dim=-1).tolist())
        if want is not None:
            if not len(want):
                return torch.empty(0, self.args.vocab_size, device=self.device), info
            want = torch.tensor(list(want), dtype=torch.int32).to(self.device, non_blocking=True)
        return self.finish_inference(h, st, want), info

    def _decode(self, tokens, start_pos, slots):
        B = tokens.shape[0]
        for s in slots:
            self.cache.extend(s, start_pos, 1)
        if B not in self._recorded:
            self._recorded[B] = RecordedStep(self, B)
        return self._recorded[B].run(tokens, start_pos, slots)


class RecordedStep:
    """The kernels of a one-token step of B sequences: the first run records the calls with their buffers, later runs
    issue them again.  Tokens, positions and slots are device inputs."""

    def __init__(self, model, B):
        dev = model.device
        self.model, self.calls = model, None
        self.tokens = torch.zeros(B, 1, dtype=torch.int64, device=dev)
        self.meta = torch.zeros(2, B, dtype=torch.int32, device=dev)
        self.host = torch.zeros(2, B, dtype=torch.int32).pin_memory()
        self.rows = torch.arange(B, dtype=torch.int32, device=dev)
        self.copied = torch.cuda.Event()

    def run(self, tokens, start_pos, slots):
        self.copied.synchronize()         # the previous step's inputs have left the pinned buffer
        self.host[0].fill_(start_pos)
        for b, s in enumerate(slots):
            self.host[1, b] = s
        self.meta.copy_(self.host, non_blocking=True)
        self.tokens.copy_(tokens, non_blocking=True)
        self.copied.record()
        if self.calls is not None:
            self.calls.replay()
            return self.logits.clone()
        m = self.model
        st = Step(self.tokens.shape[0], 1, None, self.meta[0], self.meta[1], None, m.cache)
        with K.Recording() as calls:
            h = m._embed(self.tokens)
            for layer in m.layers:
                layer(h[0], h[1], st)
            self.logits = m.finish_inference(h, st, self.rows)
        self.calls = calls
        return self.logits.clone()
