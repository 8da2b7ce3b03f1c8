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

Attention has two forms with the same result.  A step with few tokens works on the latents themselves: the queries go
through W_uk^T, attention reads the cache rows of the window once for all heads, and the result goes through W_uv.
A step with many tokens expands the latents of its context to per-head keys and values first.
"""
import math

import torch
from torch import nn

try:
    from . import float_kernel as K
    from .latent_cache import LatentCache
except ImportError:  # pragma: no cover - this directory first on sys.path
    import float_kernel as K
    from latent_cache import LatentCache

# a step with at most this many tokens per sequence attends over the latents, a longer one expands them
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
    def __init__(self, dim, eps):
        super().__init__()
        self.dim, self.eps = dim, eps
        self.register_buffer("weight", None)

    def load(self, w, device):
        self.weight = _padded(w, (K.pad8(self.dim),), torch.float32, device)

    def forward(self, x, out, index=None):
        K.norm_rows(x, index, self.weight, out, self.dim, self.eps)
        return out

    def add_to(self, x, y, xb):
        """x += norm(y), xb = bfloat16(x)"""
        K.add_norm(x, y, self.weight, xb, self.dim, self.eps)


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

    def load(self, W, prefix, dtype, device, table):
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
        self.table = table

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


class DenseFF(nn.Module):
    """W_down (silu(W_gate h) * (W_up h)); gate and up rows are interleaved in one product"""

    def __init__(self, layer_id, args, cfg):
        super().__init__()
        self.dim, self.ff = args.dim, cfg.ff
        self.register_buffer("w_gate_up", None)
        self.register_buffer("w_down", None)

    @staticmethod
    def tensors(prefix, cfg):
        return [prefix + "mlp." + n for n in ("gate", "up", "down")]

    def load(self, W, prefix, dtype, device):
        p, width, ff = prefix + "mlp.", K.pad8(self.dim), K.pad8(self.ff)
        w = torch.zeros(ff, 2, width, dtype=dtype, device=device)
        w[:self.ff, 0, :self.dim] = W(p + "gate", (self.ff, self.dim))
        w[:self.ff, 1, :self.dim] = W(p + "up", (self.ff, self.dim))
        self.w_gate_up = w.view(2 * ff, width)
        self.w_down = _padded(W(p + "down", (self.dim, self.ff)), (width, ff), dtype, device)

    def forward(self, h):
        hid = torch.empty(h.shape[0], self.w_down.shape[1], dtype=h.dtype, device=h.device)
        K.linear(h, self.w_gate_up, hid, K.GLU)
        out = torch.empty(h.shape[0], self.w_down.shape[0], dtype=torch.float32, device=h.device)
        return K.linear(hid, self.w_down, out)


MIXERS = {"latent_attention": LatentAttention}
FEEDFORWARDS = {"dense": DenseFF}


class DecoderLayer(nn.Module):
    """x <- x + norm1(mixer(x)); x <- x + norm2(ff(x)): norms on the outputs of the sublayers only"""

    def __init__(self, layer_id, args, cfg):
        super().__init__()
        self.prefix = "l%d." % layer_id
        self.mixer = MIXERS[cfg.mixer_kind](layer_id, args, cfg.mixer)
        self.norm1 = RMSNorm(args.dim, args.eps)
        self.ff = FEEDFORWARDS[cfg.mlp_kind](layer_id, args, cfg.mlp) if cfg.mlp_kind else None
        self.norm2 = RMSNorm(args.dim, args.eps) if self.ff is not None else None

    def load(self, W, dtype, device, table):
        self.mixer.load(W, self.prefix, dtype, device, table)
        self.norm1.load(W(self.prefix + "norm1", (self.norm1.dim,)), device)
        if self.ff is not None:
            self.ff.load(W, self.prefix, dtype, device)
            self.norm2.load(W(self.prefix + "norm2", (self.norm2.dim,)), device)

    def forward(self, x, xb, st):
        h = x if xb is None else xb
        self.norm1.add_to(x, self.mixer(h, st), xb)
        if self.ff is not None:
            self.norm2.add_to(x, self.ff(h), xb)


class FloatTransformer(nn.Module):
    """Embedding, layers, final norm and tied output of a floating-point decoder design.

    `step` runs the next tokens of a batch of sequences that stand at the same position; `begin_batch` /
    `end_batch` hand out and take back their cache slots.  The per-layer calls `prep_inference`,
    `layer_inference` and `finish_inference` have the shape of the integer model's.
    """

    def __init__(self, args, dtype=torch.bfloat16):
        super().__init__()
        if args.design.norm_placement != "output" or not args.design.tied_output or args.design.activation != "silu":
            raise NotImplementedError("design %s" % args.design.name)
        self.args, self.dtype = args, dtype
        self.layers = nn.ModuleList([DecoderLayer(i, args, c) for i, c in enumerate(args.layers)])
        self.norm = RMSNorm(args.dim, args.eps)
        self.register_buffer("embed", None)
        self.cache = None
        self._tables = {}
        self._recorded = {}         # batch size -> recorded one-token step

    # -- weights and cache --------------------------------------------------------------------------
    def load_weights(self, W, device):
        """W(name, shape) returns a checked tensor"""
        args = self.args
        for layer in self.layers:
            rot = layer.mixer.cfg.rot
            if rot not in self._tables:
                self._tables[rot] = rotary_table(rot, args.max_seq_len, device)
            layer.load(W, self.dtype, device, self._tables[rot])
        self.norm.load(W("final.norm", (args.dim,)), device)
        self.embed = _padded(W("embed", (args.vocab_size, args.dim)),
                             (K.pad8(args.vocab_size), K.pad8(args.dim)), self.dtype, device)
        owners = [i if l.mixer.own_kv else l.mixer.cfg.kv_from for i, l in enumerate(self.layers)]
        self.cache = LatentCache([l.mixer.pitch if l.mixer.own_kv else None for l in self.layers], owners,
                                 args.max_batch_size, args.max_seq_len, self.dtype, device)
        return self

    def tensor_names(self):
        names = ["embed", "final.norm"]
        for layer, cfg in zip(self.layers, self.args.layers):
            names += layer.mixer.tensors(layer.prefix, cfg.mixer) + [layer.prefix + "norm1"]
            if layer.ff is not None:
                names += layer.ff.tensors(layer.prefix, cfg.mlp) + [layer.prefix + "norm2"]
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
        xb = torch.empty(rows, pitch, dtype=self.dtype, device=self.device) if self.dtype != torch.float32 else None
        K.embed(tokens.contiguous().view(-1), self.embed, self.args.vocab_size, x, xb)
        return x, xb

    def layer_inference(self, layer_id, h, st):
        self.layers[layer_id](h[0], h[1], st)
        return h

    def finish_inference(self, h, st, want=None):
        """float32 logits [n, vocab] of the wanted rows (default: the last row of every sequence)"""
        if want is None:
            want = torch.arange(st.batch, dtype=torch.int32, device=self.device) * st.seq + (st.seq - 1)
        x = torch.empty(want.shape[0], self.embed.shape[1], dtype=self.dtype, device=self.device)
        self.norm(h[0], x, want)
        logits = torch.empty(want.shape[0], self.embed.shape[0], dtype=torch.float32, device=self.device)
        return K.linear(x, self.embed, logits)[:, :self.args.vocab_size]

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
