"""Configuration of the floating-point decoder designs, read from a checkpoint's config.json.

A config lists its layers; each names a mixer (with its own sizes and constants) and a feed-forward.  Sizes that the
file leaves out are taken from the shapes of the weights.  What a design fixes for all of its models (where the norms
sit, how their weights are stored, the activation, biases, the output projection) is in `Design`.
"""
import json
import os
from dataclasses import dataclass, field
from typing import List, Optional, Tuple, Union


@dataclass(frozen=True)
class Design:
    name: str
    norm_placement: str = "output"      # "output": x <- x + N(f(x)); "both": x <- x + N(f(N(x)))
    norm_offset: float = 0.0            # the norms multiply by this + the stored weight
    activation: str = "silu"
    ff_bias: bool = False
    scaled_embedding: bool = False      # config embedding.scale multiplies the embedding
    tied_output: bool = True            # logits through the embedding, else through the tensor 'head'


DESIGNS = {"Munalorn": Design("Munalorn"),
           "Vifelix": Design("Vifelix", norm_placement="both", norm_offset=1.0, ff_bias=True, scaled_embedding=True,
                             tied_output=False)}


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int                           # rotated dimensions
    layout: str = "pairs"               # turns (2i, 2i + 1), or with "half" (i, i + dims / 2)


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int                            # unrotated query / key size per head
    rot_dim: int                        # rotated query / key size per head
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotary
    window: int = 0                     # visible keys including the query's own, 0 = all
    kv_from: Optional[int] = None       # layer whose latents this layer reads


@dataclass(frozen=True)
class KeyValuedAttentionConfig:
    """softmax attention over a window whose values are the projected keys before norm and rotation"""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: Rotary
    window: int = 0                     # visible keys including the query's own, 0 = all


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]            # per head
    rot: Rotary


@dataclass(frozen=True)
class ParallelConfig:
    """two mixers on the same input, added with fixed weights"""
    left: KeyValuedAttentionConfig
    right: RetentionConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                           # taps
    norm_groups: int


MixerConfig = Union[LatentAttentionConfig, ParallelConfig, Mamba2Config]


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    bias: bool = False


@dataclass(frozen=True)
class LayerConfig:
    mixer_kind: str
    mixer: MixerConfig
    mlp_kind: Optional[str] = None
    mlp: Optional[DenseConfig] = None


@dataclass
class DecoderArgs:
    design: Design
    vocab_size: int
    dim: int
    eps: float
    embed_scale: float = 1.0
    layers: List[LayerConfig] = field(default_factory=list)
    max_seq_len: int = 4096
    max_batch_size: int = 1

    @property
    def n_layers(self):
        return len(self.layers)


class ConfigError(ValueError):
    pass


def _size(d, key, shapes, tensor, axis, divide=1, less=0):
    """d[key], or the size that a weight's shape implies"""
    if d.get(key) is not None:
        return int(d[key])
    if tensor not in shapes:
        raise ConfigError("config has no '%s' and the checkpoint no '%s' to take it from" % (key, tensor))
    return (int(shapes[tensor][axis]) - less) // divide


def _latent_attention(i, mx, shapes, layers):
    p = "l%d.mix." % i
    kv_from = mx.get("kv_from")
    if kv_from is not None:
        kv_from = int(kv_from)
        if not 0 <= kv_from < i or layers[kv_from].mixer.kv_from is not None:
            raise ConfigError("layer %d reads the latents of layer %d, which has none of its own" % (i, kv_from))
    H = int(mx["heads"])
    rot = mx.get("rot")
    if rot is None and kv_from is not None:
        rot = {"base": layers[kv_from].mixer.rot.base, "dims": layers[kv_from].mixer.rot.dims}
    if not rot:
        raise ConfigError("layer %d has no rotation" % i)
    rot_dim = int(mx["rot_dim"]) if mx.get("rot_dim") is not None else int(rot["dims"])
    rotary = Rotary(float(rot["base"]), int(rot.get("dims", rot_dim)))
    if rotary.dims != rot_dim or rot_dim % 2:
        raise ConfigError("layer %d: the rotated part has %d dimensions, the rotation %d" % (i, rot_dim, rotary.dims))
    mask = mx.get("mask") or {}
    cfg = LatentAttentionConfig(
        heads=H, rot_dim=rot_dim, rot=rotary, kv_from=kv_from, scale=float(mx["scale"]),
        dim=_size(mx, "dim", shapes, p + "uk", 0, H), vdim=_size(mx, "vdim", shapes, p + "uv", 0, H),
        q_rank=_size(mx, "q_rank", shapes, p + "dq", 0), kv_rank=_size(mx, "kv_rank", shapes, p + "uk", 1),
        window=int(mask.get("size") or 0))
    if kv_from is not None:
        src = layers[kv_from].mixer
        if (src.kv_rank, src.rot_dim, src.rot) != (cfg.kv_rank, cfg.rot_dim, cfg.rot):
            raise ConfigError("layers %d and %d do not agree on the latents they share" % (kv_from, i))
    return cfg


def _rotary(where, mx, dim):
    rot = mx.get("rot")
    if not rot:
        raise ConfigError("%s has no rotation" % where)
    r = Rotary(float(rot["base"]), int(rot.get("dims", dim)), "half")
    if r.dims % 2 or not 0 < r.dims <= dim:
        raise ConfigError("%s: a rotation of %d of %d dimensions" % (where, r.dims, dim))
    return r


def _key_valued_attention(where, p, mx, shapes):
    dim = _size(mx, "dim", shapes, p + "q.norm", 0)
    if mx.get("vdim") is not None and int(mx["vdim"]) != dim:
        raise ConfigError("%s: the values are the keys, but their sizes are %s and %d" % (where, mx["vdim"], dim))
    heads, kv = _size(mx, "heads", shapes, p + "q", 0, dim), _size(mx, "kv_heads", shapes, p + "k", 0, dim)
    if kv < 1 or heads % kv:
        raise ConfigError("%s: %d heads over %d key heads" % (where, heads, kv))
    mask = mx.get("mask") or {}
    return KeyValuedAttentionConfig(heads, kv, dim, float(mx["scale"]), _rotary(where, mx, dim), int(mask.get("size") or 0))


def _retention(where, p, mx, shapes):
    decay = tuple(float(x) for x in mx["decay"])
    heads = int(mx.get("heads") or len(decay))
    if len(decay) != heads or not all(0.0 <= d <= 1.0 for d in decay):
        raise ConfigError("%s: %d heads with decays %s" % (where, heads, list(decay)))
    dim = _size(mx, "dim", shapes, p + "q", 0, heads)
    return RetentionConfig(heads, dim, _size(mx, "vdim", shapes, p + "v", 0, heads), decay, _rotary(where, mx, dim))


def _parallel(i, mx, shapes, layers):
    p, where = "l%d.mix." % i, "layer %d" % i
    return ParallelConfig(_key_valued_attention(where + " left", p + "left.", mx["left"], shapes),
                          _retention(where + " right", p + "right.", mx["right"], shapes),
                          float(mx["left_scale"]), float(mx["right_scale"]))


def _mamba2(i, mx, shapes, layers):
    p = "l%d.mix." % i
    heads = _size(mx, "heads", shapes, p + "A_log", 0)
    vdim = _size(mx, "vdim", shapes, p + "norm", 0, heads)
    groups = int(mx.get("groups") or 1)
    c = Mamba2Config(heads, vdim, _size(mx, "state", shapes, p + "conv", 0, 2 * groups, heads * vdim), groups,
                     _size(mx, "conv", shapes, p + "conv", 1), int(mx.get("norm_groups") or 1))
    if heads % groups or (heads * vdim) % c.norm_groups or c.conv < 1:
        raise ConfigError("layer %d: %d heads of %d in %d groups, %d norm groups, %d taps"
                          % (i, heads, vdim, groups, c.norm_groups, c.conv))
    return c


MIXER_CONFIGS = {"latent_attention": _latent_attention, "parallel": _parallel, "mamba2": _mamba2}
MLP_CONFIGS = {"dense": lambda i, m, shapes, design: DenseConfig(_size(m, "ff", shapes, "l%d.mlp.down" % i, 1),
                                                                 design.ff_bias)}


def parse_config(cfg, shapes=None):
    """DecoderArgs of a parsed config.json; `shapes` maps tensor names to shapes"""
    shapes = shapes or {}
    name = cfg.get("architecture")
    if name not in DESIGNS:
        raise ConfigError("unknown design %r (known: %s)" % (name, ", ".join(sorted(DESIGNS))))
    args = DecoderArgs(DESIGNS[name], _size(cfg, "vocab", shapes, "embed", 0), _size(cfg, "width", shapes, "embed", 1),
                       float(cfg["norm"]["eps"]))
    if args.design.scaled_embedding:
        args.embed_scale = float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i, L in enumerate(cfg["layers"]):
        kind = L["type"]
        if kind not in MIXER_CONFIGS:
            raise ConfigError("layer %d: unknown mixer %r" % (i, kind))
        mixer = MIXER_CONFIGS[kind](i, L["mixer"], shapes, args.layers)
        m = L.get("mlp")
        if m is None:
            args.layers.append(LayerConfig(kind, mixer))
            continue
        if m["kind"] not in MLP_CONFIGS:
            raise ConfigError("layer %d: unknown feed-forward %r" % (i, m["kind"]))
        args.layers.append(LayerConfig(kind, mixer, m["kind"], MLP_CONFIGS[m["kind"]](i, m, shapes, args.design)))
    return args


def read_config(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)
