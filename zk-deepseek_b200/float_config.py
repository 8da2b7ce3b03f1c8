"""Configuration of the floating-point decoder designs, read from a checkpoint's config.json.

A config lists its layers; each names a mixer (with its own sizes and constants) and a feed-forward.  Sizes that the
file leaves out are taken from the shapes of the weights.  What a design fixes for all of its models (where the norms
sit, the activation, the tied output) is in `Design`.
"""
import json
import os
from dataclasses import dataclass, field
from typing import List, Optional


@dataclass(frozen=True)
class Design:
    name: str
    norm_placement: str = "output"      # x <- x + norm(sublayer(x))
    activation: str = "silu"
    tied_output: bool = True


DESIGNS = {"Munalorn": Design("Munalorn")}


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int                           # rotated dimensions, interleaved pairs


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
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class LayerConfig:
    mixer_kind: str
    mixer: LatentAttentionConfig
    mlp_kind: Optional[str] = None
    mlp: Optional[DenseConfig] = None


@dataclass
class DecoderArgs:
    design: Design
    vocab_size: int
    dim: int
    eps: float
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


MIXER_CONFIGS = {"latent_attention": _latent_attention}
MLP_CONFIGS = {"dense": lambda i, m, shapes: DenseConfig(_size(m, "ff", shapes, "l%d.mlp.down" % i, 1))}


def parse_config(cfg, shapes=None):
    """DecoderArgs of a parsed config.json; `shapes` maps tensor names to shapes"""
    shapes = shapes or {}
    name = cfg.get("architecture")
    if name not in DESIGNS:
        raise ConfigError("unknown design %r (known: %s)" % (name, ", ".join(sorted(DESIGNS))))
    args = DecoderArgs(DESIGNS[name], _size(cfg, "vocab", shapes, "embed", 0), _size(cfg, "width", shapes, "embed", 1),
                       float(cfg["norm"]["eps"]))
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
        args.layers.append(LayerConfig(kind, mixer, m["kind"], MLP_CONFIGS[m["kind"]](i, m, shapes)))
    return args


def read_config(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)
