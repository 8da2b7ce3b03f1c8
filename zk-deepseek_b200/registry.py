"""Model registry: which class a checkpoint directory belongs to, and how it is loaded.

A config.json with an "architecture" entry names a floating-point decoder design; one without is the integer
DeepSeek model, whose file holds the fields of `model.ModelArgs`.  Each family is imported (and its CUDA library
built, if that is missing) only when a model of it is loaded.
"""
import dataclasses
import importlib
import json
import os
import struct
import sys

try:
    from . import build as _build
    from . import float_config
except ImportError:  # pragma: no cover - this directory first on sys.path
    import build as _build
    import float_config

INTEGER_MODEL = "DeepseekV3Int"


def architectures():
    return sorted(float_config.DESIGNS) + [INTEGER_MODEL]


def architecture_of(cfg):
    name = cfg.get("architecture", INTEGER_MODEL)
    if name not in architectures():
        raise float_config.ConfigError("unknown architecture %r (known: %s)" % (name, ", ".join(architectures())))
    return name


def _module(name):
    return importlib.import_module("." + name, __package__) if __package__ else importlib.import_module(name)


# ---- safetensors files ----------------------------------------------------------------------------------
_DTYPES = {"F32": "float32", "BF16": "bfloat16", "F16": "float16", "I32": "int32", "I64": "int64"}


class TensorFiles:
    """The *.safetensors files of a directory: 8-byte little-endian header length, a JSON header
    name -> {dtype, shape, data_offsets}, the data.  Tensors are mapped, not read, until they are used."""

    def __init__(self, model_dir):
        self.where, self._maps = {}, {}
        for fn in sorted(os.listdir(model_dir)):
            if not fn.endswith(".safetensors"):
                continue
            path = os.path.join(model_dir, fn)
            with open(path, "rb") as f:
                n = struct.unpack("<Q", f.read(8))[0]
                if n > os.path.getsize(path) - 8:
                    raise ValueError("%s: header of %d bytes" % (fn, n))
                header = json.loads(f.read(n))
            for name, t in header.items():
                if name != "__metadata__":
                    self.where[name] = (path, t["dtype"], tuple(t["shape"]), 8 + n + t["data_offsets"][0],
                                        t["data_offsets"][1] - t["data_offsets"][0])
        if not self.where:
            raise FileNotFoundError("no tensors in %s" % model_dir)

    def shapes(self):
        return {k: v[2] for k, v in self.where.items()}

    def __call__(self, name, shape):
        """the tensor (CPU), whose shape must be `shape`"""
        import numpy as np
        import torch
        if name not in self.where:
            raise KeyError("the checkpoint has no tensor '%s'" % name)
        path, kind, got, offset, nbytes = self.where[name]
        if tuple(shape) != got:
            raise ValueError("tensor '%s' is %s, the configuration says %s" % (name, list(got), list(shape)))
        dtype = getattr(torch, _DTYPES[kind])
        if path not in self._maps:
            self._maps[path] = np.memmap(path, dtype=np.uint8, mode="r")
        raw = np.array(self._maps[path][offset:offset + nbytes])
        return torch.from_numpy(raw).view(dtype).view(got) if nbytes else torch.empty(got, dtype=dtype)


# ---- loading ---------------------------------------------------------------------------------------------
def load_float_model(model_dir, dtype="bfloat16", device="cuda", max_seq_len=4096, max_batch_size=1, cfg=None):
    import torch
    cfg = cfg if cfg is not None else float_config.read_config(model_dir)
    files = TensorFiles(model_dir)
    args = float_config.parse_config(cfg, files.shapes())
    args.max_seq_len, args.max_batch_size = int(max_seq_len), int(max_batch_size)
    _build.build(library=_build.FLOAT_LIBRARY)
    fm = _module("float_model")
    model = fm.FloatTransformer(args, getattr(torch, dtype) if isinstance(dtype, str) else dtype)
    unused = sorted(set(files.where) - set(model.tensor_names()))
    if unused:
        print("tensors the configuration has no place for: %s%s" % (", ".join(unused[:5]), " ..." if unused[5:] else ""),
              file=sys.stderr)
    return model.load_weights(files, torch.device(device))


def load_integer_model(model_dir, device="cuda", max_seq_len=None, max_batch_size=1, cfg=None):
    cfg = cfg if cfg is not None else float_config.read_config(model_dir)
    _build.build(library=_build.INT_LIBRARY)
    M = _module("model")
    fields = {f.name for f in dataclasses.fields(M.ModelArgs)}
    args = M.ModelArgs(**{k: v for k, v in cfg.items() if k in fields})
    if max_seq_len:
        args.max_seq_len = int(max_seq_len)
    return _module("generate").load_resident(model_dir, args, device=device, cache_batch=max_batch_size)


def load(model_dir, dtype="bfloat16", device="cuda", max_seq_len=4096, max_batch_size=1):
    """The model of a checkpoint directory, ready to run on `device`.  dtype belongs to the floating-point designs;
    the integer model has one number format."""
    cfg = float_config.read_config(model_dir)
    if architecture_of(cfg) == INTEGER_MODEL:
        return load_integer_model(model_dir, device, max_seq_len, max_batch_size, cfg)
    return load_float_model(model_dir, dtype, device, max_seq_len, max_batch_size, cfg)
