"""Token generation with every layer resident on the GPU: the loop that serves the integer model and the
floating-point decoder designs, and the command line.

Follows the loop of the reference's `generate()` (inference/generate.py:164-286): the prompt
is run as one prefill, then one position per step; `prompt_mask` keeps prompt tokens from being
overwritten when the prompts of a batch have different lengths; a sequence finishes at `eos_id`;
with `snark` set in the model module every step writes `pos_{p}/tokens.bin` next to the layer
dumps (generate.py:218-220).

Differences, all on the host side of the hot path:
  * the reference rebuilds `Block(i)` from its state dict and moves the latent caches to the GPU
    for every layer of every step (generate.py:231-244) because the 671B model does not fit one
    GPU; here the layers, their limb planes, the caches and the lookup tables stay resident;
  * the per-layer debug projection through `norm` and `head` (generate.py:246-259) is off unless
    `layer_probe=True`; it then returns the same per-layer candidate token ids instead of printing;
  * `sample()` in the reference has its stochastic branch switched off (`sample_open = False`,
    generate.py:80) and returns the argmax for every temperature; the same is done here.
"""
import argparse
import importlib
import json
import os
import sys
from typing import List, Optional

import torch


def _module(name):
    # drop-in use: this directory first on sys.path, no package
    return importlib.import_module("." + name, __package__) if __package__ else importlib.import_module(name)


def load_resident(ckpt_path: str, args, device="cuda", cache_batch: int = 1, prepare: bool = True):
    """Builds a `Transformer` with every layer on `device` from a converted checkpoint directory:
    `embed_int.safetensors`, `norm_int.safetensors`, `head_int.safetensors` (generate.py:53-60),
    `layer-{i}.safetensors` (generate.py:344-345, loaded with strict=False as generate.py:238 does) and
    `experts-{layer}/{i}.safetensors` (model.py:1361-1363).  The reference keeps the layer state dicts on the
    host and rebuilds one `Block` at a time; here all of them stay resident, and with `prepare` the limb
    planes of every static weight are built once at load instead of at first use."""
    from safetensors.torch import load_file, load_model
    M = _module("model")
    with torch.device(device):
        model = M.Transformer(args)
    load_model(model.embed, os.path.join(ckpt_path, "embed_int.safetensors"))
    load_model(model.norm, os.path.join(ckpt_path, "norm_int.safetensors"))
    load_model(model.head, os.path.join(ckpt_path, "head_int.safetensors"))
    for i in range(args.n_layers):
        with torch.device(device):
            blk = M.Block(i, args, ckpt_path, cache_batch=cache_batch)
        blk.load_state_dict(load_file(os.path.join(ckpt_path, f"layer-{i}.safetensors"), device=str(device)),
                            strict=False)
        if isinstance(blk.ffn, M.MoE):
            blk.ffn.set_experts()
        model.layers[i] = blk
    if prepare:
        for mod in model.modules():
            if isinstance(mod, M.Linear_int):
                mod.planes()
            elif isinstance(mod, M.MoE):
                mod._prepared()
    return model


def sample(logits: torch.Tensor, temperature: float = 1.0) -> torch.Tensor:
    """generate.py:62-143 with `sample_open = False`: the argmax over the vocabulary."""
    return logits.argmax(dim=-1)


@torch.inference_mode()
def generate(model, prompt_tokens: List[List[int]], max_new_tokens: int, eos_id: int,
             temperature: float = 1.0, layer_probe: bool = False,
             trace: Optional[list] = None) -> List[List[int]]:
    """Returns the completion tokens of every prompt (generate.py:164-286).

    model: what `registry.load` returns: a `Transformer` whose `layers[i]` are loaded `Block`s (caches sized for
    the batch), or a `FloatTransformer`.  The loop only uses begin_batch / step / end_batch, `args` and `device`.
    trace: optional list; receives one dict per step (`pos`, `next_token`, and `layer_tokens` when
    `layer_probe` is set) in place of the reference's progress prints.
    """
    args = model.args
    device = model.device
    prompt_lens = [len(t) for t in prompt_tokens]
    assert max(prompt_lens) <= args.max_seq_len, \
        f"Prompt length exceeds model maximum sequence length (max_seq_len={args.max_seq_len})"
    total_len = min(args.max_seq_len, max_new_tokens + max(prompt_lens))
    tokens = torch.full((len(prompt_tokens), total_len), -1, dtype=torch.long, device=device)
    for i, t in enumerate(prompt_tokens):
        tokens[i, :len(t)] = torch.tensor(t, dtype=torch.long, device=device)
    prev_pos = 0
    finished = torch.zeros(len(prompt_tokens), dtype=torch.bool, device=device)
    prompt_mask = tokens != -1
    batch = model.begin_batch(len(prompt_tokens))
    try:
        for cur_pos in range(min(prompt_lens), total_len):
            logits, info = model.step(tokens[:, prev_pos:cur_pos], prev_pos, batch, layer_probe=layer_probe)
            next_token = (sample(logits, temperature) if temperature > 0 else logits.argmax(dim=-1)).view(-1)
            next_token = torch.where(prompt_mask[:, cur_pos], tokens[:, cur_pos], next_token)
            tokens[:, cur_pos] = next_token
            finished |= torch.logical_and(~prompt_mask[:, cur_pos], next_token == eos_id)
            prev_pos = cur_pos
            if trace is not None:
                trace.append({"pos": cur_pos, "next_token": next_token.tolist(), **info})
            if finished.all():
                break
    finally:
        model.end_batch(batch)
    completion_tokens = []
    for i, toks in enumerate(tokens.tolist()):
        toks = toks[prompt_lens[i]:prompt_lens[i] + max_new_tokens]
        if eos_id in toks:
            toks = toks[:toks.index(eos_id)]
        completion_tokens.append(toks)
    return completion_tokens


def main(argv=None):
    """Generates from prompts given as token ids (the checkpoints carry no tokenizer)."""
    reg = _module("registry")
    ap = argparse.ArgumentParser(prog="generate", description=main.__doc__)
    ap.add_argument("--model", required=True, help="directory with config.json and *.safetensors (%s)"
                    % ", ".join(reg.architectures()))
    ap.add_argument("--tokens", action="append", default=[], metavar="IDS",
                    help="one prompt: token ids separated by commas or spaces; may be given several times")
    ap.add_argument("--input-file", help="JSON list of prompts, each a list of token ids")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--max-seq-len", type=int, default=4096)
    ap.add_argument("--eos-id", type=int, default=-1)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"],
                    help="number format of the floating-point designs")
    ap.add_argument("--layer-probe", action="store_true", help="report every layer's candidate token on stderr")
    args = ap.parse_args(argv)
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in args.tokens]
    if args.input_file:
        with open(args.input_file) as f:
            prompts += json.load(f)
    if not prompts or not all(prompts):
        ap.error("give at least one prompt, none of them empty")
    model = reg.load(args.model, dtype=args.dtype, max_seq_len=args.max_seq_len, max_batch_size=len(prompts))
    vocab = model.args.vocab_size
    if any(not 0 <= t < vocab for p in prompts for t in p):
        ap.error("token ids go from 0 to %d" % (vocab - 1))
    trace = [] if args.layer_probe else None
    out = generate(model, prompts, args.max_new_tokens, args.eos_id, args.temperature, args.layer_probe, trace)
    for step in trace or []:
        print(json.dumps(step), file=sys.stderr)
    for tokens in out:
        print(json.dumps(tokens))
    return 0


if __name__ == "__main__":
    sys.exit(main())
