"""Greedy generation with any model of the registry, as a function and as a command:

    python -m ug_b200.generate --model DIR --prompt 12,7,99 [--prompt 3,1,4] -n 32 [--chunk 512] [--dtype float32]

Token ids in, token ids out (a tokenizer is not part of this package).  Prompts of one call are the rows of a batch and
share their length; a prompt is fed in portions of ``chunk`` positions, then every new token is one graph-replayed step
whose input is the device-side argmax of the previous one.
"""
import argparse
import sys

import numpy as np

from .device import DType, UgError

DTYPES = {"bfloat16": DType.BF16, "float32": DType.F32}


def generate(model, prompts, n_new, chunk=None, reset=True):
    """int32 [batch, n_new] continuations of ``prompts`` (int32 [batch, t])."""
    prompts = np.ascontiguousarray(prompts, dtype=np.int32)
    if prompts.ndim != 2 or prompts.shape[0] != model.batch or prompts.shape[1] < 1:
        raise UgError(3, f"prompts must be [batch={model.batch}, t >= 1], got {prompts.shape}")
    if reset:
        model.reset()
    t = prompts.shape[1]
    for lo in range(0, t, chunk or t):
        model.prefill(prompts[:, lo:lo + (chunk or t)])
    out = np.empty((model.batch, n_new), np.int32)
    for i in range(n_new):
        if i:
            model.decode(1)
        out[:, i] = model.next_tokens()
    model.dev.synchronize()
    return out


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m ug_b200.generate", description="greedy generation from token ids")
    ap.add_argument("--model", required=True, help="folder with config.json and .safetensors files")
    ap.add_argument("--prompt", action="append", required=True, metavar="IDS", help="comma-separated token ids; repeat for a batch")
    ap.add_argument("-n", "--new-tokens", type=int, default=32)
    ap.add_argument("--chunk", type=int, default=None, help="positions of the prompt per portion")
    ap.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    from . import registry
    from .device import Device
    prompts = [[int(x) for x in p.split(",")] for p in a.prompt]
    if len({len(p) for p in prompts}) != 1:
        ap.error("the prompts of a batch must have one length")
    dev = Device(a.device)
    model = registry.load(a.model, dev, len(prompts), len(prompts[0]) + a.new_tokens, DTYPES[a.dtype])
    for row in generate(model, np.array(prompts, np.int32), a.new_tokens, a.chunk):
        print(",".join(str(t) for t in row))
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
