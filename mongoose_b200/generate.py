"""Greedy generation from the command line.

    python -m mongoose_b200.generate --model DIR --prompt 5,17,3 --new 32 [--dtype float32]
    python -m mongoose_b200.generate --config tiny --prompt 1,2,3 --new 16

--model loads a folder (config.json, model.safetensors); --config runs a named configuration with
random-init weights.  Prints the generated token ids.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m mongoose_b200.generate", description=__doc__.split("\n")[0])
    src = ap.add_mutually_exclusive_group(required=True)
    src.add_argument("--model", help="folder with config.json and model.safetensors")
    src.add_argument("--config", help="named configuration, random-init weights")
    ap.add_argument("--prompt", required=True, help="comma-separated token ids")
    ap.add_argument("--new", type=int, default=16, help="tokens to generate")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="arithmetic of layer-described models")
    ap.add_argument("--max-seq", type=int, default=0)
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    try:
        prompt = [int(t) for t in a.prompt.split(",")]
    except ValueError:
        ap.error("--prompt takes comma-separated token ids")

    from . import _lib, registry, synthetic
    if a.model:
        arch, _ = registry.read_config(a.model)
        _lib.provision(arch.family)
        engine = registry.load_model(a.model, dtype=a.dtype, max_seq=a.max_seq or len(prompt) + a.new, device=a.device)
    else:
        cfg = registry.named_config(a.config)
        cfg = cfg.with_(max_seq=a.max_seq or max(len(prompt) + a.new, 1))
        if isinstance(cfg, registry.LayeredConfig):
            _lib.provision("layered")
            engine = registry.create_engine(cfg.with_(math=registry.MATH[a.dtype]), a.device)
            synthetic.load_layered(engine, seed=0)
        else:
            engine = registry.create_engine(cfg, a.device)
            synthetic.load_engine(engine, cfg, seed=0)
    print(",".join(str(t) for t in engine.Generate(prompt, a.new)))
    engine.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
