"""Paged engine: AR vs batched decode, checking that a batch reproduces per-prompt outputs.

    python examples/engine_generate.py [/path/to/model | karuzen | zasipel | kizezen | sogidra]

Any registered model family loads from its directory; ``karuzen``, ``zasipel``, ``kizezen`` and ``sogidra`` are tiny random
models of those designs, no argument a tiny random Qwen3.  The batch is run once more with its prompts fed in portions beside the others' decode steps.

Reference counterpart: ``examples/engine/jetspec_engine_generate.py:19-64``."""
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))   # run from a checkout

from jetspec_b200 import JetSpecEngine, SamplingParams  # noqa: E402
from jetspec_b200.models import (KaruzenForCausalLM, KizezenForCausalLM, Qwen3ForCausalLM, SogidraForCausalLM,  # noqa: E402
                                 ZasipelForCausalLM, karuzen_tiny_config, kizezen_tiny_config, sogidra_tiny_config, tiny_config,
                                 zasipel_tiny_config)

TINY = {"karuzen": (KaruzenForCausalLM, karuzen_tiny_config), "zasipel": (ZasipelForCausalLM, zasipel_tiny_config),
        "kizezen": (KizezenForCausalLM, kizezen_tiny_config), "sogidra": (SogidraForCausalLM, sogidra_tiny_config)}

if __name__ == "__main__":
    dev = "cuda" if torch.cuda.is_available() else "cpu"
    dt = torch.bfloat16 if dev == "cuda" else torch.float32
    name = sys.argv[1] if len(sys.argv) > 1 else None
    if name in TINY:
        cls, config = TINY[name]
        model = cls.random_init(config(), seed=0, dtype=dt, init="stable")
    else:
        model = name if name is not None else Qwen3ForCausalLM.random_init(tiny_config(), seed=0, dtype=dt)
    eng = JetSpecEngine(model, device=dev, dtype=dt, block_size=16)
    g = torch.Generator().manual_seed(0)
    prompts = [torch.randint(0, eng.cfg.vocab_size, (1, n), generator=g) for n in (7, 19, 12)]
    sp = SamplingParams(0.0, 24)
    singles = [eng.generate(p, sp)["token_ids"] for p in prompts]
    batch = [r["token_ids"] for r in eng.generate_batch(prompts, sp)]
    print("batch == single:", [a == b for a, b in zip(batch, singles)], eng.last_stats)
    portions = [r["token_ids"] for r in eng.generate_batch(prompts, sp, prefill_chunk=8)]
    print("batch in portions == single:", [a == b for a, b in zip(portions, singles)], eng.last_stats)
