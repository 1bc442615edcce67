"""The model registry: a checkpoint names its architecture, the registry picks the design that serves it.

    python -m skainet_b200.models --model PATH --tokens 5,17,3 [--steps 32] [--dtype bfloat16|float32] [--max-seq N]

loads a model and prints the tokens greedy decoding appends. A folder with config.json and model.safetensors is chosen by
its "architecture", a .gguf file by its general.architecture."""
from __future__ import annotations

import argparse
import json
import os
from typing import Callable, Dict, List, Sequence

from .decoder import Decoder
from .fomalix import Fomalix
from .llama import Llama
from .tivazen import Tivazen

FOLDERS: Dict[str, Callable[..., Decoder]] = {Tivazen.architecture: Tivazen.from_dir, Fomalix.architecture: Fomalix.from_dir}
GGUF: Dict[str, Callable[..., Decoder]] = {"llama": Llama.from_gguf}


def load_model(path: str, dtype: str = "bfloat16", max_seq: int = 1024, max_batch: int = 1) -> Decoder:
    """A finalized model. dtype chooses the arithmetic where the design has a choice; packed models have one."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
        name, table = config.get("architecture"), FOLDERS
    else:
        from .gguf import StreamingGGUFReader
        r = StreamingGGUFReader(path)
        name, table = r.fields.get("general.architecture"), GGUF
        r.close()
    if name not in table:
        raise ValueError(f"{path}: architecture {name!r} is not one of {sorted(table)}")
    if table is FOLDERS:
        return table[name](path, config, dtype=dtype, max_seq=max_seq, max_batch=max_batch)
    return table[name](path, max_seq=max_seq, max_batch=max_batch)


def generate(model: Decoder, tokens: Sequence[int], steps: int) -> List[int]:
    """Greedy continuation of one prompt in a slot of its own (the first: decode steps run over slots from 0 up)."""
    seq = model.acquire()
    try:
        if seq != 0:
            raise RuntimeError("generate needs the first sequence slot")
        if steps <= 0:
            return []
        first = model.prefill(tokens, seq)
        rest = model.generate([first], steps - 1)[:, 0] if steps > 1 else []
        return [int(first), *map(int, rest)]
    finally:
        model.release(seq)


def main() -> None:
    ap = argparse.ArgumentParser(prog="python -m skainet_b200.models", description="Greedy generation from token ids.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a .gguf file")
    ap.add_argument("--tokens", required=True, help="prompt token ids, comma-separated")
    ap.add_argument("--steps", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    ap.add_argument("--max-seq", type=int, default=0, help="cache capacity; default: prompt and generated tokens")
    a = ap.parse_args()
    tokens = [int(t) for t in a.tokens.split(",")]
    from .build import build
    build()
    m = load_model(a.model, a.dtype, a.max_seq or len(tokens) + a.steps)
    print(",".join(map(str, generate(m, tokens, a.steps))))


if __name__ == "__main__":
    main()
