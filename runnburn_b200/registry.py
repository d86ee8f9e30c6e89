"""Model registry: which decoder a model file or folder describes, and its loading.

    *.gguf                          quantised Llama / Qwen-style stacks (general.architecture in the file)
    folder with config.json         "architecture" names an entry of ARCHITECTURES; weights in
                                    model.safetensors
"""
from __future__ import annotations

import json
from pathlib import Path

from .decoder import Decoder
from .safetensors import SafetensorsFile
from .stack import dutivik_config, punisun_config

# architecture -> function(config.json, max_ctx, dtype) that builds the decoder's configuration
ARCHITECTURES = {"Punisun": punisun_config, "Dutivik": dutivik_config}


def read_config(folder, max_ctx: int, dtype: str = "bfloat16"):
    cfg = json.loads((Path(folder) / "config.json").read_text())
    name = cfg.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"architecture {name!r} is not known (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[name](cfg, max_ctx, dtype)


def load_model(path, max_ctx: int = 0, dtype: str = "bfloat16") -> Decoder:
    """Creates the decoder of `path` and uploads its weights.  max_ctx 0: the file's own (GGUF) or 4096."""
    path = Path(path)
    if path.suffix == ".gguf":
        from .gguf import load_decoder
        dec, f = load_decoder(str(path), max_ctx)
        dec._file = f          # the mapped pages stay alive with the decoder
        return dec
    dec = Decoder(read_config(path, max_ctx or 4096, dtype))
    for name, (dt, shape, data) in SafetensorsFile(path / "model.safetensors").items():
        dec.set_tensor(name, dt, data, shape)
    return dec
