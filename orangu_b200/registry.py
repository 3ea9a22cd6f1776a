"""Which class loads a model: by ``general.architecture`` for a .gguf file, by config.json's ``architecture`` for a folder."""
from __future__ import annotations

import json
import os

from .fenipel import FenipelModel
from .filorax import FiloraxModel
from .model import LlamaModel
from .nenodra import NenodraModel
from .senuvik import SenuvikModel

GGUF_ARCHITECTURES = {a: LlamaModel for a in ("llama", "mistral", "qwen2", "qwen3", "qwen3vl")}
FOLDER_ARCHITECTURES = {m.ARCHITECTURE: m for m in (FenipelModel, NenodraModel, SenuvikModel, FiloraxModel)}


def model_class(path: str):
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            name = json.load(f).get("architecture")
        table = FOLDER_ARCHITECTURES
    else:
        from .gguf import GgufFile

        with GgufFile(path) as g:
            name = g.get_string("general.architecture")
        table = GGUF_ARCHITECTURES
    if name not in table:
        raise ValueError(f"{path}: no model class for architecture {name!r}; known here: {', '.join(sorted(table))}")
    return table[name]


def load_model(backend, path: str, dtype: str = "bfloat16", max_seq_len: int = 4096, max_batch_tokens: int = 512, kv_pool_tokens: int = 0,
               state_slots: int = 0):
    """The model in a .gguf file or a folder with config.json and model.safetensors.  ``dtype`` and ``state_slots`` concern the
    latter; quantized files have their own arithmetic."""
    cls = model_class(path)
    if os.path.isdir(path):
        return cls.from_folder(backend, path, dtype=dtype, max_seq_len=max_seq_len, max_batch_tokens=max_batch_tokens, kv_pool_tokens=kv_pool_tokens,
                               state_slots=state_slots)
    return cls.from_gguf(backend, path, max_seq_len=max_seq_len, max_batch_tokens=max_batch_tokens, kv_pool_tokens=kv_pool_tokens)
