"""Which loader serves a model: by config.json's "architecture" for a folder, by general.architecture for a GGUF file."""
import json
import os

from .gguf import GgufFile, load_llama


def _goletar(path, config, **kw):
    from .goletar import load_goletar
    return load_goletar(path, config, **kw)


def _piditar(path, config, **kw):
    from .piditar import load_piditar
    return load_piditar(path, config, **kw)


def _llama(path, _config, dtype=None, **kw):
    if dtype not in (None, "quantized"):
        raise ValueError(f"a GGUF model runs its own quantized weights, not {dtype}")
    return load_llama(path, **kw)


FOLDER_ARCHITECTURES = {"Goletar": _goletar, "Piditar": _piditar}
GGUF_ARCHITECTURES = {a: _llama for a in ("llama", "qwen2", "qwen3", "granite")}


def load_model(path, **kw):
    """A finalized model from a folder (config.json, model.safetensors) or a GGUF file."""
    path = os.fspath(path)
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
        arch, known = config.get("architecture"), FOLDER_ARCHITECTURES
    else:
        with GgufFile(path) as g:
            arch, config = g.metadata.get("general.architecture", "llama"), None
        known = GGUF_ARCHITECTURES
    if arch not in known:
        raise ValueError(f"architecture {arch!r} is not one of {sorted(known)}")
    return known[arch](path, config, **kw)
