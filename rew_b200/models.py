"""Model registry: which family a folder's config.json names, and how it is loaded.

    model = load_model("/path/to/folder", dtype="bfloat16", max_seq=4096)
"""
import json
import os

from . import _lib

DTYPES = {"bfloat16": _lib.BF16, "float32": _lib.F32}


def _is_rezupel(cfg):
    return cfg.get("architecture") == "Rezupel"


def _load_rezupel(path, dtype, max_seq, slot):
    from . import rezupel
    return rezupel.load(path, dtype, max_seq, slot)


def _is_girulorn(cfg):
    return cfg.get("architecture") == "Girulorn"


def _load_girulorn(path, dtype, max_seq, slot):
    from . import girulorn
    return girulorn.load(path, dtype, max_seq, slot)


def _is_kugirax(cfg):
    return cfg.get("architecture") == "Kugirax"


def _load_kugirax(path, dtype, max_seq, slot):
    from . import kugirax
    return kugirax.load(path, dtype, max_seq, slot)


def _is_musavik(cfg):
    return cfg.get("architecture") == "Musavik"


def _load_musavik(path, dtype, max_seq, slot):
    from . import musavik
    return musavik.load(path, dtype, max_seq, slot)


def _is_hf_llama(cfg):
    return cfg.get("model_type") == "llama" or "LlamaForCausalLM" in (cfg.get("architectures") or [])


def _load_hf_llama(path, dtype, max_seq, slot):
    from .api import CausalLM
    kw = {} if max_seq is None else dict(max_seq=int(max_seq))
    return CausalLM.from_hf_snapshot(path, dtype=dtype, slot=slot, **kw)


# (family, does this config.json name it, loader)
FAMILIES = [
    ("rezupel", _is_rezupel, _load_rezupel),
    ("girulorn", _is_girulorn, _load_girulorn),
    ("kugirax", _is_kugirax, _load_kugirax),
    ("musavik", _is_musavik, _load_musavik),
    ("llama", _is_hf_llama, _load_hf_llama),
]


def family_of(cfg):
    """Name of the family a parsed config.json belongs to."""
    for name, match, _ in FAMILIES:
        if match(cfg):
            return name
    raise ValueError("config.json names no model family of this backend (known: %s)" % ", ".join(n for n, _, _ in FAMILIES))


def load_model(path, dtype="bfloat16", max_seq=None, slot=0):
    """The CausalLM of a model folder (config.json and *.safetensors); dtype "bfloat16" or "float32"."""
    with open(os.path.join(path, "config.json")) as f:
        name = family_of(json.load(f))
    load = {n: l for n, _, l in FAMILIES}[name]
    return load(path, DTYPES.get(dtype, dtype), max_seq, slot)
