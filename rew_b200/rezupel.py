"""Rezupel: a decoder of parallel blocks with windowed latent attention, dense or routed feed-forwards, and a range of
layers that runs several times.  Reads its config.json and maps its tensors onto a layered model (rew_b200/layered.py).
"""
import json
import os

from .layered import LayeredConfig, LayerSpec

ARCHITECTURE = "Rezupel"


def _feed_forward(mlp):
    if mlp is None:
        return dict(ff="none")
    if mlp["kind"] == "dense":
        return dict(ff="dense", ffn=int(mlp["ff"]))
    if mlp["kind"] == "moe":
        return dict(ff="experts", ffn=int(mlp["expert"]["ff"]), experts=int(mlp["router"]["experts"]), top_k=int(mlp["router"]["top"]))
    raise ValueError("config.json: unknown feed-forward kind %r" % (mlp["kind"],))


def _layer(entry):
    if entry["type"] != "latent_attention":
        raise ValueError("config.json: unknown mixer %r" % (entry["type"],))
    m = entry["mixer"]
    mask = m.get("mask") or {}
    return LayerSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), q_rank=int(m["q_rank"]),
                     kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), window=int(mask.get("size") or 0),
                     rope_base=float(m["rot"]["base"]), rope_dims=int(m["rot"]["dims"]), out_gate=True, **_feed_forward(entry.get("mlp")))


def config_from_json(path_or_dict, **overrides):
    """config.json -> LayeredConfig.  The file bounds no sequence length: max_seq is the caller's."""
    node = path_or_dict
    if not isinstance(node, dict):
        with open(node) as f:
            node = json.load(f)
    loop = node.get("loop")
    kw = dict(vocab=int(node["vocab"]), d_model=int(node["width"]), eps=float(node["norm"]["eps"]),
              layers=[_layer(e) for e in node["layers"]], norm_zero_centred=True,
              loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)
    kw.update(overrides)
    return LayeredConfig(**kw)


def canonical_tensors(cfg, tensors):
    """The canonical list from {name: array}; the file's Linear weights are [out, in], the backend's [in, out]."""
    return cfg.canonical_tensors(tensors)


def load(model_dir, dtype, max_seq=None, slot=0):
    """CausalLM from a folder with config.json and *.safetensors."""
    from . import safetensors as st
    from .api import CausalLM
    kw = {} if max_seq is None else dict(max_seq=int(max_seq))
    cfg = config_from_json(os.path.join(model_dir, "config.json"), dtype=dtype, **kw)
    return CausalLM(cfg, slot).load(canonical_tensors(cfg, st.read_safetensors_dir(model_dir)))


# Benchmark configurations (shapes only; weights are synthetic).
def dense_8b(**kw):
    """Layers of the width, heads and feed-forward of the 8B Llama shape."""
    from . import _lib
    layer = LayerSpec(heads=32, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512, scale=192 ** -0.5, window=1024,
                      rope_base=500000.0, ff="dense", ffn=14336)
    return LayeredConfig(**{**dict(vocab=128256, d_model=4096, layers=[layer] * 32, eps=1e-5, max_seq=2048, dtype=_lib.BF16), **kw})


def moe_lite(**kw):
    """As many layer runs, the width, heads, experts and expert width of the DeepSeek-V2-Lite shape; 13 layers run twice."""
    from . import _lib
    mix = dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512, scale=192 ** -0.5, window=1024, rope_base=10000.0)
    layers = [LayerSpec(ff="dense", ffn=10944, **mix)] + [LayerSpec(ff="experts", ffn=1408, experts=64, top_k=6, **mix)] * 13
    return LayeredConfig(**{**dict(vocab=102400, d_model=2048, layers=layers, loop=(1, 14, 2), eps=1e-6, max_seq=2048, dtype=_lib.BF16), **kw})
