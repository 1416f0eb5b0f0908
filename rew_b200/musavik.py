"""Musavik: a decoder whose sublayers are normed on both sides, with two kinds of mixers in any order: a recurrent block with
a linear recurrent unit, and windowed attention (kept first keys, mixed heads) beside a gated delta rule; token embeddings
with a bigram table, and a range of layers that runs several times on a mix of the stream and the embeddings.  Reads its
config.json and maps its tensors onto a layered model (rew_b200/layered.py).
"""
import json
import os

from .layered import LayeredConfig, LayerSpec

ARCHITECTURE = "Musavik"


def _feed_forward(mlp):
    if mlp is None:
        return dict(ff="none")
    if mlp["kind"] != "dense":
        raise ValueError("config.json: unknown feed-forward kind %r" % (mlp["kind"],))
    return dict(ff="dense", ffn=int(mlp["ff"]), ff_act="gelu_tanh", ff_bias=True)


def _attention(m, scale, **kw):
    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    return LayerSpec(mixer="attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                     scale=float(m["scale"]), out_gate="element", qkv_bias=True, qk_norm=True, v_norm=True, rope_pairs=True,
                     rope_base=float(rot.get("base", 10000.0)), rope_dims=int(rot.get("dims", 0)), window=int(mask.get("size") or 0),
                     keep_first=int(mask.get("keep_first") or 0), head_mix=True, mix_scale=scale, **kw)


def _delta(m, scale):
    return LayerSpec(mixer="delta", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                     conv_taps=int(m["conv"]), mix_scale=scale, ff="none")


def _layer(entry):
    m, ff = entry["mixer"], _feed_forward(entry.get("mlp"))
    if entry["type"] == "rglru":
        width, blocks = int(m["width"]), int(m["blocks"])
        if width % blocks:
            raise ValueError("config.json: %d channels do not divide into %d blocks" % (width, blocks))
        return LayerSpec(mixer="lru", heads=blocks, dim=width // blocks, vdim=width // blocks, conv_taps=int(m["conv"]), **ff)
    if entry["type"] == "parallel":
        return _attention(m["left"], float(m["left_scale"]), beside=_delta(m["right"], float(m["right_scale"])),
                          beside_names=("left.", "right."), **ff)
    raise ValueError("config.json: unknown mixer %r" % (entry["type"],))


def config_from_json(path_or_dict, **overrides):
    """config.json -> LayeredConfig.  The file bounds no sequence length: max_seq is the caller's."""
    node = path_or_dict
    if not isinstance(node, dict):
        with open(node) as f:
            node = json.load(f)
    emb, loop = node.get("embedding") or {}, node.get("loop")
    big = emb.get("bigram")
    kw = dict(vocab=int(node["vocab"]), d_model=int(node["width"]), eps=float(node["norm"]["eps"]), layers=[_layer(e) for e in node["layers"]],
              norm_zero_centred=True, block="sandwich", own_head=True, embed_scale=float(emb.get("scale", 1.0)),
              bigram=(int(big["buckets"]), int(big["mul_prev"]), int(big["mul_cur"])) if big else None,
              loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None, loop_in=bool(loop))
    kw.update(overrides)
    return LayeredConfig(**kw)


def load(model_dir, dtype, max_seq=None, slot=0):
    """CausalLM from a folder with config.json and *.safetensors."""
    from . import safetensors as st
    from .api import CausalLM
    kw = {} if max_seq is None else dict(max_seq=int(max_seq))
    cfg = config_from_json(os.path.join(model_dir, "config.json"), dtype=dtype, **kw)
    return CausalLM(cfg, slot).load(cfg.canonical_tensors(st.read_safetensors_dir(model_dir)))


# Benchmark configuration (shapes only; weights are synthetic).
def dense_8b(**kw):
    """As many layers, the width and about the weights of the 8B Llama shape, mixers and feed-forwards alike; recurrent blocks
    and attention beside the delta rule take turns, without a loop."""
    from . import _lib
    ff = dict(ff="dense", ffn=21504, ff_act="gelu_tanh", ff_bias=True)
    delta = LayerSpec(mixer="delta", heads=8, kv_heads=8, dim=128, vdim=128, conv_taps=4, ff="none")
    both = LayerSpec(mixer="attention", heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, out_gate="element", qkv_bias=True, qk_norm=True,
                     v_norm=True, rope_pairs=True, rope_base=500000.0, rope_dims=128, window=1024, keep_first=64, head_mix=True, mix_scale=0.5,
                     beside=delta, beside_names=("left.", "right."), **ff)
    lru = LayerSpec(mixer="lru", heads=12, dim=256, vdim=256, conv_taps=4, **ff)
    return LayeredConfig(**{**dict(vocab=128256, d_model=4096, layers=[both if i % 2 else lru for i in range(32)], eps=1e-5, block="sandwich",
                                   own_head=True, embed_scale=64.0, bigram=(16384, 1009, 7), max_seq=2560, dtype=_lib.BF16), **kw})
