"""Girulorn: a decoder whose sublayers read the residual itself and are normed on the way back, with gated linear attention
and grouped-query attention (distance bias, softmax sink, keys and values shared between layers) in any order and
routed feed-forwards with a shared expert.  Reads its config.json and maps its tensors onto a layered model
(rew_b200/layered.py).
"""
import json
import os

from .layered import LayeredConfig, LayerSpec

ARCHITECTURE = "Girulorn"


def _feed_forward(mlp):
    if mlp is None:
        return dict(ff="none")
    if mlp["kind"] != "moe":
        raise ValueError("config.json: unknown feed-forward kind %r" % (mlp["kind"],))
    shared = mlp.get("shared")
    return dict(ff="experts", ffn=int(mlp["expert"]["ff"]), experts=int(mlp["router"]["experts"]), top_k=int(mlp["router"]["top"]),
                renormalize=True, expert_gated=True, router_bias=True, shared_ffn=int(shared["ff"]) if shared else 0)


def _layer(entry, i, shapes):
    m, p = entry["mixer"], "l%d.mix." % i
    base = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), **_feed_forward(entry.get("mlp")))
    if entry["type"] == "gla":
        return LayerSpec(mixer="gla", tau=float(m["tau"]), decay_rank=int(shapes[p + "a1"][0]), **base)
    if entry["type"] != "attention":
        raise ValueError("config.json: unknown mixer %r" % (entry["type"],))
    temp = m.get("q_temp") or {}
    src = m.get("kv_from")
    return LayerSpec(mixer="attention", kv_heads=int(m["kv_heads"]), kv_from=-1 if src is None else int(src), scale=float(m["scale"]),
                     qk_norm=True, sink=True, out_gate=True, bias_rows=int(shapes[p + "rel"][0]), bias_max=int(m["bias_max"]),
                     temp_every=int(temp.get("every", 0)), temp_coef=float(temp.get("coef", 0.0)), **base)


def config_from_json(path_or_dict, shapes, **overrides):
    """config.json -> LayeredConfig; shapes {tensor name: shape as stored} gives what config.json leaves to the tensors (rank
    of the decay projection, rows of the bias table).  The file bounds no sequence length: max_seq is the caller's."""
    node = path_or_dict
    if not isinstance(node, dict):
        with open(node) as f:
            node = json.load(f)
    kw = dict(vocab=int(node["vocab"]), d_model=int(node["width"]), eps=float(node["norm"]["eps"]),
              layers=[_layer(e, i, shapes) for i, e in enumerate(node["layers"])], norm_zero_centred=False, block="output_norm",
              own_head=True)
    kw.update(overrides)
    return LayeredConfig(**kw)


def load(model_dir, dtype, max_seq=None, slot=0):
    """CausalLM from a folder with config.json and *.safetensors."""
    from . import safetensors as st
    from .api import CausalLM
    kw = {} if max_seq is None else dict(max_seq=int(max_seq))
    tensors = st.read_safetensors_dir(model_dir)
    cfg = config_from_json(os.path.join(model_dir, "config.json"), {k: v.shape for k, v in tensors.items()}, dtype=dtype, **kw)
    return CausalLM(cfg, slot).load(cfg.canonical_tensors(tensors))


# Benchmark configuration (shapes only; weights are synthetic).
def moe_lite(**kw):
    """As many layers, the width, heads, experts, expert and shared expert widths of the DeepSeek-V2-Lite shape; gated linear
    attention and attention take turns."""
    from . import _lib
    moe = dict(ff="experts", ffn=1408, experts=64, top_k=6, renormalize=True, expert_gated=True, router_bias=True, shared_ffn=2816)
    gla = LayerSpec(mixer="gla", heads=16, dim=128, vdim=128, tau=16.0, decay_rank=16, **moe)
    att = LayerSpec(mixer="attention", heads=16, kv_heads=16, dim=128, vdim=128, scale=128 ** -0.5, bias_rows=32, bias_max=128,
                    temp_every=1024, temp_coef=0.1, sink=True, **moe)
    layers = [att if i % 2 else gla for i in range(27)]
    return LayeredConfig(**{**dict(vocab=102400, d_model=2048, layers=layers, eps=1e-6, norm_zero_centred=False, block="output_norm",
                                   own_head=True, max_seq=2304, dtype=_lib.BF16), **kw})
