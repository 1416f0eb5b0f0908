"""Kugirax: a decoder of parallel blocks with one norm, whose mixers are grouped-query attention (short convolution, rotated
halves, values that are the unrotated keys) and windowed latent attention (learned sinks, latents shared between layers) in
any order, dense or routed feed-forwards with a gated shared expert, and capped logits.  Reads its config.json and maps its
tensors onto a layered model (rew_b200/layered.py).
"""
import json
import os

from .layered import LayeredConfig, LayerSpec

ARCHITECTURE = "Kugirax"


def _feed_forward(mlp):
    if mlp is None:
        return dict(ff="none")
    if mlp["kind"] == "dense":
        return dict(ff="dense", ffn=int(mlp["ff"]))
    if mlp["kind"] != "moe":
        raise ValueError("config.json: unknown feed-forward kind %r" % (mlp["kind"],))
    r, shared = mlp["router"], mlp.get("shared")
    return dict(ff="experts", ffn=int(mlp["expert"]["ff"]), experts=int(r["experts"]), top_k=int(r["top"]), renormalize=True,
                router_scale=float(r.get("scale", 1.0)), expert_gated=True, shared_ffn=int(shared["ff"]) if shared else 0,
                shared_gate=bool(shared))


def _layer(entry):
    m = entry["mixer"]
    src = m.get("kv_from")
    base = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), out_gate=False,
                kv_from=-1 if src is None else int(src), **_feed_forward(entry.get("mlp")))
    if entry["type"] == "attention":
        rot = m.get("rot") or {}
        return LayerSpec(mixer="attention", kv_heads=int(m["kv_heads"]), conv_taps=int(m.get("conv") or 0), values_from_keys=True,
                         qk_norm=False, sink="one", rope_base=float(rot.get("base", 10000.0)), rope_dims=int(rot.get("dims", 0)), **base)
    if entry["type"] == "latent_attention":
        mask = m.get("mask") or {}
        return LayerSpec(mixer="latent", q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), window=int(mask.get("size") or 0), sink=True, **base)
    raise ValueError("config.json: unknown mixer %r" % (entry["type"],))


def config_from_json(path_or_dict, **overrides):
    """config.json -> LayeredConfig.  The file bounds no sequence length: max_seq is the caller's."""
    node = path_or_dict
    if not isinstance(node, dict):
        with open(node) as f:
            node = json.load(f)
    kw = dict(vocab=int(node["vocab"]), d_model=int(node["width"]), eps=float(node["norm"]["eps"]), layers=[_layer(e) for e in node["layers"]],
              norm_zero_centred=False, block="parallel_one_norm", own_head=True, logit_softcap=float(node.get("logit_softcap") or 0.0))
    kw.update(overrides)
    return LayeredConfig(**kw)


def load(model_dir, dtype, max_seq=None, slot=0):
    """CausalLM from a folder with config.json and *.safetensors."""
    from . import safetensors as st
    from .api import CausalLM
    kw = {} if max_seq is None else dict(max_seq=int(max_seq))
    cfg = config_from_json(os.path.join(model_dir, "config.json"), dtype=dtype, **kw)
    return CausalLM(cfg, slot).load(cfg.canonical_tensors(st.read_safetensors_dir(model_dir)))
