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


# Benchmark configurations (shapes only; weights are synthetic).
def _turns(n, attention, latent, first_ff, ff):
    """n layers, attention and latent attention in turn; every other latent layer reads the latents of the one before it."""
    layers, own = [], -1
    for i in range(n):
        f = first_ff if i == 0 else ff
        if i % 2 == 0:
            layers.append(LayerSpec(mixer="attention", conv_taps=4, values_from_keys=True, qk_norm=False, sink="one", out_gate=False, **attention, **f))
        else:
            src, own = (own, -1) if own >= 0 else (-1, i)
            layers.append(LayerSpec(mixer="latent", sink=True, out_gate=False, kv_from=src, **latent, **f))
    return layers


def dense_8b(**kw):
    """Layers of the width, heads and feed-forward of the 8B Llama shape."""
    from . import _lib
    ff = dict(ff="dense", ffn=14336)
    layers = _turns(32, dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, rope_base=500000.0, rope_dims=128),
                    dict(heads=32, dim=128, vdim=128, q_rank=1536, kv_rank=512, scale=128 ** -0.5, window=1024), ff, ff)
    return LayeredConfig(**{**dict(vocab=128256, d_model=4096, layers=layers, eps=1e-5, norm_zero_centred=False, block="parallel_one_norm",
                                   own_head=True, logit_softcap=50.0, max_seq=2560, dtype=_lib.BF16), **kw})


def moe_lite(**kw):
    """As many layers, the width, heads, experts, expert and shared expert widths of the DeepSeek-V2-Lite shape."""
    from . import _lib
    moe = dict(ff="experts", ffn=1408, experts=64, top_k=6, renormalize=True, router_scale=1.5, expert_gated=True, shared_ffn=2816, shared_gate=True)
    layers = _turns(27, dict(heads=16, kv_heads=16, dim=128, vdim=128, scale=128 ** -0.5, rope_base=10000.0, rope_dims=128),
                    dict(heads=16, dim=128, vdim=128, q_rank=768, kv_rank=512, scale=128 ** -0.5, window=1024), dict(ff="dense", ffn=10944), moe)
    return LayeredConfig(**{**dict(vocab=102400, d_model=2048, layers=layers, eps=1e-6, norm_zero_centred=False, block="parallel_one_norm",
                                   own_head=True, logit_softcap=50.0, max_seq=1024, dtype=_lib.BF16), **kw})
