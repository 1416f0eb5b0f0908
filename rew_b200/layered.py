"""Layered models: decoders whose layers are described one by one (rewb200_model_create_layers).

LayerSpec describes the mixer and the feed-forward of one layer, LayeredConfig the stack.  tensor_specs lists the
logical tensors in the order rewb200_model_set_tensor indexes them; Linear weights are [in, out].
"""
from dataclasses import dataclass, field

import numpy as np

from . import _lib


MIXERS = {"latent": 1, "attention": 2, "gla": 3, "delta": 4, "lru": 5}
BLOCKS = ("parallel", "output_norm", "parallel_one_norm", "sandwich")
FF_ACTS = ("gated_silu", "gelu_tanh")
SINKS = {False: 0, True: 1, "one": 2}


@dataclass
class LayerSpec:
    """One layer: a mixer and a feed-forward.

    mixer "latent": latent attention; "attention": grouped-query attention with a short convolution, rotation, a learned
    distance bias, query / key norms, a query temperature, a softmax sink, a window with kept first keys, normed values and
    mixed heads, each optional; "gla": gated linear attention with a state per sequence; "delta": gated delta rule; "lru":
    linear recurrent unit whose `heads` blocks have `dim` (= `vdim`) channels each.  `beside`: a second mixer (a LayerSpec of
    which only the mixer counts) on the same input.
    """
    heads: int
    dim: int                    # query / key features per head (latent: the unrotated ones)
    vdim: int
    mixer: str = "latent"
    scale: float = 1.0          # of the attention scores
    out_gate: object = True     # latent, attention: a sigmoid gate per head on the output; "element" (attention): per feature
    sink: object = False        # latent, attention: a further term of the softmax denominator, exp of a learned number per
                                # head (True) or one ("one")
    kv_from: int = -1           # latent, attention: layer whose cached latents, or keys and values, are used; -1: its own
    rope_base: float = 10000.0
    rope_dims: int = None       # latent: rotated features of the rot_dim part, interleaved pairs (None: all); attention:
                                # rotated features of every head, pairs (i, i + rope_dims / 2) (None: none)
    # latent
    rot_dim: int = 0            # rotated features per head; the key part is shared by all heads
    q_rank: int = 0
    kv_rank: int = 0
    window: int = 0             # latent, attention: keys a query sees, itself included; 0: all
    # attention
    kv_heads: int = 0           # delta too
    conv_taps: int = 0          # causal convolution over time per channel of queries and keys (delta: values too; lru); 0: none
    qkv_bias: bool = False
    rope_pairs: bool = False    # features (2i, 2i + 1) are rotated together
    v_norm: bool = False        # values divided by their root mean square
    keep_first: int = 0         # first keys of the sequence that every query sees besides its window
    head_mix: bool = False      # after the softmax the heads' weights are mixed by a matrix
    values_from_keys: bool = False   # the values are the keys as they leave the convolution; there is no value projection
    qk_norm: bool = True
    bias_rows: int = 0          # rows of the distance bias table; 0: no bias
    bias_max: int = 0           # distance at which the buckets end
    temp_every: int = 0         # query temperature 1 + temp_coef ln(floor((p + 1) / temp_every) + 1); 0: none
    temp_coef: float = 0.0
    # gla
    decay_rank: int = 0
    tau: float = 1.0
    # feed-forward
    ff: str = "dense"           # "none", "dense" or "experts"
    ff_act: str = "gated_silu"  # dense: or "gelu_tanh", W_down gelu(W_up x)
    ff_bias: bool = False       # dense "gelu_tanh": biases
    ffn: int = 0                # hidden width of the dense feed-forward or of one expert
    experts: int = 0
    top_k: int = 0
    renormalize: bool = False   # routing weights divided by the sum of the chosen ones
    router_scale: float = 1.0   # ... times this
    expert_gated: bool = False  # gated SiLU experts; False: W_down relu(W_up x)^2
    router_bias: bool = False
    shared_ffn: int = 0         # hidden width of the shared expert; 0: none
    shared_gate: bool = False   # its output is scaled by a sigmoid of a projection of the input
    beside: object = None       # a second mixer
    beside_names: tuple = ("", "")   # prefixes of the tensor names of the two mixers
    mix_scale: float = 1.0      # attention, delta, lru: factor of the mixer's output

    def to_c(self, beside=0):
        kinds = ("none", "dense", "experts")
        if self.ff not in kinds:
            raise ValueError("unknown feed-forward %r" % (self.ff,))
        if self.mixer not in MIXERS:
            raise ValueError("unknown mixer %r" % (self.mixer,))
        return _lib.Layer(mixer=MIXERS[self.mixer], heads=self.heads, dim=self.dim, rot_dim=self.rot_dim, vdim=self.vdim, q_rank=self.q_rank,
                          kv_rank=self.kv_rank, window=self.window,
                          rope_dims=self.rope_dims if self.rope_dims is not None else self.rot_dim,
                          out_gate=self.gate_kind, ff=kinds.index(self.ff), ffn=self.ffn,
                          experts=self.experts, top_k=self.top_k, renormalize=int(self.renormalize),
                          expert_gated=int(self.expert_gated), rope_base=self.rope_base, scale=self.scale, kv_heads=self.kv_heads,
                          kv_from=self.kv_from, qk_norm=int(self.qk_norm), sink=SINKS[self.sink], bias_rows=self.bias_rows,
                          bias_max=self.bias_max, temp_every=self.temp_every, temp_coef=self.temp_coef, decay_rank=self.decay_rank,
                          tau=self.tau, router_bias=int(self.router_bias), shared_ffn=self.shared_ffn, conv_taps=self.conv_taps,
                          values_from_keys=int(self.values_from_keys), router_scale=self.router_scale, shared_gate=int(self.shared_gate),
                          qkv_bias=int(self.qkv_bias), rope_pairs=int(self.rope_pairs), v_norm=int(self.v_norm),
                          keep_first=self.keep_first, head_mix=int(self.head_mix), ff_act=FF_ACTS.index(self.ff_act),
                          ff_bias=int(self.ff_bias), beside=beside, mix_scale=self.mix_scale)

    @property
    def gate_kind(self):
        """0 none, 1 per head, 2 per feature of the output."""
        return 0 if self.mixer not in ("latent", "attention") else 2 if self.out_gate == "element" else int(bool(self.out_gate))

    def mixer_specs(self, d):
        """[(name, shape)] of the mixer's tensors, Linear weights [in, out]."""
        H, K, V, own = self.heads, self.dim, self.vdim, self.kv_from < 0
        if self.mixer == "latent":
            specs = [("dq", (d, self.q_rank)), ("dq.norm", (self.q_rank,)), ("uq", (self.q_rank, H * (K + self.rot_dim)))]
            if own:
                specs += [("dkv", (d, self.kv_rank + self.rot_dim)), ("dkv.norm", (self.kv_rank,))]
            specs += [("uk", (self.kv_rank, H * K)), ("uv", (self.kv_rank, H * V))]
            if self.sink is True:
                specs.append(("sink", (H,)))
        elif self.mixer == "attention":
            specs = [("q", (d, H * K))]
            if own:
                specs += [("k", (d, self.kv_heads * K))] + ([] if self.values_from_keys else [("v", (d, self.kv_heads * V))])
            if self.conv_taps:
                specs += [("q.conv", (H * K, self.conv_taps))] + ([("k.conv", (self.kv_heads * K, self.conv_taps))] if own else [])
            if self.qk_norm:
                specs += [("q.norm", (K,))] + ([("k.norm", (K,))] if own else [])
            if self.bias_rows:
                specs.append(("rel", (self.bias_rows, H)))
            if self.sink is True:
                specs.append(("sink", (H,)))
            if self.head_mix:
                specs.append(("talk", (H, H)))
            if self.qkv_bias:
                specs += [("q.b", (H * K,))] + ([("k.b", (self.kv_heads * K,))] + ([] if self.values_from_keys else [("v.b", (self.kv_heads * V,))])
                                                if own else [])
        elif self.mixer == "gla":
            specs = [("q", (d, H * K)), ("k", (d, H * K)), ("v", (d, H * V)), ("a1", (d, self.decay_rank)),
                     ("a2", (self.decay_rank, H * K)), ("a2.b", (H * K,)), ("g", (d, H * V)), ("norm", (V,))]
        elif self.mixer == "delta":
            G, taps = self.kv_heads, self.conv_taps
            specs = [("q", (d, G * K)), ("k", (d, G * K)), ("v", (d, H * V)), ("q.conv", (G * K, taps)), ("k.conv", (G * K, taps)),
                     ("v.conv", (H * V, taps)), ("b", (d, H)), ("a", (d, H)), ("A_log", (H,)), ("dt_bias", (H,)), ("g", (d, H * V)),
                     ("norm", (V,))]
        else:
            n = H * K
            specs = [("y", (d, n)), ("y.b", (n,)), ("x", (d, n)), ("x.b", (n,)), ("conv", (n, self.conv_taps)), ("conv.b", (n,)),
                     ("ra", (n, K)), ("ri", (n, K)), ("ra.b", (n,)), ("ri.b", (n,)), ("lam", (n,))]
        if self.gate_kind:
            specs.append(("g", (d, H if self.gate_kind == 1 else H * V)))
        return specs + [("o", (H * V, d))]

    def step_traffic(self, d, batch, ctx):
        """Elements a decode step of `batch` sequences at context ctx reads or writes for the mixer, without
        recurrent state."""
        n = sum(s[0] * s[1] for _, s in self.mixer_specs(d) if len(s) == 2)
        if self.mixer == "latent":
            seen = min(ctx, self.window) if self.window else ctx
            return n + batch * seen * (self.kv_rank + self.rot_dim)
        if self.mixer == "attention":
            seen = min(ctx, self.window + self.keep_first) if self.window else ctx
            return n + batch * seen * self.kv_heads * (self.dim + self.vdim)
        return n

    @property
    def state_elements(self):
        """f32 elements of recurrent state per sequence."""
        if self.mixer == "attention" and self.conv_taps:
            return (self.conv_taps - 1) * (self.heads + (self.kv_heads if self.kv_from < 0 else 0)) * self.dim
        if self.mixer == "delta":
            return self.heads * self.dim * self.vdim + (self.conv_taps - 1) * (2 * self.kv_heads * self.dim + self.heads * self.vdim)
        if self.mixer == "lru":
            return self.conv_taps * self.heads * self.dim
        return self.heads * self.dim * self.vdim if self.mixer == "gla" else 0


@dataclass
class LayeredConfig:
    vocab: int
    d_model: int
    layers: list                # LayerSpec
    eps: float = 1e-6
    loop: tuple = None          # (start, stop, times): layers[start:stop] are repeated, `times` passes in all
    norm_zero_centred: bool = True   # block and final norm weights are stored as the distance from one
    block: str = "parallel"     # "parallel": x += mixer(norm1 x) + ff(norm2 x); "output_norm": x += norm1(mixer x), x += norm2(ff x);
                                # "parallel_one_norm": x += mixer(h) + ff(h), h = norm1 x; "sandwich": x += norm1b(mixer(norm1 x)),
                                # x += norm2b(ff(norm2 x))
    own_head: bool = False      # the output head is a tensor of its own; False: the embedding table
    logit_softcap: float = 0.0  # logits <- cap * tanh(logits / cap); 0: none
    embed_scale: float = 1.0    # "sandwich": factor of the token embeddings
    bigram: tuple = None        # "sandwich": (buckets, mul_prev, mul_cur) of a table added to the embeddings: row
                                # (previous id * mul_prev + id * mul_cur) mod buckets, row `buckets` for a first token
    loop_in: bool = False       # "sandwich": every pass of the loop opens with x <- W [x; embeddings]
    max_seq: int = 4096
    dtype: int = _lib.F32
    tp_size: int = field(default=1, init=False)
    n_routed: int = field(default=0, init=False)

    @property
    def n_layers(self):
        return len(self.layers)

    @property
    def top_k(self):
        return max([l.top_k for l in self.layers if l.ff == "experts"] or [0])

    @property
    def layer_runs(self):
        """Layer index of every layer run of a step, in order."""
        n = list(range(self.n_layers))
        if not self.loop:
            return n
        a, b, k = self.loop
        return n[:a] + n[a:b] * k + n[b:]

    def step_bytes(self, batch, ctx):
        """Bytes a decode step of `batch` sequences streams at context ctx: every layer run's weights (a loop reads them once
        a pass), the lm_head, the cache rows the windows see and the recurrent state."""
        es = 2 if self.dtype == _lib.BF16 else 4
        d, total, state = self.d_model, self.d_model * self.vocab, 0
        for i in self.layer_runs:
            l = self.layers[i]
            for m in (l, l.beside):
                if m is not None:
                    total += m.step_traffic(d, batch, ctx)
                    state += 2 * batch * m.state_elements          # read and written
            if l.ff == "dense":
                total += (2 if l.ff_act == "gelu_tanh" else 3) * d * l.ffn
            elif l.ff == "experts":
                total += d * l.experts + min(l.experts, batch * l.top_k) * (3 if l.expert_gated else 2) * d * l.ffn + 3 * d * l.shared_ffn
        if self.loop_in and self.loop:
            total += self.loop[2] * 2 * d * d
        return total * es + state * 4

    def create(self, slot, out):
        """rewb200_model_create_layers into the handle `out`."""
        import ctypes as C
        base = _lib.Config(vocab=self.vocab, d_model=self.d_model, n_layers=self.n_layers, max_seq=self.max_seq, eps=self.eps,
                           dtype=self.dtype, tp_size=1, ep_size=1)
        second = [l.beside for l in self.layers if l.beside is not None]
        descs, n = [], 0
        for l in self.layers:
            n += l.beside is not None
            descs.append(l.to_c(beside=n if l.beside is not None else 0))
        descs += [m.to_c() for m in second]
        arr = (_lib.Layer * len(descs))(*descs)
        a, b, k = self.loop or (0, 0, 0)
        buckets, mul_prev, mul_cur = self.bigram or (0, 0, 0)
        stack = _lib.Stack(loop_start=a, loop_stop=b, loop_times=k, norm_zero_centred=int(self.norm_zero_centred),
                           block=BLOCKS.index(self.block), own_head=int(self.own_head), logit_softcap=self.logit_softcap,
                           embed_scale=self.embed_scale, bigram_buckets=buckets, bigram_mul_prev=mul_prev, bigram_mul_cur=mul_cur,
                           loop_in=int(bool(self.loop) and self.loop_in), n_beside=len(second))
        _lib.check(_lib.lib().rewb200_model_create_layers(slot, C.byref(base), arr, C.byref(stack), out))

    def tensor_specs(self):
        """[(name, shape)] in canonical order."""
        d = self.d_model
        specs = [("embed", (self.vocab, d))]
        if self.bigram:
            specs.append(("bigram", (self.bigram[0] + 1, d)))
        if self.loop:
            specs.append(("loop.in", (2 * d, d)) if self.loop_in else ("loop.step", (self.loop[2], d)))
        back = ("", "b") if self.block == "sandwich" else ("",)
        for i, l in enumerate(self.layers):
            p = "l%d." % i
            specs += [(p + "norm1" + s, (d,)) for s in back]
            for m, sub in zip((l, l.beside), l.beside_names):
                if m is not None:
                    specs += [(p + "mix." + sub + n, shape) for n, shape in m.mixer_specs(d)]
            if l.ff == "none":
                continue
            if self.block != "parallel_one_norm":
                specs += [(p + "norm2" + s, (d,)) for s in back]
            if l.ff == "dense" and l.ff_act == "gelu_tanh":
                for n, shape in (("up", (d, l.ffn)), ("down", (l.ffn, d))):
                    specs += [(p + "mlp." + n, shape)] + ([(p + "mlp." + n + ".b", shape[1:])] if l.ff_bias else [])
            elif l.ff == "dense":
                specs += [(p + "mlp.gate", (d, l.ffn)), (p + "mlp.up", (d, l.ffn)), (p + "mlp.down", (l.ffn, d))]
            else:
                specs.append((p + "mlp.router", (d, l.experts)))
                if l.router_bias:
                    specs.append((p + "mlp.router.b", (l.experts,)))
                for e in range(l.experts):
                    q = p + "mlp.e%d." % e
                    if l.expert_gated:
                        specs.append((q + "gate", (d, l.ffn)))
                    specs += [(q + "up", (d, l.ffn)), (q + "down", (l.ffn, d))]
                if l.shared_ffn:
                    q = p + "mlp.shared."
                    specs += [(q + "gate", (d, l.shared_ffn)), (q + "up", (d, l.shared_ffn)), (q + "down", (l.shared_ffn, d))]
                    if l.shared_gate:
                        specs.append((q + "sg", (d, 1)))
        specs.append(("final.norm", (d,)))
        if self.own_head:
            specs.append(("head", (d, self.vocab)))
        return specs

    def canonical_tensors(self, tensors, tables=("embed", "bigram", "loop.step", "mix.rel", ".conv", ".talk", ".ra", ".ri")):
        """The canonical list from {name: array} of a file whose Linear weights are [out, in]; names that end in one of
        `tables` are matrices that are no Linear and stay as they are ([heads, ..] stacks of the file as one matrix)."""
        out = []
        for name, shape in self.tensor_specs():
            if name not in tensors:
                raise KeyError("model.safetensors: missing tensor " + name)
            t = np.asarray(tensors[name], np.float32)
            if t.ndim > len(shape):
                t = t.reshape((-1,) + t.shape[t.ndim - len(shape) + 1:])
            elif t.ndim == 2 and not name.endswith(tables):
                t = t.T
            if tuple(t.shape) != tuple(shape):
                raise ValueError("model.safetensors: %s is %r, config.json asks for %r" % (name, t.shape, tuple(shape)))
            out.append(np.ascontiguousarray(t))
        return out
