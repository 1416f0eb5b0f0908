"""Layered models: decoders whose layers are described one by one (rewb200_model_create_layers).

LayerSpec describes the mixer and the feed-forward of one layer, LayeredConfig the stack.  tensor_specs lists the
logical tensors in the order rewb200_model_set_tensor indexes them; Linear weights are [in, out].
"""
from dataclasses import dataclass, field

from . import _lib


@dataclass
class LayerSpec:
    """Latent attention and a feed-forward, both reading their own norm of the layer's input."""
    heads: int
    dim: int                    # unrotated query / key features per head
    rot_dim: int                # rotated ones; the key part is shared by all heads
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int = 0             # keys a query sees, itself included; 0: all
    rope_base: float = 10000.0
    rope_dims: int = None       # rotated features of the rot_dim part (None: all)
    out_gate: bool = True
    ff: str = "dense"           # "none", "dense" (gated SiLU) or "experts"
    ffn: int = 0                # hidden width of the dense feed-forward or of one expert
    experts: int = 0
    top_k: int = 0
    renormalize: bool = False   # routing weights divided by the sum of the chosen ones
    expert_gated: bool = False  # gated SiLU experts; False: W_down relu(W_up x)^2

    def to_c(self):
        kinds = ("none", "dense", "experts")
        if self.ff not in kinds:
            raise ValueError("unknown feed-forward %r" % (self.ff,))
        return _lib.Layer(mixer=1, heads=self.heads, dim=self.dim, rot_dim=self.rot_dim, vdim=self.vdim, q_rank=self.q_rank,
                          kv_rank=self.kv_rank, window=self.window,
                          rope_dims=self.rot_dim if self.rope_dims is None else self.rope_dims, out_gate=int(self.out_gate),
                          ff=kinds.index(self.ff), ffn=self.ffn, experts=self.experts, top_k=self.top_k,
                          renormalize=int(self.renormalize), expert_gated=int(self.expert_gated), rope_base=self.rope_base,
                          scale=self.scale, reserved=0)


@dataclass
class LayeredConfig:
    vocab: int
    d_model: int
    layers: list                # LayerSpec
    eps: float = 1e-6
    loop: tuple = None          # (start, stop, times): layers[start:stop] are repeated, `times` passes in all
    norm_zero_centred: bool = True   # block and final norm weights are stored as the distance from one
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
        a pass), the lm_head, and the cache rows the windows see."""
        es = 2 if self.dtype == _lib.BF16 else 4
        d, total = self.d_model, self.d_model * self.vocab
        for i in self.layer_runs:
            l = self.layers[i]
            total += d * (l.q_rank + l.kv_rank + l.rot_dim + (l.heads if l.out_gate else 0)) + l.q_rank * l.heads * (l.dim + l.rot_dim)
            total += l.kv_rank * l.heads * (l.dim + l.vdim) + l.heads * l.vdim * d
            if l.ff == "dense":
                total += 3 * d * l.ffn
            elif l.ff == "experts":
                total += d * l.experts + min(l.experts, batch * l.top_k) * (3 if l.expert_gated else 2) * d * l.ffn
            seen = min(ctx, l.window) if l.window else ctx
            total += batch * seen * (l.kv_rank + l.rot_dim)
        return total * es

    def create(self, slot, out):
        """rewb200_model_create_layers into the handle `out`."""
        import ctypes as C
        base = _lib.Config(vocab=self.vocab, d_model=self.d_model, n_layers=self.n_layers, max_seq=self.max_seq, eps=self.eps,
                           dtype=self.dtype, tp_size=1, ep_size=1)
        arr = (_lib.Layer * self.n_layers)(*[l.to_c() for l in self.layers])
        a, b, k = self.loop or (0, 0, 0)
        stack = _lib.Stack(loop_start=a, loop_stop=b, loop_times=k, norm_zero_centred=int(self.norm_zero_centred))
        _lib.check(_lib.lib().rewb200_model_create_layers(slot, C.byref(base), arr, C.byref(stack), out))

    def tensor_specs(self):
        """[(name, shape)] in canonical order."""
        d = self.d_model
        specs = [("embed", (self.vocab, d))]
        if self.loop:
            specs.append(("loop.step", (self.loop[2], d)))
        for i, l in enumerate(self.layers):
            p = "l%d." % i
            x = p + "mix."
            specs += [(p + "norm1", (d,)), (x + "dq", (d, l.q_rank)), (x + "dq.norm", (l.q_rank,)),
                      (x + "uq", (l.q_rank, l.heads * (l.dim + l.rot_dim))), (x + "dkv", (d, l.kv_rank + l.rot_dim)),
                      (x + "dkv.norm", (l.kv_rank,)), (x + "uk", (l.kv_rank, l.heads * l.dim)),
                      (x + "uv", (l.kv_rank, l.heads * l.vdim))]
            if l.out_gate:
                specs.append((x + "g", (d, l.heads)))
            specs.append((x + "o", (l.heads * l.vdim, d)))
            if l.ff == "none":
                continue
            specs.append((p + "norm2", (d,)))
            if l.ff == "dense":
                specs += [(p + "mlp.gate", (d, l.ffn)), (p + "mlp.up", (d, l.ffn)), (p + "mlp.down", (l.ffn, d))]
            else:
                specs.append((p + "mlp.router", (d, l.experts)))
                for e in range(l.experts):
                    q = p + "mlp.e%d." % e
                    if l.expert_gated:
                        specs.append((q + "gate", (d, l.ffn)))
                    specs += [(q + "up", (d, l.ffn)), (q + "down", (l.ffn, d))]
        specs.append(("final.norm", (d,)))
        return specs
