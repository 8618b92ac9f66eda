"""Decoders described as a list of layers (``ModelConfig.layer_specs``), each with its own mixer, its own sizes and an
optional feed-forward, on an fp32 residual stream:

    x = embed[token] * scale (+ positions[p])
    x = x + wrap1(mixer(norm1(x)));   x = x + wrap2(ff(norm2(x)))     per layer; a layer may have no feed-forward
    logits = head norm(x) * scale

or, where ``layer_norms`` is "parallel", with one norm that both sublayers read, the mixer through a short convolution:

    h = norm1(x);   x = x + residual_mult * (mixer(h + conv(h)) + ff(h))

Norms (``ModelConfig.layer_norms``): Dynamic Tanh, ``tanh(alpha x) * w + b`` (Zhu, Chen, He, LeCun, Liu, "Transformers
without Normalization") with a learned per-column scale as ``wrap``; layer norm with a second layer norm as ``wrap``; no
norm in front and an RMS norm as ``wrap`` (the sublayers then read the stream itself); layer norm in front of both.
Every sublayer hands the activations in front of its output projection to the next norm's ``join``, which projects,
wraps, adds to the residual and normalises in as few kernels as the shapes allow (``ops/dyt.py``, ``ops/layer_norm.py``),
so the model is a flat list of sublayers between the embedding and the head.

Mixers (``MIXERS``): HGRN2 (``models/hgrn2.py``), lightning attention with configured decays
(``models/lightning.py``), latent attention over a compressed cache (``models/mla.py``), grouped-query attention
(``models/gqa.py``), mLSTM (``models/mlstm.py``), attention and a gated delta rule side by side (``models/delta.py``).
Feed-forwards (``make_mlp``): dense with PolyNorm, squared ReLU or SwiGLU, mixture of gated experts, with or without a shared
expert. A layer may run with an earlier layer's weights (``ModelConfig.weights_layer``) and a cache of
its own. A sublayer has ``hidden(y, ctx, cache, rec)``, an output
projection ``o`` (None: ``hidden`` is the sublayer's result) and ``tensors(prefix)``; what a mixer keeps per sequence is
declared by ``ModelConfig.cache_shapes`` / ``state_shapes``, allocated by the rollout engine and passed in.

The Fofosun, Gatolix, Felosun and Dikopel families are built this way. The class shares loading, the head and the engine interface
(``prefill`` / ``decode``) with ``QwenModel``. It is served by the rollout engine and runs forward and backward for
training on one process per replica (data parallelism).
"""

from __future__ import annotations

import contextlib
from dataclasses import dataclass, field
from typing import Any, Iterator

import torch
import torch.nn as nn

from ..ops import dyt, layer_norm as ln, residual_rms as rms, residual_sum as rs
from ..ops.attention import VarlenMeta
from ..ops.gemm import linear, linear_relu2, linear_slices
from ..ops.latent_attn import rotary_tables
from ..ops.lm_head import soft_cap_
from ..ops.moe import ExpertRows, GatedAct, gated_experts, gated_linear, route_tokens
from ..ops.short_conv import ConvTail, conv_prefill
from .config import ModelConfig
from .delta import MixerPair
from .gqa import GroupedAttention
from .hgrn2 import HGRN2
from .lightning import ConstantDecayLightning
from .mla import LatentAttention
from .mlstm import MLSTM
from .qwen import QwenModel

MIXERS = {"hgrn2": HGRN2, "lightning": ConstantDecayLightning, "latent_attention": LatentAttention,
          "grouped_attention": GroupedAttention, "mlstm": MLSTM, "mixer_pair": MixerPair}


class ColumnScale(nn.Module):
    """Learned scale on a sublayer's result."""

    def __init__(self, n: int, dtype, device):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(n, dtype=dtype, device=device))

    def tensors(self, name: str):
        yield name, self.weight


class DynamicTanh(nn.Module):
    def __init__(self, n: int, eps: float, dtype, device):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(n, dtype=dtype, device=device))
        self.bias = nn.Parameter(torch.zeros(n, dtype=dtype, device=device))
        self.alpha = nn.Parameter(torch.full((), 0.5, dtype=dtype, device=device))

    @property
    def args(self):
        return self.alpha, self.weight, self.bias

    def embed(self, ids, table):
        """``(norm(res), res)`` of ``res = table[ids]``."""
        return dyt.embed_dyt(ids, table, self.args)

    def join(self, a, o, wrap: ColumnScale, res):
        """``(norm(res), res)`` of ``res + wrap * (a @ o.T)``: this norm stands in front of the next sublayer."""
        if o is None:
            return dyt.residual_dyt(a, wrap.weight, res, self.args)
        return dyt.linear_residual_dyt(a, o, wrap.weight, res, self.args)

    def tensors(self, name: str):
        yield name, self.weight
        yield name + ".b", self.bias
        yield name + ".alpha", self.alpha


class LayerNorm(nn.Module):
    def __init__(self, n: int, eps: float, dtype, device):
        super().__init__()
        self.eps = eps
        self.weight = nn.Parameter(torch.ones(n, dtype=dtype, device=device))
        self.bias = nn.Parameter(torch.zeros(n, dtype=dtype, device=device))

    @property
    def args(self):
        return self.weight, self.bias

    def embed(self, ids, table):
        return ln.embed_ln(ids, table, self.args, self.eps)

    def join(self, a, o, wrap: "LayerNorm", res):
        """``(norm(res), res)`` of ``res + wrap(a @ o.T)``; without ``o``, ``a`` is the sublayer's result, also as the
        experts' uncombined rows."""
        if isinstance(a, ExpertRows):
            return ln.experts_residual_ln(a, wrap.args, res, self.args, self.eps)
        if o is None:
            return ln.residual_ln(a, wrap.args, res, self.args, self.eps)
        return ln.linear_residual_ln(a, o, wrap.args, res, self.args, self.eps)

    def tensors(self, name: str):
        yield name, self.weight
        yield name + ".b", self.bias


class Stream(nn.Module):
    """No norm: the next sublayer reads the residual stream, rounded to the model's dtype. Results are RMS normed."""

    def __init__(self, n: int, eps: float, dtype, device):
        super().__init__()
        self.eps, self.scale, self.weight = eps, 1.0, None

    def embed(self, ids, table, scale: float = 1.0, pos=None, pos_table=None):
        return rms.embed_residual(ids, table, scale, pos, pos_table, self.weight, self.eps, self.scale)

    def join(self, a, o, wrap: "RMSNorm", res):
        """``(norm(res), res)`` of ``res + wrap(a @ o.T)``; without ``o``, ``a`` is the sublayer's result, also as the
        experts' uncombined rows."""
        tail = (wrap.weight, res, self.weight, self.eps, self.scale)
        if isinstance(a, ExpertRows):
            return rms.experts_residual_rms(a, *tail)
        return rms.residual_rms(a, *tail) if o is None else rms.linear_residual_rms(a, o, *tail)

    def tensors(self, name: str):
        return iter(())


class RMSNorm(Stream):
    """RMS norm of the stream (behind the last layer, where ``scale`` multiplies its result) or of a sublayer's result."""

    def __init__(self, n: int, eps: float, dtype, device, scale: float = 1.0):
        super().__init__(n, eps, dtype, device)
        self.scale = scale
        self.weight = nn.Parameter(torch.ones(n, dtype=dtype, device=device))

    def tensors(self, name: str):
        yield name, self.weight


class SharedLayerNorm(LayerNorm):
    """The layer norm that both sublayers of a layer read. ``conv``: the input convolution behind it (decode steps), see
    :class:`ops.short_conv.ConvTail`; the norm then hands over a pair."""

    def embed(self, ids, table, conv=None, scale: float = 1.0, pos=None, pos_table=None):
        return rs.embed_sum(ids, table, scale, pos, self.args, self.eps, conv)

    def join(self, a: rs.ParallelSum, o, wrap: float, res, conv=None):
        """``(norm(res), res)`` of ``res + wrap * (what both sublayers of the layer in front add)``."""
        return rs.residual_sum(a, wrap, res, self.args, self.eps, conv)


# norm, what is wrapped around a sublayer's result, the latter's checkpoint names, and the norm in front of the head
NORMS = {"dynamic_tanh": (DynamicTanh, lambda n, eps, dtype, device: ColumnScale(n, dtype, device), ("ls1", "ls2"), DynamicTanh),
         "layer_norm": (LayerNorm, LayerNorm, ("norm1b", "norm2b"), LayerNorm),
         "post_rms": (Stream, RMSNorm, ("norm1", "norm2"), RMSNorm),
         "parallel": (SharedLayerNorm, None, (), SharedLayerNorm)}


class Relu2MLP(nn.Module):
    """``relu(W_up y)^2``, to be projected by ``o`` (the down projection)."""

    def __init__(self, hidden: int, spec: dict, eps: float, dtype, device):
        super().__init__()
        self.up = nn.Parameter(torch.empty(spec["ff"], hidden, dtype=dtype, device=device))
        self.o = nn.Parameter(torch.empty(hidden, spec["ff"], dtype=dtype, device=device))

    def hidden(self, y, ctx=None, cache=None, rec=None):
        return linear_relu2(y, self.up)

    def tensors(self, p: str):
        yield p + "up", self.up
        yield p + "down", self.o


class ExpertsMLP(nn.Module):
    """Mixture of gated experts. Scores ``s`` are the softmax of the router's logits (32-bit) over all experts, or each
    expert's sigmoid (``router["score"]``); the ``top`` largest of ``s``, plus a learned correction unless
    ``router["correction"]`` is false, are chosen, with ``router["groups"]`` from the best groups only, and weighted by ``s``,
    renormalised with ``router["renorm"]``, times ``router["scale"]``. The weight multiplies an expert's result, or what goes
    into it (``spec["weight"]`` "input"). Every token also passes through the ``shared`` expert, when there is one; with its
    ``gate`` that result is multiplied by the sigmoid of one more row of the router. An expert is ``W_down act(W_gate y, W_up y)`` with the activation of ``ops/moe.py::GatedAct``. Gate and
    up rows alternate in ``gate_up`` so that the activation runs in the product's epilogue."""

    o = None

    def __init__(self, hidden: int, spec: dict, act, dtype, device):
        """``act``: the activation for an expert's ``limit``."""
        super().__init__()
        router = spec["router"]
        E, ff = router["experts"], spec["expert"]["ff"]
        mk = lambda *shape: nn.Parameter(torch.empty(*shape, dtype=dtype, device=device))
        self.top, self.score = router["top"], router.get("score", "softmax")
        self.renorm, self.scale = bool(router.get("renorm")), float(router.get("scale", 1.0))
        groups = router.get("groups") or {"count": 1, "keep": 1}
        self.groups = (groups["count"], groups["keep"])
        self.act, self.scale_input = act(spec["expert"].get("limit", INF)), spec.get("weight") == "input"
        self.gates = int(bool(spec.get("shared") and spec["shared"].get("gate")))
        self.router = mk(E + self.gates, hidden)
        self.correction = nn.Parameter(torch.zeros(E, dtype=dtype, device=device)) if router.get("correction", True) else None
        self.gate_up = mk(E, 2 * ff, hidden)
        self.down = mk(E, hidden, ff)
        self.shared = GatedMLP(hidden, spec["shared"]["ff"], act(spec["shared"].get("limit", INF)), dtype, device) \
            if spec.get("shared") else None

    def hidden(self, y, ctx=None, cache=None, rec=None):
        idx, w, *gate = route_tokens(y, self.router, self.top, self.renorm, self.correction, self.score, self.groups, self.scale,
                                     self.gates)
        e = gated_experts(y, idx, w, self.gate_up, self.down, self.act, self.scale_input)
        if self.shared is None:
            return e
        if not isinstance(e, ExpertRows):
            s = linear(self.shared.hidden(y), self.shared.o).float()
            return e + (s * torch.sigmoid(gate[0]) if gate else s)
        e.add_gate = gate[0] if gate else None
        e.add = linear_slices(self.shared.hidden(y), self.shared.o)
        return e

    def tensors(self, p: str):
        E = self.down.shape[0]
        for e in range(E):
            yield f"{p}e{e}.gate", self.gate_up[e, 0::2]
            yield f"{p}e{e}.up", self.gate_up[e, 1::2]
            yield f"{p}e{e}.down", self.down[e]
        yield p + "router", self.router[:E]
        if self.correction is not None:
            yield p + "correction", self.correction
        if self.shared is not None:
            yield from self.shared.tensors(p + "shared.")
        if self.gates:
            yield p + "shared.sg", self.router[E:]


class GatedMLP(nn.Module):
    """``act(W_gate y, W_up y)``, to be projected by ``o`` (the down projection); gate and up rows alternate in ``gate_up``."""

    def __init__(self, hidden: int, ff: int, act: GatedAct, dtype, device):
        super().__init__()
        self.act = act
        self.gate_up = nn.Parameter(torch.empty(2 * ff, hidden, dtype=dtype, device=device))
        self.o = nn.Parameter(torch.empty(hidden, ff, dtype=dtype, device=device))

    def hidden(self, y, ctx=None, cache=None, rec=None):
        return gated_linear(y, self.gate_up, self.act)

    def tensors(self, p: str):
        yield p + "gate", self.gate_up[0::2]
        yield p + "up", self.gate_up[1::2]
        yield p + "down", self.o


INF = float("inf")


def make_mlp(hidden: int, spec: dict, eps: float, dtype, device):
    if spec.get("act") == "swiglu":
        if spec["kind"] == "moe":
            return ExpertsMLP(hidden, spec, lambda limit: GatedAct(limit=float(limit)), dtype, device)
        return GatedMLP(hidden, spec["ff"], GatedAct(), dtype, device)
    if spec["kind"] == "moe":
        # x * sigmoid(1.702 x) approximates GELU (Hendrycks and Gimpel, "Gaussian Error Linear Units")
        return ExpertsMLP(hidden, spec, lambda limit: GatedAct(alpha=1.702, beta=1.0, limit=float(limit)), dtype, device)
    return {"polynorm": PolyNormMLP, "relu2": Relu2MLP}[spec.get("act", "polynorm")](hidden, spec, eps, dtype, device)


class PolyNormMLP(nn.Module):
    """``polynorm(W_up y)``, to be projected by ``o`` (the down projection). PolyNorm mixes the row-normalised first,
    second and third powers with the learned coefficients ``act``."""

    def __init__(self, hidden: int, spec: dict, eps: float, dtype, device):
        super().__init__()
        self.eps = eps
        self.up = nn.Parameter(torch.empty(spec["ff"], hidden, dtype=dtype, device=device))
        self.o = nn.Parameter(torch.empty(hidden, spec["ff"], dtype=dtype, device=device))
        self.act = nn.Parameter(torch.tensor([1 / 3, 1 / 3, 1 / 3, 0.0], device=device).to(dtype))

    def hidden(self, y, ctx=None, cache=None, rec=None):
        return dyt.polynorm(linear(y, self.up), self.act, self.eps)

    def tensors(self, p: str):
        yield p + "up", self.up
        yield p + "act", self.act
        yield p + "down", self.o


class ParallelBlock(nn.Module):
    """A layer whose mixer and feed-forward read the same norm, the mixer through ``h + conv(h)``. To the decoder it is one
    sublayer: ``hidden`` returns an :class:`ops.residual_sum.ParallelSum`."""

    o = None

    def __init__(self, cfg: ModelConfig, i: int, dtype, device):
        super().__init__()
        h, spec, eps = cfg.hidden_size, cfg.layer_specs[i], cfg.rms_norm_eps
        self.norm1 = NORMS[cfg.layer_norms][0](h, eps, dtype, device)
        self.attn = MIXERS[spec["type"]](h, spec["mixer"], eps, dtype, device)
        self.attn.index = i
        self.mlp = make_mlp(h, spec["mlp"], eps, dtype, device) if spec["mlp"] is not None else None
        self.conv = nn.Parameter(torch.empty(h, cfg.input_conv, dtype=dtype, device=device))
        self.mult = cfg.residual_mult

    def sublayers(self, cache, rec):
        return [(self, self.mult, self.norm1, cache, rec)]

    def tail(self, ctx, rec):
        """What the norm in front goes on to in a decode step."""
        return ConvTail(self.conv, rec["conv"], ctx.state_slots, ctx.pos) if ctx.decode else None

    def hidden(self, y, ctx, cache=None, rec=None):
        if ctx.decode:
            h, hc = y
        else:
            h = y
            hc = conv_prefill(h, self.conv, ctx.meta, ctx.pos, add=True, ring=rec["conv"] if rec is not None else None,
                              slots=ctx.state_slots)
        with ctx.beside(h):  # the two do not depend on each other
            ff = self._feed_forward(h, ctx)
        if self.attn.o is None:
            mixer = self.attn.results(hc, ctx, cache, rec)
        else:
            mixer = [(linear_slices(self.attn.hidden(hc, ctx, cache, rec), self.attn.o), None)]
        ctx.join(h)
        return rs.ParallelSum(mixer, ff)

    def _feed_forward(self, h, ctx):
        if self.mlp is None:
            return None
        ff = self.mlp.hidden(h, ctx)
        return ff if self.mlp.o is None else linear_slices(ff, self.mlp.o)

    def tensors(self, p: str):
        yield from self.norm1.tensors(p + "norm1")
        yield from self.attn.tensors(p + "mix.")
        if self.mlp is not None:
            yield from self.mlp.tensors(p + "mlp.")
        yield p + "canon1", self.conv


class LayeredBlock(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int, dtype, device):
        super().__init__()
        h, spec, eps = cfg.hidden_size, cfg.layer_specs[i], cfg.rms_norm_eps
        norm, wrap, self.wrap_names, _ = NORMS[cfg.layer_norms]
        self.norm1 = norm(h, eps, dtype, device)
        self.attn = MIXERS[spec["type"]](h, spec["mixer"], eps, dtype, device)
        self.attn.index = i
        self.wrap1 = wrap(h, eps, dtype, device)
        self.norm2 = self.mlp = self.wrap2 = None
        if spec["mlp"] is not None:
            self.norm2 = norm(h, eps, dtype, device)
            self.mlp = make_mlp(h, spec["mlp"], eps, dtype, device)
            self.wrap2 = wrap(h, eps, dtype, device)

    def sublayers(self, cache, rec):
        """``(sublayer, its wrap, its norm, its cache, its state)`` in order."""
        out = [(self.attn, self.wrap1, self.norm1, cache, rec)]
        return out if self.mlp is None else out + [(self.mlp, self.wrap2, self.norm2, None, None)]

    def tensors(self, p: str):
        yield from self.norm1.tensors(p + "norm1")
        yield from self.attn.tensors(p + "mix.")
        yield from self.wrap1.tensors(p + self.wrap_names[0])
        if self.mlp is not None:
            yield from self.norm2.tensors(p + "norm2")
            yield from self.mlp.tensors(p + "mlp.")
            yield from self.wrap2.tensors(p + self.wrap_names[1])


@dataclass
class StepContext:
    """What the mixers of one forward share. ``decode``: one token per sequence (pages and state slots); otherwise a
    packed batch described by ``meta``, with or without a cache to fill."""

    model: "LayeredModel"
    pos: torch.Tensor
    decode: bool = False
    meta: VarlenMeta | None = None
    slot_mapping: torch.Tensor | None = None
    block_table: torch.Tensor | None = None
    seq_lens: torch.Tensor | None = None
    max_seq_len: int | None = None
    state_slots: torch.Tensor | None = None
    # latents and rotated key parts of the batch, by layer, of the layers in ``shared`` (those that others read)
    shared: frozenset = frozenset()
    latents: dict = field(default_factory=dict)

    def beside(self, x: torch.Tensor):
        """What is launched inside may run beside what follows up to :meth:`join`: in a decode step, whose kernels leave much
        of the device idle, on a second stream (a branch of a captured graph). Memory that either side frees is used again
        only behind the join: the second stream waits for the first whenever it starts."""
        side = self.model.side_stream(x) if self.decode else None
        if side is None:
            return contextlib.nullcontext()
        side.wait_stream(torch.cuda.current_stream(x.device))
        return torch.cuda.stream(side)

    def join(self, x: torch.Tensor):
        side = self.model.side_stream(x) if self.decode else None
        if side is not None:
            torch.cuda.current_stream(x.device).wait_stream(side)

    def rotary(self, rot: dict):
        n = self.max_seq_len if self.decode else self.meta.max_seqlen
        return self.model.rotary(rot, n or 1, self.pos.device)


class LayeredModel(QwenModel):
    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", pctx=None):
        nn.Module.__init__(self)
        if pctx is not None and max(pctx.tp_size, pctx.pp_size, pctx.sp_size, pctx.ep_size, pctx.etp_size) > 1:
            raise NotImplementedError(f"{cfg.model_type} runs under data parallelism only")
        if cfg.lora_rank > 0 or cfg.fp8 or cfg.is_critic:
            raise NotImplementedError(f"{cfg.model_type} takes no LoRA adapters, fp8 projections or value head")
        self.cfg, self.pctx = cfg, pctx
        self.first_stage = self.last_stage = True
        self.vpp = 1
        self.chunk_ranges = self.chunk_slices = [(0, cfg.num_hidden_layers)]
        self.layer_ids = list(range(cfg.num_hidden_layers))
        self.layer_start, self.layer_end = 0, cfg.num_hidden_layers
        mk = lambda *shape: nn.Parameter(torch.empty(*shape, dtype=dtype, device=device))
        self.embed = mk(cfg.vocab_size, cfg.hidden_size)
        self.pos = mk(cfg.max_position_embeddings, cfg.hidden_size) if cfg.learned_positions else None
        self.layers = nn.ModuleList()
        block = ParallelBlock if cfg.layer_norms == "parallel" else LayeredBlock
        for i in self.layer_ids:  # a layer that runs with another's weights is the same module once more
            j = cfg.weights_layer(i)
            self.layers.append(block(cfg, i, dtype, device) if j == i else self.layers[j])
        # the head is linear: the logits' scale is the last norm's
        scaled = dict(scale=cfg.logit_scale) if cfg.logit_scale != 1.0 else {}
        self.norm = NORMS[cfg.layer_norms][3](cfg.hidden_size, cfg.rms_norm_eps, dtype, device, **scaled)
        self.lm_head = mk(cfg.vocab_size, cfg.hidden_size)
        self.score = None
        self.checkpoint_every = 0
        self._tables: dict[tuple, tuple[torch.Tensor, torch.Tensor]] = {}
        self._positions = 1
        self._side = None
        self._shared = frozenset(j for i in self.layer_ids if (j := cfg.cache_layer(i)) != i)

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: float = 0.02):
        gens: dict[str, torch.Generator] = {}
        for name, p in self.named_parameters():
            if p.dim() < 2:
                continue  # norms, scales, gates and coefficients keep their constructors' values
            dev = "cuda" if p.is_cuda else "cpu"
            if dev not in gens:
                gens[dev] = torch.Generator(device=p.device).manual_seed(seed)
            p.copy_(torch.randn(p.shape, generator=gens[dev], device=p.device) * std)
        return self

    # ------------------------------------------------------------------ positions
    def reserve_positions(self, n: int):
        """Positions up to ``n`` will be used: rotary tables are built that long from the start (a captured decode step
        keeps their addresses)."""
        self._positions = max(self._positions, int(n))

    def side_stream(self, x: torch.Tensor):
        """A second stream on ``x``'s device (None on the CPU)."""
        if not x.is_cuda:
            return None
        if self._side is None:
            self._side = torch.cuda.Stream(x.device, priority=-1)
        return self._side

    def rotary(self, rot: dict, n: int, device):
        dims, base, scaling = rot["dims"], rot["base"], rot.get("scaling")
        key = (dims, base, tuple(sorted(scaling.items())) if scaling else None)
        t = self._tables.get(key)
        if t is None or t[0].shape[0] < n or t[0].device != device:
            t = self._tables[key] = rotary_tables(max(n, self._positions), dims, base, device, scaling)
        return t

    def logits(self, hidden, out_dtype=torch.float32):
        return soft_cap_(super().logits(hidden, out_dtype), self.cfg.logit_softcap)

    # -------------------------------------------------------------------- forward
    def _run(self, input_ids, ctx: StepContext, kv_caches=None, state=None):
        """Embedding, every sublayer, final norm: ``[T, hidden]`` in the model's dtype."""
        ctx.shared = self._shared
        subs = []
        for i, layer in enumerate(self.layers):
            cache = kv_caches[self.cfg.cache_layer(i)] if kv_caches is not None else None
            if cache is not None and len(cache) == 1:
                cache = cache[0]
            subs += layer.sublayers(cache, state.rec[i] if state is not None else None)
        norms = [s[2] for s in subs] + [self.norm]
        # what a norm goes on to for the sublayer behind it
        tails = [(s[0].tail(ctx, s[4]),) if hasattr(s[0], "tail") else () for s in subs] + [()]
        extra = {}
        if self.pos is not None or self.cfg.embedding_scale != 1.0 or self.cfg.sinusoid_positions:
            extra = dict(scale=self.cfg.embedding_scale, pos=ctx.pos, pos_table=self.pos)
        y, res = norms[0].embed(input_ids, self.embed, *tails[0], **extra)
        for k, (sub, wrap, _, cache, rec) in enumerate(subs):
            y, res = norms[k + 1].join(sub.hidden(y, ctx, cache, rec), sub.o, wrap, res, *tails[k + 1])
        return y

    def forward(self, input_ids, position_ids, meta: VarlenMeta, attn_fn=None, **unsupported):
        if attn_fn is not None or any(v is not None for v in unsupported.values()):
            raise NotImplementedError(f"{self.cfg.model_type} takes packed token batches only")
        return self._run(input_ids, StepContext(self, position_ids.to(torch.int32), meta=meta))

    @torch.no_grad()
    def prefill(self, input_ids, position_ids, meta: VarlenMeta, kv_caches, slot_mapping, hybrid_state=None,
                state_slots=None):
        ctx = StepContext(self, position_ids.to(torch.int32), meta=meta, slot_mapping=slot_mapping,
                          state_slots=_int32(state_slots))
        return self._run(input_ids, ctx, kv_caches, hybrid_state)

    @torch.no_grad()
    def decode(self, input_ids, position_ids, kv_caches, block_table, seq_lens, slot_mapping, max_seq_len=None,
               hybrid_state=None, state_slots=None):
        ctx = StepContext(self, position_ids.to(torch.int32), decode=True, slot_mapping=slot_mapping,
                          block_table=block_table, seq_lens=seq_lens, max_seq_len=max_seq_len,
                          state_slots=_int32(state_slots))
        return self._run(input_ids, ctx, kv_caches, hybrid_state)

    # ----------------------------------------------------------------- checkpoint
    def to_hf_local(self, export: bool = False) -> Iterator[tuple[str, torch.Tensor]]:
        yield "embed", self.embed
        if self.pos is not None:
            yield "pos", self.pos
        for i, layer in enumerate(self.layers):
            if self.cfg.weights_layer(i) == i:
                yield from layer.tensors(f"l{i}.")
        yield from self.norm.tensors("final.norm")
        yield "head", self.lm_head


def _int32(t: Any):
    return None if t is None else t.to(torch.int32).contiguous()
