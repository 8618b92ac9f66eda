"""Decoders described as a list of layers (``ModelConfig.layer_specs``), each with its own mixer, its own sizes and an
optional feed-forward, on an fp32 residual stream. The Fofosun family is built this way:

    x = embed[token]
    x = x + ls1 * mixer(norm1(x));   x = x + ls2 * ff(norm2(x))     per layer; a layer may have no feed-forward
    logits = head norm(x)

Norms are Dynamic Tanh, ``tanh(alpha x) * w + b`` (Zhu, Chen, He, LeCun, Liu, "Transformers without Normalization"),
the feed-forward is ``W_down polynorm(W_up x)``. Every sublayer hands the activations in front of its output
projection to :func:`ops.dyt.linear_residual_dyt`, which projects, scales, adds to the residual and applies the NEXT
sublayer's norm in one kernel, so the model is a flat list of sublayers between the embedding and the head.

Mixers (``MIXERS``): HGRN2 (``models/hgrn2.py``), lightning attention with configured decays
(``models/lightning.py``), latent attention over a compressed cache (``models/mla.py``). A mixer has
``hidden(y, ctx, cache, rec)``, an output projection ``o`` and ``tensors(prefix)``; what it keeps per sequence is
declared by ``ModelConfig.cache_shapes`` / ``recurrent_shape``, allocated by the rollout engine and passed in.

The class shares loading, the head and the engine interface (``prefill`` / ``decode``) with ``QwenModel``. It is served
by the rollout engine and runs forward and backward for training on one process per replica (data parallelism).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Iterator

import torch
import torch.nn as nn

from ..ops import dyt
from ..ops.attention import VarlenMeta
from ..ops.gemm import linear
from ..ops.latent_attn import rotary_tables
from .config import ModelConfig
from .hgrn2 import HGRN2
from .lightning import ConstantDecayLightning
from .mla import LatentAttention
from .qwen import QwenModel

MIXERS = {"hgrn2": HGRN2, "lightning": ConstantDecayLightning, "latent_attention": LatentAttention}


class DynamicTanh(nn.Module):
    def __init__(self, n: int, dtype, device):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(n, dtype=dtype, device=device))
        self.bias = nn.Parameter(torch.zeros(n, dtype=dtype, device=device))
        self.alpha = nn.Parameter(torch.full((), 0.5, dtype=dtype, device=device))

    @property
    def args(self):
        return self.alpha, self.weight, self.bias

    def tensors(self, name: str):
        yield name, self.weight
        yield name + ".b", self.bias
        yield name + ".alpha", self.alpha


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


class LayeredBlock(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int, dtype, device):
        super().__init__()
        h, spec = cfg.hidden_size, cfg.layer_specs[i]
        scale = lambda: nn.Parameter(torch.ones(h, dtype=dtype, device=device))
        self.norm1 = DynamicTanh(h, dtype, device)
        self.attn = MIXERS[spec["type"]](h, spec["mixer"], cfg.rms_norm_eps, dtype, device)
        self.ls1 = scale()
        self.norm2 = self.mlp = self.ls2 = None
        if spec["mlp"] is not None:
            self.norm2 = DynamicTanh(h, dtype, device)
            self.mlp = PolyNormMLP(h, spec["mlp"], cfg.rms_norm_eps, dtype, device)
            self.ls2 = scale()

    def tensors(self, p: str):
        yield from self.norm1.tensors(p + "norm1")
        yield from self.attn.tensors(p + "mix.")
        yield p + "ls1", self.ls1
        if self.mlp is not None:
            yield from self.norm2.tensors(p + "norm2")
            yield from self.mlp.tensors(p + "mlp.")
            yield p + "ls2", self.ls2


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

    def rotary(self, dims: int, base: float):
        n = self.max_seq_len if self.decode else self.meta.max_seqlen
        return self.model.rotary(dims, base, n or 1, self.pos.device)


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
        self.layers = nn.ModuleList(LayeredBlock(cfg, i, dtype, device) for i in self.layer_ids)
        self.norm = DynamicTanh(cfg.hidden_size, dtype, device)
        self.lm_head = mk(cfg.vocab_size, cfg.hidden_size)
        self.score = None
        self.checkpoint_every = 0
        self._tables: dict[tuple[int, float], tuple[torch.Tensor, torch.Tensor]] = {}
        self._positions = 1

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

    def rotary(self, dims: int, base: float, n: int, device):
        t = self._tables.get((dims, base))
        if t is None or t[0].shape[0] < n or t[0].device != device:
            t = self._tables[(dims, base)] = rotary_tables(max(n, self._positions), dims, base, device)
        return t

    # -------------------------------------------------------------------- forward
    def _run(self, input_ids, ctx: StepContext, kv_caches=None, state=None):
        """Embedding, every sublayer, final norm: ``[T, hidden]`` in the model's dtype."""
        subs = []  # (sublayer, its scale, its norm, its cache, its state)
        for i, layer in enumerate(self.layers):
            cache = kv_caches[i][0] if kv_caches is not None and kv_caches[i] is not None else None
            subs.append((layer.attn, layer.ls1, layer.norm1, cache, state.rec[i] if state is not None else None))
            if layer.mlp is not None:
                subs.append((layer.mlp, layer.ls2, layer.norm2, None, None))
        norms = [s[2] for s in subs] + [self.norm]
        y, res = dyt.embed_dyt(input_ids, self.embed, norms[0].args)
        for k, (sub, scale, _, cache, rec) in enumerate(subs):
            y, res = dyt.linear_residual_dyt(sub.hidden(y, ctx, cache, rec), sub.o, scale, res, norms[k + 1].args)
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
        for i, layer in enumerate(self.layers):
            yield from layer.tensors(f"l{i}.")
        yield from self.norm.tensors("final.norm")
        yield "head", self.lm_head


def _int32(t: Any):
    return None if t is None else t.to(torch.int32).contiguous()
