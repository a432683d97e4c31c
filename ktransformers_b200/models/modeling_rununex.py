"""Rununex — a pre-norm decoder (layer norm without bias) whose residual sums are scaled by one constant m,

    x <- x + m mix(norm1 x) ;  x <- x + m ffn(norm2 x)          (fp32 residual stream, x starts as the scaled embedding)

with one of two mixers per layer — chunked soft-max attention (unit-rms queries and keys, a logarithmic distance bias, a sink, an element-wise
output gate) side by side with a Mamba-2 state space; or chunked differential attention behind short convolutions and a partial rotation —
and a mixture of experts whose sigmoid weights multiply the experts' inputs, plus a shared expert (or no feed-forward).  Logits are scaled by
a constant.  The layer list, every size and every constant come from `RununexConfig`.

The model is assembled from the framework's operators (operators/norm.py, attention.py, linear_attention.py, side_by_side.py, experts.py,
gate.py, mlp.py); its `forward(batch, cache)` is the step function the engine drives: a flattened ragged batch of prompt portions and decode
tokens (models/custom_cache.ForwardBatch) against the paged cache rows and per-sequence state rows of models/custom_cache.PagedStateCache.
The embedding lookup and every residual sum are folded into the norm launch that follows."""
from __future__ import annotations

from typing import List, Optional

import torch
import torch.nn.functional as F
from torch import nn

from ..operators.attention import KBiasedSinkAttention, KDifferentialAttention
from ..operators.experts import KSharedSigmoidMoE
from ..operators.linear_attention import KStateSpace
from ..operators.norm import KLayerNorm
from ..operators.side_by_side import KSideBySide
from .configuration_rununex import RununexConfig
from .custom_cache import ForwardBatch, PagedStateCache


def _parallel(width, spec, eps, dtype, device):
    kw = dict(dtype=dtype, device=device, stacked=True)
    return KSideBySide(width, [KBiasedSinkAttention(width, spec.left, eps, **kw), KStateSpace(width, spec.right, eps, **kw)], [spec.left_scale, spec.right_scale], ["left.", "right."],
                       dtype=dtype, device=device)


def _differential(width, spec, eps, dtype, device):
    return KDifferentialAttention(width, spec, eps, dtype=dtype, device=device)


MIXERS = {"parallel": _parallel, "attention": _differential}


class RununexDecoderLayer(nn.Module):
    def __init__(self, config: RununexConfig, layer_idx: int, dtype, device):
        super().__init__()
        spec, norm = config.layers[layer_idx], lambda: KLayerNorm(config.width, config.norm_eps, dtype=dtype, device=device)
        self.layer_idx = layer_idx
        self.norm1, self.mix = norm(), MIXERS[spec.type](config.width, spec.mixer, config.norm_eps, dtype, device)
        f = spec.mlp
        if f is None:
            self.mlp = self.norm2 = None
        else:
            self.norm2, self.mlp = norm(), KSharedSigmoidMoE(config.width, f.ff, f.experts, f.top, f.shared_ff, dtype=dtype, device=device)

    def load(self, loader, prefix: str):
        self.norm1.load(loader, prefix + "norm1")
        self.mix.load(loader, prefix + "mix.")
        if self.mlp is not None:
            self.norm2.load(loader, prefix + "norm2")
            self.mlp.load(loader, prefix + "mlp.")


class RununexForCausalLM(nn.Module):
    config_class = RununexConfig

    def __init__(self, config: RununexConfig, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        self.config, self.dtype, self.device = config, dtype, torch.device(device)
        P = lambda *shape: nn.Parameter(torch.empty(shape, dtype=dtype, device=device), requires_grad=False)
        self.embed = P(config.vocab, config.width)
        self.layers = nn.ModuleList([RununexDecoderLayer(config, i, dtype, device) for i in range(len(config.layers))])
        self.final_norm = KLayerNorm(config.width, config.norm_eps, dtype=dtype, device=device)
        self.head = P(config.vocab, config.width)

    def load(self, loader):
        self.embed.data.copy_(loader.load_tensor("embed", "cpu"))
        for i, layer in enumerate(self.layers):
            layer.load(loader, f"l{i}.")
        self.final_norm.load(loader, "final.norm")
        self.head.data.copy_(loader.load_tensor("head", "cpu"))

    def make_cache(self, max_tokens: int, max_slots: int = 8, page_size: int = 64) -> PagedStateCache:
        c = self.config
        return PagedStateCache(c.cache_row_widths(), c.state_widths(), max_tokens, max_slots, self.device, dtype=self.dtype, page_size=page_size, window=None, chunks=c.chunks())

    def decode_is_capturable(self, max_batch: int = 47) -> bool:
        """Whether a decode step of up to `max_batch` sequences makes no host read (then the engine may replay it as a CUDA graph)."""
        return all(layer.mlp is None or layer.mlp.experts.small_batches_stay_on_device(layer.mlp.router.top, self.dtype, max_batch) for layer in self.layers)

    @torch.no_grad()
    def forward(self, batch: ForwardBatch, cache: PagedStateCache, residual_trace: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Runs the batch's tokens from the cache and state earlier steps left; returns fp32 logits [len(batch.want), vocab]."""
        c, m = self.config, self.config.residual_mult
        # (x, a, b): the residual before the pending sublayer outputs a and b (None: nothing pending), which the next norm launch adds
        x = a = b = None
        for i, layer in enumerate(self.layers):
            if i == 0:
                x, h = layer.norm1(None, self.embed, mult=c.embedding_scale, rows=batch.tokens)
            else:
                x, h = layer.norm1(x, a, b, m)
            a, b = layer.mix(h, batch, cache, i), None
            if layer.mlp is not None:
                x, h = layer.norm2(x, a, b, m)
                a, b = layer.mlp(h)
            if residual_trace is not None:
                residual_trace.append(self.final_norm(x, a, b, m, want_h=False)[0])
        if batch.want.shape[0] == 0:      # a prompt portion whose logits nobody asked for: its cache rows and states are written, that is all
            return torch.empty((0, c.vocab), dtype=torch.float32, device=self.head.device)
        # the last sum and the final norm in one launch, for the rows asked for only; the logits' constant rides on the normed row
        _, h = self.final_norm(x, a, b, m, rows=batch.want, keep_x=False, h_scale=c.logit_scale)
        return F.linear(h, self.head).float()
