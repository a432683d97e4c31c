"""Lipadra — a decoder whose norms follow the residual sums,

    x <- norm1(alpha x + mix(x)) ;  x <- norm2(alpha x + ffn(x))          (RMS norms, fp32 residual stream, x starts as the embedding)

with one of three mixers per layer — chunked soft-max attention with one added to the denominator (query / key norms ahead of a partial
rotation), retention (linear attention with a fixed decay per head) or the selective scan of Mamba — and a mixture of experts behind a grouped
soft-max router, some of whose choices are identity experts, plus a gated shared expert (or no feed-forward).  A layer may run on another
layer's tensors with a cache or state of its own.  The embedding table is also the output projection.  The layer list, every size and every
constant come from `LipadraConfig`.

The model is assembled from the framework's operators (operators/norm.py, attention.py, linear_attention.py, experts.py, gate.py, mlp.py); its
`forward(batch, cache)` is the step function the engine drives: a flattened ragged batch of prompt portions and decode tokens
(models/custom_cache.ForwardBatch) against the paged cache rows and per-sequence state rows of models/custom_cache.PagedStateCache, one
cache layer per layer.  Every residual sum is one norm launch, which also takes in the identity experts and the shared expert's gate."""
from __future__ import annotations

from typing import List, Optional

import torch
import torch.nn.functional as F
from torch import nn

from ..operators.attention import KPlusOneAttention
from ..operators.experts import KIdentityMoE
from ..operators.linear_attention import KRetention, KSelectiveScan
from ..operators.norm import KSumRMSNorm
from .configuration_lipadra import LipadraConfig
from .custom_cache import ForwardBatch, PagedStateCache

MIXERS = {"attention": KPlusOneAttention, "retention": KRetention, "mamba1": KSelectiveScan}


class LipadraDecoderLayer(nn.Module):
    def __init__(self, config: LipadraConfig, layer_idx: int, dtype, device):
        super().__init__()
        spec, norm = config.layers[layer_idx], lambda: KSumRMSNorm(config.width, config.norm_eps, dtype=dtype, device=device)
        self.layer_idx = layer_idx
        self.norm1, self.mix = norm(), MIXERS[spec.type](config.width, spec.mixer, config.norm_eps, dtype=dtype, device=device)
        f = spec.mlp
        if f is None:
            self.mlp = self.norm2 = None
        else:
            self.norm2 = norm()
            self.mlp = KIdentityMoE(config.width, f.ff, f.experts, f.identity, f.top, f.groups, f.keep_groups, f.out_scale, f.shared_ff, dtype=dtype, device=device)

    def load(self, loader, prefix: str):
        self.norm1.load(loader, prefix + "norm1")
        self.mix.load(loader, prefix + "mix.")
        if self.mlp is not None:
            self.norm2.load(loader, prefix + "norm2")
            self.mlp.load(loader, prefix + "mlp.")


class LipadraForCausalLM(nn.Module):
    config_class = LipadraConfig

    def __init__(self, config: LipadraConfig, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        self.config, self.dtype, self.device = config, dtype, torch.device(device)
        self.embed = nn.Parameter(torch.empty((config.vocab, config.width), dtype=dtype, device=device), requires_grad=False)
        self.owned = nn.ModuleDict({str(i): LipadraDecoderLayer(config, i, dtype, device) for i, l in enumerate(config.layers) if l.weights_of == i})
        self.final_norm = KSumRMSNorm(config.width, config.norm_eps, dtype=dtype, device=device)

    @property
    def layers(self) -> List[LipadraDecoderLayer]:
        """the layers in the order they run; one that uses another's tensors is that layer once more"""
        return [self.owned[str(l.weights_of)] for l in self.config.layers]

    def load(self, loader):
        self.embed.data.copy_(loader.load_tensor("embed", "cpu"))
        for i, layer in self.owned.items():
            layer.load(loader, f"l{i}.")
        self.final_norm.load(loader, "final.norm")

    def make_cache(self, max_tokens: int, max_slots: int = 8, page_size: int = 64) -> PagedStateCache:
        c = self.config
        return PagedStateCache(c.cache_row_widths(), c.state_widths(), max_tokens, max_slots, self.device, dtype=self.dtype, page_size=page_size, window=None, chunks=c.chunks())

    def decode_is_capturable(self, max_batch: int = 47) -> bool:
        """Whether a decode step of up to `max_batch` sequences makes no host read (then the engine may replay it as a CUDA graph)."""
        return all(layer.mlp is None or layer.mlp.experts.small_batches_stay_on_device(layer.mlp.router.top, self.dtype, max_batch) for layer in self.owned.values())

    @torch.no_grad()
    def forward(self, batch: ForwardBatch, cache: PagedStateCache, residual_trace: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Runs the batch's tokens from the cache and state earlier steps left; returns fp32 logits [len(batch.want), vocab]."""
        c, layers = self.config, self.layers
        want = batch.want
        x = h = self.embed.index_select(0, batch.tokens)
        for i, layer in enumerate(layers):
            last = i + 1 == len(layers)
            y = layer.mix(h, batch, cache, i)
            if last and want.shape[0] == 0 and residual_trace is None:      # a portion whose logits nobody asked for: caches and states are written
                break
            rows = want if last and residual_trace is None else None      # behind the last mixer only the rows asked for go on
            mlp = layer.mlp
            x, h, gate = layer.norm1(x, c.alpha, a=y, rows=rows, dot=mlp.shared_gate if mlp is not None else None)
            if mlp is not None:
                routed, ids, weights, shared = mlp(h)
                x, h, _ = layer.norm2(x, c.alpha, a=routed, b=shared, b_scale=gate, identity=(ids, weights, mlp.experts.experts) if mlp.identity else None)
            if residual_trace is not None:
                residual_trace.append(x)
        if want.shape[0] == 0:
            return torch.empty((0, c.vocab), dtype=torch.float32, device=h.device)
        _, h, _ = self.final_norm(x, rows=want if residual_trace is not None or not layers else None, keep_x=False)
        return F.linear(h, self.embed).float()
