"""Mixers that run side by side on the same input and whose outputs are added with fixed factors:

    out = sum_i scale_i W_o,i mix_i(W_in,i h)

    P   = [W_in,1 ; W_in,2 ; ...] h                one GEMM over everything that reads the mixer input
    o   = [scale_1 mix_1(P_1) | scale_2 mix_2(P_2) | ...]      each mixer writes its columns, its factor applied in fp32 before the one rounding
    out = [W_o,1 | W_o,2 | ...] o                   one GEMM: the sum over the mixers is part of its accumulation

A mixer takes part with `n_rows` / `n_out`, `load_in`, `load_rest` and `mix` (operators/attention.KBiasedSinkAttention,
operators/linear_attention.KStateSpace).  All of them use the same cache layer index: one may keep per-token rows, another a state row.
(The reference has no such layer.)"""
from __future__ import annotations

import torch
from torch import nn


class KSideBySide(nn.Module):
    ALIGN = 8      # columns of P and o at which a mixer starts: 16-byte aligned rows

    def __init__(self, width: int, mixers, scales, names, dtype=torch.bfloat16, device="cuda"):
        """mixers: built with `stacked=True`; names: their tensors' sub-prefixes"""
        super().__init__()
        up = lambda n: (n + self.ALIGN - 1) // self.ALIGN * self.ALIGN
        self.mixers, self.scales, self.names = nn.ModuleList(mixers), [float(s) for s in scales], list(names)
        self.in_off, self.out_off, n_in, n_out = [], [], 0, 0
        for m in self.mixers:
            self.in_off.append(n_in)
            self.out_off.append(n_out)
            n_in, n_out = n_in + up(m.n_rows), n_out + up(m.n_out)
        self.n_out = n_out
        self.gapless = all(m.n_out % self.ALIGN == 0 for m in self.mixers)      # else columns between the mixers' outputs stay zero
        P = lambda *shape: nn.Parameter(torch.zeros(shape, dtype=dtype, device=device), requires_grad=False)
        self.w_in, self.o = P(n_in, width), P(width, n_out)

    def load(self, loader, prefix: str):
        for m, name, i, j in zip(self.mixers, self.names, self.in_off, self.out_off):
            self.w_in.data[i:i + m.n_rows].copy_(m.load_in(loader, prefix + name))
            m.load_rest(loader, prefix + name)
            self.o.data[:, j:j + m.n_out].copy_(loader.load_tensor(prefix + name + "o", "cpu"))

    def forward(self, h: torch.Tensor, batch, cache, cache_idx: int) -> torch.Tensor:
        proj = nn.functional.linear(h, self.w_in)
        o = (torch.empty if self.gapless else torch.zeros)((h.shape[0], self.n_out), dtype=h.dtype, device=h.device)
        for m, scale, i, j in zip(self.mixers, self.scales, self.in_off, self.out_off):
            m.mix(proj, i, batch, cache, cache_idx, o[:, j:j + m.n_out], scale)
        return nn.functional.linear(o, self.o)
