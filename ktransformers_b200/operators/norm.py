"""KGroupRMSNormShift — grouped RMS norm fused with the residual sum before it and the token shift after it.

One launch of `ktb200_group_rmsnorm_shift` (csrc/seq_ops.cu) per call:

    x_out = x_in + mult * (a + b) + row                   (a, b: the previous layer's branch outputs, when passed in; row: one
                                                           vector added to every token, e.g. the step vector of a looped pass)
    h     = x_out / sqrt(mean_g(x_out^2) + eps) * weight   per group g of `groups` equal consecutive parts, fp32
    hs_t  = h_t + (h_{t-1} - h_t) * shift                  (layers that mix in the previous token's normed row)

The residual stream stays fp32; h and hs are rounded once to the compute dtype.  h_{t-1} of the first token of a portion
comes from the cache manager's state rows (models/custom_cache.PagedStateCache), which hold it in fp32 — the same value the
kernel recomputes when the previous token is part of the same launch, so results do not depend on where a prompt was cut.
(The reference's norms are plain torch modules, archive/ktransformers/models/modeling_deepseek_v3.py:65-80.)"""
from __future__ import annotations

import ctypes as C
from typing import Optional, Tuple

import torch
from torch import nn

from .. import native

GGML_OF = {torch.bfloat16: native.GGML_BF16, torch.float32: native.GGML_F32}


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


class KGroupRMSNormShift(nn.Module):
    def __init__(self, width: int, groups: int, eps: float, shift: bool, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        if width % groups:
            raise ValueError("the width must divide into the norm groups")
        self.width, self.groups, self.eps = width, groups, eps
        self.weight = nn.Parameter(torch.ones(width, dtype=dtype, device=device), requires_grad=False)
        self.shift = nn.Parameter(torch.zeros(width, dtype=dtype, device=device), requires_grad=False) if shift else None

    def load(self, loader, norm_key: str, shift_key: Optional[str] = None):
        self.weight.data.copy_(loader.load_tensor(norm_key, "cpu"))
        if self.shift is not None:
            self.shift.data.copy_(loader.load_tensor(shift_key, "cpu"))

    def forward(self, x: torch.Tensor, delta_a=None, delta_b=None, mult: float = 1.0, batch=None, state: Optional[torch.Tensor] = None, want_h: bool = True,
                row_add: Optional[torch.Tensor] = None):
        """x [T, width] fp32; delta_a / delta_b [T, width] fp32 or the compute dtype; row_add [width] fp32.  Returns (residual after
        the sum, h or None, hs or None)."""
        T = x.shape[0]
        dt = self.weight.dtype
        add = delta_a is not None or delta_b is not None or row_add is not None
        assert row_add is None or (row_add.dtype == torch.float32 and row_add.is_contiguous() and row_add.shape == (self.width,))
        x_out = torch.empty_like(x) if add else x
        h = torch.empty((T, self.width), dtype=dt, device=x.device) if want_h else None
        hs = torch.empty((T, self.width), dtype=dt, device=x.device) if self.shift is not None else None
        for d in (delta_a, delta_b):
            assert d is None or (d.is_contiguous() and d.shape == x.shape)
        native.check_seq(native.seq_lib().ktb200_group_rmsnorm_shift(
            x.data_ptr(), _ptr(delta_a), GGML_OF[delta_a.dtype] if delta_a is not None else 0, _ptr(delta_b),
            GGML_OF[delta_b.dtype] if delta_b is not None else 0, float(mult), _ptr(row_add), x_out.data_ptr() if add else None, self.weight.data_ptr(), self.groups,
            float(self.eps), _ptr(self.shift), _ptr(batch.prev_idx) if hs is not None else None, _ptr(batch.rd_row) if hs is not None else None,
            _ptr(batch.wr_row) if hs is not None else None, _ptr(state) if hs is not None else None, _ptr(h), _ptr(hs), T, self.width, GGML_OF[dt],
            torch.cuda.current_stream(x.device).cuda_stream))
        return x_out, h, hs


class KGroupRMSNorm(nn.Module):
    """One grouped RMS norm weight of a layer that norms BOTH sides of every sublayer, `x <- x + post(sublayer(pre(x)))`.
    The norms never run alone: `KGroupRMSNorm.fused` is one `ktb200_group_rmsnorm_sandwich` launch (csrc/seq_mixers.cu) for

        x_out = x_in + gnorm(y) * post.weight + row       the sublayer's output y normed and added to the fp32 residual
        h     = gnorm(x_out) * pre.weight                  the NEXT sublayer's input, rounded once to the compute dtype

    with every term optional (no x_in / post: the stream restarts from y; no pre: nothing follows, or with `cast_h` the next
    sublayer reads the residual itself and h is x_out rounded to the compute dtype).  `weight_offset = 1`: the weight is
    zero-centred and the row is scaled by 1 + weight (added in fp32 in the kernel)."""

    def __init__(self, width: int, groups: int, eps: float, dtype=torch.bfloat16, device="cuda", weight_offset: float = 0.0):
        super().__init__()
        if width % groups:
            raise ValueError("the width must divide into the norm groups")
        self.width, self.groups, self.eps, self.weight_offset = width, groups, eps, float(weight_offset)
        self.weight = nn.Parameter(torch.full((width,), 1.0 - float(weight_offset), dtype=dtype, device=device), requires_grad=False)

    def load(self, loader, key: str):
        self.weight.data.copy_(loader.load_tensor(key, "cpu"))

    @staticmethod
    def fused(x_in: Optional[torch.Tensor], y: torch.Tensor, post: Optional["KGroupRMSNorm"], pre: Optional["KGroupRMSNorm"], row_add: Optional[torch.Tensor] = None,
              keep_x: bool = True, cast_h: bool = False):
        """x_in [T, width] fp32 or None, y [T, width] fp32 or the compute dtype.  Returns (x_out fp32 or None, h or None); with
        `cast_h` and no `pre`, h is x_out in the compute dtype (x_out itself when that is fp32)."""
        ref = pre if pre is not None else post
        T, D = y.shape
        assert y.is_contiguous() and (x_in is None or x_in.is_contiguous()) and D == ref.width
        dt = ref.weight.dtype
        x_out = torch.empty((T, D), dtype=torch.float32, device=y.device) if keep_x or pre is None else None
        plain_h = cast_h and pre is None and dt != torch.float32
        h = torch.empty((T, D), dtype=dt, device=y.device) if pre is not None or plain_h else None
        native.check_seq(native.seq_lib().ktb200_group_rmsnorm_sandwich(
            _ptr(x_in), y.data_ptr(), GGML_OF[y.dtype], post.weight.data_ptr() if post is not None else None, _ptr(row_add), _ptr(x_out),
            pre.weight.data_ptr() if pre is not None else None, _ptr(h), ref.groups, float(ref.eps), float(ref.weight_offset), T, D, GGML_OF[dt],
            torch.cuda.current_stream(y.device).cuda_stream))
        if cast_h and pre is None and not plain_h:
            h = x_out
        return x_out, h


class KLayerNorm(nn.Module):
    """Layer norm with a weight and no bias, fused with the residual sum before it: one `ktb200_residual_layernorm` launch (csrc/seq_ops.cu) for

        x = x_in + mult * (a + b)                            (every term optional; an embedding lookup is a = table, rows = token ids)
        h = (x - mean) / sqrt(mean((x - mean)^2) + eps) * weight * h_scale

    The residual stream stays fp32; h is rounded once to the compute dtype.  `rows` [T] int64 picks the rows of x_in, a and b."""

    def __init__(self, width: int, eps: float, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        self.width, self.eps = width, float(eps)
        self.weight = nn.Parameter(torch.ones(width, dtype=dtype, device=device), requires_grad=False)

    def load(self, loader, key: str):
        self.weight.data.copy_(loader.load_tensor(key, "cpu"))

    def forward(self, x: Optional[torch.Tensor], a: Optional[torch.Tensor] = None, b: Optional[torch.Tensor] = None, mult: float = 1.0, rows: Optional[torch.Tensor] = None,
                keep_x: bool = True, want_h: bool = True, h_scale: float = 1.0):
        """Returns (x after the sum in fp32 or None, h or None)."""
        ref = x if x is not None else a
        T, dt, dev = (ref.shape[0] if rows is None else rows.shape[0]), self.weight.dtype, ref.device
        for d in (x, a, b):
            assert d is None or (d.is_contiguous() and d.shape[-1] == self.width)
        assert rows is None or (rows.dtype == torch.int64 and rows.is_contiguous())
        plain = rows is None and a is None and b is None and x is not None      # nothing to add: the stream stays where it is
        x_out = torch.empty((T, self.width), dtype=torch.float32, device=dev) if keep_x and not plain else None
        h = torch.empty((T, self.width), dtype=dt, device=dev) if want_h else None
        native.check_seq(native.seq_lib().ktb200_residual_layernorm(
            _ptr(x), _ptr(a), GGML_OF[a.dtype] if a is not None else 0, _ptr(b), GGML_OF[b.dtype] if b is not None else 0, float(mult), _ptr(rows), _ptr(x_out), self.weight.data_ptr(),
            self.eps, float(h_scale), _ptr(h), T, self.width, GGML_OF[dt], torch.cuda.current_stream(dev).cuda_stream))
        return (x if plain else x_out), h


class KSumRMSNorm(nn.Module):
    """An RMS norm that follows the residual sum, so that the normed row is the new stream: one `ktb200_sum_rmsnorm` launch (csrc/seq_ops.cu) for

        s = (x_scale + w_id) x + a + b_scale b ;  y = s / sqrt(mean(s^2) + eps) * weight           (every term but x optional)

    with w_id the summed weights of the token's choices that are identity experts (whose output is x itself) and b_scale one number per token.
    y is kept in fp32 (the stream) and rounded once to the compute dtype (what the next sublayer reads).  `rows` [T] int64 picks the rows of every
    input; `dot` [width]: also sigmoid(y . dot) per token, from the fp32 row."""

    def __init__(self, width: int, eps: float, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        self.width, self.eps = width, float(eps)
        self.weight = nn.Parameter(torch.ones(width, dtype=dtype, device=device), requires_grad=False)

    def load(self, loader, key: str):
        self.weight.data.copy_(loader.load_tensor(key, "cpu"))

    def forward(self, x: torch.Tensor, x_scale: float = 1.0, a: Optional[torch.Tensor] = None, b: Optional[torch.Tensor] = None, b_scale: Optional[torch.Tensor] = None,
                identity: Optional[Tuple[torch.Tensor, torch.Tensor, int]] = None, rows: Optional[torch.Tensor] = None, dot: Optional[torch.Tensor] = None, keep_x: bool = True):
        """x, a, b [T, width], each fp32 or the compute dtype; b_scale [T] fp32; identity: (ids [T, top] int64, weights [T, top] fp32, first
        identity expert).  Returns (y in fp32 or None, y in the compute dtype, the sigmoids [T] fp32 or None)."""
        T, dt, dev = (x.shape[0] if rows is None else rows.shape[0]), self.weight.dtype, x.device
        for d in (x, a, b):
            assert d is None or (d.is_contiguous() and d.shape[-1] == self.width)
        assert rows is None or (rows.dtype == torch.int64 and rows.is_contiguous())
        ids, id_w, first = identity if identity is not None else (None, None, 0)
        y = torch.empty((T, self.width), dtype=torch.float32, device=dev) if keep_x or dt == torch.float32 else None
        h = torch.empty((T, self.width), dtype=dt, device=dev) if dt != torch.float32 else None
        gate = torch.empty(T, dtype=torch.float32, device=dev) if dot is not None else None
        p = native.SumRmsnormParams(x=x.data_ptr(), x_type=GGML_OF[x.dtype], x_scale=float(x_scale), a=_ptr(a), a_type=GGML_OF[a.dtype] if a is not None else 0, b=_ptr(b),
                                    b_type=GGML_OF[b.dtype] if b is not None else 0, b_scale=_ptr(b_scale), ids=_ptr(ids), id_weights=_ptr(id_w), top=ids.shape[1] if ids is not None else 0,
                                    first_identity=first, rows=_ptr(rows), weight=self.weight.data_ptr(), eps=self.eps, x_out=_ptr(y), h_out=_ptr(h), dot_weight=_ptr(dot), dot_out=_ptr(gate))
        native.check_seq(native.seq_lib().ktb200_sum_rmsnorm(C.byref(p), T, self.width, GGML_OF[dt], torch.cuda.current_stream(dev).cuda_stream))
        return y, h if h is not None else y, gate
