"""Recurrent mixers with a matrix state per head.  KGatedDeltaRule (below) — the gated delta rule behind short convolutions.
KStateSpace (below) — Mamba-2 (state-space duality): one decay per token and head.
KRetention (below) — a fixed decay per head.  KSelectiveScan (below) — Mamba: a state per channel, one decay per token, channel and state.
KGatedLinearAttention — linear attention with a decay per key channel and a recurrent matrix state per head:

    q = W_q h / sqrt(dim) ,  k = W_k h ,  v = W_v h ,  a = sigmoid(W_a2 (W_a1 h) + b) ** (1 / tau)        (a per head and key channel)
    S_t = diag(a_t) S_{t-1} + k_t v_t^T ,  o_t = S_t^T q_t                                                  (S: dim x vdim per head, fp32)
    out = W_o (rmsnorm_vdim(o) * w * silu(W_g h))

    P     = [W_q ; W_k ; W_v ; W_g ; W_a1] h        one GEMM over the matrices that read the mixer input
    z     = W_a2 P[a1]                              GEMM (the low-rank decay logits; the bias joins in fp32 in the kernel)
    o     = scan over each sequence portion         ktb200_gla_scan: state rows of the cache manager in, state rows out
    out   = W_o (norm, gate)                        ktb200_gla_out + GEMM

The state starts at zero, is carried per sequence in the cache manager's double-buffered fp32 state rows
(models/custom_cache.PagedStateCache) and is the only thing a step keeps: there are no per-token cache rows.  Decay logits,
their log-sigmoid and exponential, the state and the per-head norm are fp32.  Tokens of a portion run in order, so a position's
result does not depend on where the prompt was cut.  `cache_idx` picks the cache layer (state rows), so one set of weights
can run several times per step with separate states.  (The reference has no recurrent mixer; its caches are per-token:
archive/ktransformers/models/custom_cache.py:26-200.)"""
from __future__ import annotations

import ctypes as C
import math

import torch
from torch import nn

from .. import native


class KGatedLinearAttention(nn.Module):
    def __init__(self, width: int, spec, eps: float, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        P = lambda *shape: nn.Parameter(torch.zeros(shape, dtype=dtype, device=device), requires_grad=False)
        s = self.spec = spec
        self.width, self.eps = width, eps
        self.n_qk, self.n_v = s.heads * s.dim, s.heads * s.vdim
        self.rank = None           # rows of W_a1: known when the weights arrive
        self.w_in = None
        self.a2, self.a2_b = None, P(self.n_qk)
        self.norm = P(s.vdim)
        self.o = P(width, self.n_v)
        self._dtype, self._device = dtype, device

    def set_rank(self, rank: int):
        self.rank = rank
        n = 2 * self.n_qk + 2 * self.n_v + rank
        self.n_in = (n + 7) // 8 * 8
        self.a1_off = 2 * self.n_qk + 2 * self.n_v
        self.w_in = nn.Parameter(torch.zeros((self.n_in, self.width), dtype=self._dtype, device=self._device), requires_grad=False)
        self.a2 = nn.Parameter(torch.zeros((self.n_qk, rank), dtype=self._dtype, device=self._device), requires_grad=False)

    def load(self, loader, prefix: str):
        t = lambda n: loader.load_tensor(prefix + n, "cpu")
        a1 = t("a1")
        self.set_rank(a1.shape[0])
        self.w_in.data[:self.a1_off + self.rank].copy_(torch.cat([t("q"), t("k"), t("v"), t("g"), a1], 0))
        self.a2.data.copy_(t("a2"))
        self.a2_b.data.copy_(t("a2.b"))
        self.norm.data.copy_(t("norm"))
        self.o.data.copy_(t("o"))

    def forward(self, h: torch.Tensor, batch, cache, cache_idx: int) -> torch.Tensor:
        s, T, dev, dt = self.spec, h.shape[0], h.device, h.dtype
        lib, code, st = native.seq_lib(), native.GGML_BF16 if dt == torch.bfloat16 else native.GGML_F32, torch.cuda.current_stream(h.device).cuda_stream
        proj = torch.nn.functional.linear(h, self.w_in)
        z = torch.nn.functional.linear(proj[:, self.a1_off:self.a1_off + self.rank], self.a2)
        o = torch.empty((T, self.n_v), dtype=torch.float32, device=dev)
        native.check_seq(lib.ktb200_gla_scan(proj.data_ptr(), self.n_in, 0, self.n_qk, 2 * self.n_qk, z.data_ptr(), self.n_qk, self.a2_b.data_ptr(), float(s.tau), s.heads,
                                             s.dim, s.vdim, batch.seqs.data_ptr(), batch.seqs.stride(0), batch.n_seqs, T, cache.state[cache_idx].data_ptr(), o.data_ptr(),
                                             code, st))
        og = torch.empty((T, self.n_v), dtype=dt, device=dev)
        native.check_seq(lib.ktb200_gla_out(o.data_ptr(), self.norm.data_ptr(), float(self.eps), proj[:, 2 * self.n_qk + self.n_v:].data_ptr(), self.n_in, og.data_ptr(), T,
                                            s.heads, s.vdim, code, st))
        return torch.nn.functional.linear(og, self.o)


class KGatedDeltaRule(nn.Module):
    """The gated delta rule behind short causal convolutions — a recurrent mixer with a matrix state per value head:

        q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))     conv: a causal filter of `conv` taps along time on every channel, without bias
        q, k    = x * rsqrt(|x|^2 + unit_eps) per head ;  q also / sqrt(dim)              (kv_heads query/key heads, shared by
                                                                                            heads / kv_heads value heads each)
        eta     = sigmoid(W_b h) ;  a = exp(-rate * softplus(W_a h + dt_bias)), rate = exp(A_log)      one of each per value head
        M <- a M ;  r = eta (v - M^T k) ;  M <- M + k r^T ;  y = M^T q                     (M: dim x vdim per head, fp32)
        out     = W_o (rmsnorm_vdim(o) * w * silu(W_g h))

        P     = [W_q ; W_k ; W_v ; W_g ; W_b ; W_a] h      one GEMM over the matrices that read the mixer input
        prep                                               ktb200_delta_prep: convolution, activations, unit vectors, eta, a
        o     = scan over each sequence portion            ktb200_delta_scan: state rows of the cache manager in, state rows out
        out   = W_o (norm, gate)                           ktb200_gla_out + GEMM

    A sequence's state — the matrices and the last conv - 1 inputs of every convolved channel — lives in the cache manager's
    double-buffered fp32 state rows (models/custom_cache.PagedStateCache); there are no per-token cache rows.  Tokens of a
    portion run in order with the same arithmetic wherever the portion starts, so a position's result does not depend on
    where the prompt was cut.  `cache_idx` picks the cache layer.  (The reference has no recurrent mixer.)"""

    def __init__(self, width: int, spec, eps: float, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        P = lambda *shape, dt=dtype: nn.Parameter(torch.zeros(shape, dtype=dt, device=device), requires_grad=False)
        s = self.spec = spec
        if s.heads % s.kv_heads:
            raise ValueError("value heads must divide into the query/key heads")
        self.width, self.eps = width, eps
        self.n_qk, self.n_v = s.kv_heads * s.dim, s.heads * s.vdim
        self.g_off = 2 * self.n_qk + self.n_v
        self.b_off = self.g_off + self.n_v
        self.a_off = self.b_off + s.heads
        self.n_in = (self.a_off + s.heads + 7) // 8 * 8
        self.w_in = P(self.n_in, width)
        self.conv_w = P(s.channels, s.conv)
        self.a_log, self.dt_bias = P(s.heads, dt=torch.float32), P(s.heads, dt=torch.float32)
        self.norm = P(s.vdim)
        self.o = P(width, self.n_v)

    def load(self, loader, prefix: str):
        t = lambda n: loader.load_tensor(prefix + n, "cpu")
        self.w_in.data[:self.a_off + self.spec.heads].copy_(torch.cat([t("q"), t("k"), t("v"), t("g"), t("b"), t("a")], 0))
        self.conv_w.data.copy_(torch.cat([t("q.conv"), t("k.conv"), t("v.conv")], 0))
        self.a_log.data.copy_(t("A_log").float())
        self.dt_bias.data.copy_(t("dt_bias").float())
        self.norm.data.copy_(t("norm"))
        self.o.data.copy_(t("o"))

    def forward(self, h: torch.Tensor, batch, cache, cache_idx: int) -> torch.Tensor:
        s, T, dev, dt = self.spec, h.shape[0], h.device, h.dtype
        lib, code, st = native.seq_lib(), native.GGML_BF16 if dt == torch.bfloat16 else native.GGML_F32, torch.cuda.current_stream(h.device).cuda_stream
        state = cache.state[cache_idx]
        proj = torch.nn.functional.linear(h, self.w_in)
        f32 = lambda *shape: torch.empty(shape, dtype=torch.float32, device=dev)
        qn, kn, vv, beta, decay = f32(T, self.n_qk), f32(T, self.n_qk), f32(T, self.n_v), f32(T, s.heads), f32(T, s.heads)
        native.check_seq(lib.ktb200_delta_prep(proj.data_ptr(), self.n_in, 0, self.b_off, self.a_off, self.conv_w.data_ptr(), s.conv, self.a_log.data_ptr(),
                                               self.dt_bias.data_ptr(), s.heads, s.kv_heads, s.dim, s.vdim, float(s.unit_eps), batch.seq_of.data_ptr(), batch.seqs.data_ptr(),
                                               batch.seqs.stride(0), state.data_ptr(), state.stride(0), qn.data_ptr(), kn.data_ptr(), vv.data_ptr(), beta.data_ptr(),
                                               decay.data_ptr(), T, code, st))
        o = f32(T, self.n_v)
        native.check_seq(lib.ktb200_delta_scan(qn.data_ptr(), kn.data_ptr(), vv.data_ptr(), beta.data_ptr(), decay.data_ptr(), s.heads, s.kv_heads, s.dim, s.vdim,
                                               batch.seqs.data_ptr(), batch.seqs.stride(0), batch.n_seqs, state.data_ptr(), state.stride(0), o.data_ptr(), st))
        og = torch.empty((T, self.n_v), dtype=dt, device=dev)
        native.check_seq(lib.ktb200_gla_out(o.data_ptr(), self.norm.data_ptr(), float(self.eps), proj[:, self.g_off:].data_ptr(), self.n_in, og.data_ptr(), T,
                                            s.heads, s.vdim, code, st))
        return torch.nn.functional.linear(og, self.o)


class KStateSpace(nn.Module):
    """Mamba-2 (state-space duality), a recurrent mixer with a state_size x vdim matrix per head whose decay is one number per token and head:

        [z | x | B | C | dt] = W_in h                          x: heads x vdim; B, C: groups x state_size, shared by heads / groups heads each
        x, B, C = silu(filter(x, B, C) + b)                     a causal filter of `conv` taps along time on every channel
        dt      = softplus(dt + dt_bias) ;  S <- exp(-exp(A_log) dt) S + dt B x^T ;  y = S^T C + D x      per head, S in fp32
        out     = W_o (norm(y silu(z)) w)                       norm: `norm_groups` equal parts, each to unit rms

        P     = W_in h                                          one GEMM
        y     = prompt portions: ktb200_ssd_conv + ktb200_ssd_scan; decode steps (one token per sequence): ktb200_ssd_step
        o     = ktb200_gated_group_norm                         (gated first, then normed)
        out   = W_o o                                           GEMM

    A sequence's state — the matrices and the last conv - 1 inputs of every filtered channel — lives in the cache manager's double-buffered
    fp32 state rows (models/custom_cache.PagedStateCache).  Alone (`forward`), or side by side with another mixer of the same input
    (operators/side_by_side.py) through `load_in` and `mix`, as KBiasedSinkAttention.  Sizes are constructor parameters
    (models/configuration_rununex.StateSpaceSpec).

    Two forms of the scan (csrc/ssd.cu): in bf16 with a state size that is a multiple of 16, chunks of 64 tokens on the tensor cores, operands
    that carry fp32 factors as two bf16 terms, the state in fp32 accumulators; otherwise, in fp32 and for batches of mostly single tokens,
    token by token with fp32 products.  (The reference has no recurrent mixer.)"""

    use_tensor_cores = True
    chunk_min_tokens = 32       # tokens beyond one per portion from which the chunked form runs

    def __init__(self, width: int, spec, eps: float, dtype=torch.bfloat16, device="cuda", stacked: bool = False):
        """`stacked`: the input and output matrices belong to whoever stacks this mixer with others."""
        super().__init__()
        P = lambda *shape, dt=dtype: nn.Parameter(torch.zeros(shape, dtype=dt, device=device), requires_grad=False)
        s = self.spec = spec
        if s.heads % s.groups or s.inner % s.norm_groups:
            raise ValueError("state-space heads must divide into the groups, and the inner size into the norm groups")
        self.width, self.eps = width, eps
        self.n_out = s.inner
        self.n_rows = s.inner + s.channels + s.heads
        self.n_in = (self.n_rows + 7) // 8 * 8
        self.w_in, self.o = (None, None) if stacked else (P(self.n_in, width), P(width, self.n_out))
        self.conv_w, self.conv_b = P(s.channels, s.conv), P(s.channels)
        self.dt_bias, self.a_log, self.d_skip = P(s.heads, dt=torch.float32), P(s.heads, dt=torch.float32), P(s.heads, dt=torch.float32)
        self.norm = P(s.inner)

    def load_in(self, loader, prefix: str) -> torch.Tensor:
        return loader.load_tensor(prefix + "in", "cpu")

    def load_rest(self, loader, prefix: str):
        t = lambda n: loader.load_tensor(prefix + n, "cpu")
        self.conv_w.data.copy_(t("conv"))
        self.conv_b.data.copy_(t("conv.b"))
        self.dt_bias.data.copy_(t("dt_bias").float())
        self.a_log.data.copy_(t("A_log").float())
        self.d_skip.data.copy_(t("D").float())
        self.norm.data.copy_(t("norm"))

    def load(self, loader, prefix: str):
        self.w_in.data[:self.n_rows].copy_(self.load_in(loader, prefix))
        self.load_rest(loader, prefix)
        self.o.data.copy_(loader.load_tensor(prefix + "o", "cpu"))

    def mix(self, proj: torch.Tensor, off: int, batch, cache, cache_idx: int, out: torch.Tensor, out_scale: float = 1.0) -> torch.Tensor:
        """proj [T, >= off + n_rows]; out [T, n_out], a view of any row stride"""
        s, T, dev, dt = self.spec, proj.shape[0], proj.device, proj.dtype
        lib, code, st = native.seq_lib(), native.GGML_BF16 if dt == torch.bfloat16 else native.GGML_F32, torch.cuda.current_stream(dev).cuda_stream
        state = cache.state[cache_idx]
        a = native.SsdParams(proj=proj.data_ptr(), proj_stride=proj.stride(0), xbc_off=off + s.inner, dt_off=off + s.inner + s.channels, conv_w=self.conv_w.data_ptr(),
                             conv_b=self.conv_b.data_ptr(), taps=s.conv, dt_bias=self.dt_bias.data_ptr(), a_log=self.a_log.data_ptr(), d_skip=self.d_skip.data_ptr(), heads=s.heads,
                             groups=s.groups, state_size=s.state_size, vdim=s.vdim, seq_of=batch.seq_of.data_ptr(), seqs=batch.seqs.data_ptr(), seqs_stride=batch.seqs.stride(0),
                             n_seqs=batch.n_seqs, state=state.data_ptr(), state_stride=state.stride(0))
        y = torch.empty((T, s.inner), dtype=torch.float32, device=dev)
        if T == batch.n_seqs:
            native.check_seq(lib.ktb200_ssd_step(C.byref(a), y.data_ptr(), code, st))
        else:
            xbc = torch.empty((T, s.channels), dtype=dt, device=dev)
            native.check_seq(lib.ktb200_ssd_conv(C.byref(a), xbc.data_ptr(), T, code, st))
            chunked = self.use_tensor_cores and T - batch.n_seqs >= self.chunk_min_tokens
            native.check_seq(lib.ktb200_ssd_scan(C.byref(a), xbc.data_ptr(), y.data_ptr(), code, int(chunked), st))
        native.check_seq(lib.ktb200_gated_group_norm(y.data_ptr(), proj[:, off:].data_ptr(), proj.stride(0), self.norm.data_ptr(), s.norm_groups, float(self.eps), float(out_scale),
                                                     out.data_ptr(), out.stride(0), T, s.inner, code, st))
        return out

    def forward(self, h: torch.Tensor, batch, cache, cache_idx: int) -> torch.Tensor:
        proj = nn.functional.linear(h, self.w_in)
        o = torch.empty((h.shape[0], self.n_out), dtype=h.dtype, device=h.device)
        return nn.functional.linear(self.mix(proj, 0, batch, cache, cache_idx, o), self.o)


class KRetention(nn.Module):
    """Retention — linear attention whose matrix state per head decays by one fixed number, with rotated queries and keys, unit-rms head outputs and an
    output gate:

        S <- decay_h S + k v^T ,  o = S^T q                     per head, q = rot(W_q h), k = rot(W_k h) / sqrt(dim), v = W_v h; S in fp32
        out = W_o (o / sqrt(mean_vdim(o^2) + eps) * silu(W_g h))

        P     = [W_q ; W_k ; W_v ; W_g] h                       one GEMM over the matrices that read the mixer input
        turns                                                    ktb200_turn_table, once per step for all layers of one rotation
        o     = prompt portions: ktb200_retention_chunk (bf16: chunks of 64 tokens in parallel, norm and gate included), or
                ktb200_retention_scan + ktb200_gla_out (fp32, other sizes, short portions); decode steps: ktb200_retention_step
        out   = W_o o                                           GEMM

    The state starts at zero and lives in the cache manager's double-buffered fp32 state rows (models/custom_cache.PagedStateCache); there are no
    per-token cache rows.  Sizes, decays and the rotation are constructor parameters (models/configuration_lipadra.RetentionSpec); `cache_idx`
    picks the cache layer.  (The reference has no recurrent mixer.)"""

    use_tensor_cores = True
    chunk_min_tokens = 32       # tokens beyond one per portion from which the chunked form runs

    def __init__(self, width: int, spec, eps: float, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        P = lambda *shape: nn.Parameter(torch.zeros(shape, dtype=dtype, device=device), requires_grad=False)
        s = self.spec = spec
        self.width, self.eps = width, eps
        up = lambda n: (n + 7) // 8 * 8       # q, k, v and g start 16-byte aligned in every row of P
        self.n_qk, self.n_v = s.heads * s.dim, s.heads * s.vdim
        self.offsets = [0, up(self.n_qk), 2 * up(self.n_qk), 2 * up(self.n_qk) + up(self.n_v)]
        self.n_in = self.offsets[3] + up(self.n_v)
        self.w_in, self.o = P(self.n_in, width), P(width, self.n_v)
        self.register_buffer("decay", torch.tensor(s.decay, dtype=torch.float32, device=device), persistent=False)
        self.register_buffer("decay_low", torch.tensor([x - float(y) for x, y in zip(s.decay, self.decay.tolist())], dtype=torch.float32, device=device), persistent=False)
        self.register_buffer("log2_decay", torch.tensor([math.log2(x) for x in s.decay], dtype=torch.float32, device=device), persistent=False)
        self.register_buffer("inv_freq", s.rot.inv_freq(device) if s.rot is not None else torch.zeros(1, dtype=torch.float64, device=device), persistent=False)

    def load(self, loader, prefix: str):
        for name, at in zip(("q", "k", "v", "g"), self.offsets):
            w = loader.load_tensor(prefix + name, "cpu")
            self.w_in.data[at:at + w.shape[0]].copy_(w)
        self.o.data.copy_(loader.load_tensor(prefix + "o", "cpu"))

    def forward(self, h: torch.Tensor, batch, cache, cache_idx: int) -> torch.Tensor:
        s, T, dev, dt = self.spec, h.shape[0], h.device, h.dtype
        lib, code, st = native.seq_lib(), native.GGML_BF16 if dt == torch.bfloat16 else native.GGML_F32, torch.cuda.current_stream(h.device).cuda_stream
        state = cache.state[cache_idx]
        proj = nn.functional.linear(h, self.w_in)
        turn = batch.turn_table(s.rot, self.inv_freq) if s.rot is not None else None
        q, k, v, g = self.offsets
        a = native.RetentionParams(proj=proj.data_ptr(), proj_stride=self.n_in, q_off=q, k_off=k, v_off=v, g_off=g, heads=s.heads, dim=s.dim, vdim=s.vdim,
                                   rot_dims=s.rot.dims if s.rot is not None else 0, rot_layout=s.rot.layout_code if s.rot is not None else 0,
                                   turn=turn.data_ptr() if turn is not None else None, k_scale=s.dim ** -0.5, decay=self.decay.data_ptr(), decay_low=self.decay_low.data_ptr(), log2_decay=self.log2_decay.data_ptr(),
                                   eps=float(self.eps), seqs=batch.seqs.data_ptr(), seqs_stride=batch.seqs.stride(0), n_seqs=batch.n_seqs, state=state.data_ptr(),
                                   state_stride=state.stride(0))
        out = torch.empty((T, self.n_v), dtype=dt, device=dev)
        if T == batch.n_seqs and s.vdim <= lib.ktb200_retention_step_max_vdim():
            native.check_seq(lib.ktb200_retention_step(C.byref(a), out.data_ptr(), code, st))
        elif self.use_tensor_cores and T - batch.n_seqs >= self.chunk_min_tokens and lib.ktb200_retention_chunk_supported(s.dim, s.vdim, code):
            ws = torch.empty(lib.ktb200_retention_chunk_workspace(s.heads, s.dim, s.vdim, T, batch.n_seqs), dtype=torch.uint8, device=dev)
            native.check_seq(lib.ktb200_retention_chunk(C.byref(a), out.data_ptr(), T, ws.data_ptr(), ws.numel(), code, st))
        else:
            o = torch.empty((T, self.n_v), dtype=torch.float32, device=dev)
            native.check_seq(lib.ktb200_retention_scan(C.byref(a), o.data_ptr(), code, st))
            native.check_seq(lib.ktb200_gla_out(o.data_ptr(), None, float(self.eps), proj[:, g:].data_ptr(), self.n_in, out.data_ptr(), T, s.heads, s.vdim, code, st))
        return nn.functional.linear(out, self.o)


class KSelectiveScan(nn.Module):
    """Mamba, the selective scan — a recurrent mixer whose channels keep `state_size` numbers each, every one with a decay of its own per token:

        [x | z] = W_in h ;  x = silu(filter(x) + b)             a causal filter of `conv` taps along time on every channel
        [r | B | C] = W_x x ;  dt = softplus(W_dt r + dt_b)     one dt per channel
        S_cn <- exp(-exp(A_log_cn) dt_c) S_cn + dt_c x_c B_n ;  y_c = sum_n S_cn C_n + D_c x_c             S in fp32
        out = W_o (y silu(z))

        P     = W_in h                                          GEMM
        x     = ktb200_conv_silu ;  p = W_x x ,  W_dt p[r]       two GEMMs
        y     = ktb200_selective_scan                           softplus, recurrence, skip and gate in one launch, prompts and decode steps alike
        out   = W_o y                                           GEMM

    A sequence's state — S and the last conv - 1 inputs of every channel — lives in the cache manager's double-buffered fp32 state rows
    (models/custom_cache.PagedStateCache).  Tokens of a portion run in order.  Sizes are constructor parameters
    (models/configuration_lipadra.SelectiveScanSpec); `cache_idx` picks the cache layer.  (The reference has no recurrent mixer.)"""

    def __init__(self, width: int, spec, eps: float, dtype=torch.bfloat16, device="cuda"):
        super().__init__()
        P = lambda *shape, dt=dtype: nn.Parameter(torch.zeros(shape, dtype=dt, device=device), requires_grad=False)
        s = self.spec = spec
        self.width = width
        up = lambda n: (n + 7) // 8 * 8       # x and z, and the step's, B's and C's columns, start 16-byte aligned in their rows
        self.z_off, self.b_off = up(s.inner), up(s.dt_rank)
        self.c_off = self.b_off + up(s.state_size)
        self.w_in, self.w_x = P(self.z_off + up(s.inner), width), P(self.c_off + up(s.state_size), s.inner)
        self.w_dt, self.o = P(s.inner, s.dt_rank), P(width, s.inner)
        self.conv_w, self.conv_b = P(s.inner, s.conv), P(s.inner)
        self.dt_bias, self.a, self.d_skip = P(s.inner, dt=torch.float32), P(s.inner, s.state_size, dt=torch.float32), P(s.inner, dt=torch.float32)

    def load(self, loader, prefix: str):
        s, t = self.spec, lambda n: loader.load_tensor(prefix + n, "cpu")
        w = t("in")
        self.w_in.data[:s.inner].copy_(w[:s.inner])
        self.w_in.data[self.z_off:self.z_off + s.inner].copy_(w[s.inner:])
        w = t("x")
        for at, lo, n in ((0, 0, s.dt_rank), (self.b_off, s.dt_rank, s.state_size), (self.c_off, s.dt_rank + s.state_size, s.state_size)):
            self.w_x.data[at:at + n].copy_(w[lo:lo + n])
        self.w_dt.data.copy_(t("dt"))
        self.conv_w.data.copy_(t("conv"))
        self.conv_b.data.copy_(t("conv.b"))
        self.dt_bias.data.copy_(t("dt.b").float())
        self.a.data.copy_(-torch.exp(t("A_log").float()))
        self.d_skip.data.copy_(t("D").float())
        self.o.data.copy_(t("o"))

    def forward(self, h: torch.Tensor, batch, cache, cache_idx: int) -> torch.Tensor:
        s, T, dev, dt = self.spec, h.shape[0], h.device, h.dtype
        lib, code, st = native.seq_lib(), native.GGML_BF16 if dt == torch.bfloat16 else native.GGML_F32, torch.cuda.current_stream(h.device).cuda_stream
        state = cache.state[cache_idx]
        proj = nn.functional.linear(h, self.w_in)
        x = torch.empty((T, s.inner), dtype=dt, device=dev)
        native.check_seq(lib.ktb200_conv_silu(proj.data_ptr(), proj.stride(0), self.conv_w.data_ptr(), self.conv_b.data_ptr(), s.conv, s.inner, batch.seq_of.data_ptr(),
                                              batch.seqs.data_ptr(), batch.seqs.stride(0), state.data_ptr(), state.stride(0), s.inner * s.state_size, x.data_ptr(), T, batch.n_seqs, code, st))
        p = nn.functional.linear(x, self.w_x)
        step = nn.functional.linear(p[:, :s.dt_rank], self.w_dt)
        a = native.SelectiveScanParams(x=x.data_ptr(), dt_logit=step.data_ptr(), b=p[:, self.b_off:].data_ptr(), c=p[:, self.c_off:].data_ptr(), z=proj[:, self.z_off:].data_ptr(),
                                       dt_stride=step.stride(0), bc_stride=p.stride(0), z_stride=proj.stride(0), dt_bias=self.dt_bias.data_ptr(), a=self.a.data_ptr(),
                                       d_skip=self.d_skip.data_ptr(), inner=s.inner, state_size=s.state_size, seqs=batch.seqs.data_ptr(), seqs_stride=batch.seqs.stride(0),
                                       n_seqs=batch.n_seqs, state=state.data_ptr(), state_stride=state.stride(0))
        y = torch.empty((T, s.inner), dtype=dt, device=dev)
        native.check_seq(lib.ktb200_selective_scan(C.byref(a), y.data_ptr(), T, code, st))
        return nn.functional.linear(y, self.o)
