"""Throughput and per-kernel rooflines of a step-function model at layer sizes of real models, with random weights, beside
the closest existing model's kernels at equal size (`bench.py --model lekapel`, `bench.py --model mabidra`,
`bench.py --model zivulix`, `bench.py --model bilurax`, `bench.py --model rununex`, `bench.py --model lipadra`).

Two parts:
  * end to end through the Engine (scheduler, paged cache, step function): prompt tokens/s for a long prompt cut into portions,
    decode tokens/s for 1 and 8 concurrent sequences, CUDA events around the steps;
  * kernel by kernel at DeepSeek-V3 attention / MoE sizes: each token-major kernel against its counterpart of the DeepSeek path
    (fused norm, latent prep, paged latent attention for decode, expert GEMVs), algorithmic bytes / event time / measured HBM
    peak.  L2 is flushed between timed launches (a 256 MB write)."""
from __future__ import annotations

import ctypes as C
import json
import os
import statistics
import sys

import torch

from .. import native

SIZES = {
    # name: (width, layers, mixer, dense ff, experts, top, expert ff, vocab)
    "2k-wide": dict(width=2048, n_layers=6, heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=768, window=1024, dense_ff=8192, experts=32, top=4, ff=1024, vocab=32768),
    "v3-layer": dict(width=7168, n_layers=2, heads=128, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536, window=4096, dense_ff=18432, experts=32, top=8, ff=2048, vocab=32768),
}


def make_config(s):
    mixer = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot_dim"], "vdim": s["vdim"], "kv_rank": s["kv_rank"], "q_rank": s["q_rank"],
             "rot": {"base": 10000.0, "dims": s["rot_dim"]}, "scale": (s["dim"] + s["rot_dim"]) ** -0.5, "mask": {"size": s["window"]}}
    layers = [{"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": s["dense_ff"]}}]
    layers += [{"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}}
               for _ in range(s["n_layers"] - 1)]
    return {"architecture": "Lekapel", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5, "groups": 4}, "residual_mult": 0.6, "logit_scale": 1.0, "layers": layers}


MABIDRA_SIZES = {
    # the same widths, feed-forward sizes and layer-run counts as SIZES; attention and linear-attention layers alternate, and the
    # span `loop` runs twice (6 layer runs for 5 layers / 3 for 2)
    "2k-wide": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, gla_heads=16, gla_dim=128, gla_vdim=128, rank=64, dense_ff=8192, experts=32, top=4, ff=1024, vocab=32768,
                    order="AGAGA", loop=(1, 2, 2), ctx=2048),
    "v3-layer": dict(width=7168, heads=64, kv_heads=8, dim=128, vdim=128, gla_heads=56, gla_dim=128, gla_vdim=128, rank=128, dense_ff=18432, experts=32, top=8, ff=2048, vocab=32768,
                     order="AG", loop=(1, 2, 2), ctx=4096),
}


def make_mabidra_config(s):
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "bias_max": 1024, "q_temp": {"coef": 0.1, "every": 512}}
    gla = {"heads": s["gla_heads"], "dim": s["gla_dim"], "vdim": s["gla_vdim"], "tau": 16.0}
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}
    layers = [{"type": "attention" if c == "A" else "gla", "mixer": attn if c == "A" else gla, "mlp": {"kind": "dense", "ff": s["dense_ff"]} if i == 0 else moe}
              for i, c in enumerate(s["order"])]
    return {"architecture": "Mabidra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5, "groups": 4}, "embedding": {"scale": 1.0}, "layers": layers,
            "loop": {"start": s["loop"][0], "stop": s["loop"][1], "times": s["loop"][2]}}


ZIVULIX_SIZES = {
    # the same widths and feed-forward sizes as SIZES, every feed-forward dense; A: soft-max window attention over grouped heads, D: gated
    # delta rule, L: latent attention at DeepSeek's latent sizes.  The closest existing model at equal size is Mabidra with sigmoid
    # attention where this has A or L and gated linear attention where this has D, the same dense feed-forward in every layer, no loop.
    "2k-wide": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, window=1024, d_heads=16, d_kv_heads=8, d_dim=128, d_vdim=128, conv=4, l_heads=16, dense_ff=8192,
                    vocab=32768, order="ADLAD", ctx=2048, rank=64),
    "v3-layer": dict(width=7168, heads=64, kv_heads=8, dim=128, vdim=128, window=4096, d_heads=56, d_kv_heads=28, d_dim=128, d_vdim=128, conv=4, l_heads=128, dense_ff=18432,
                     vocab=32768, order="ADL", ctx=4096, rank=128),
}


def make_zivulix_config(s):
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "softcap": 30.0, "mask": {"size": s["window"]},
            "rot": {"base": 10000.0, "dims": s["dim"] // 2, "scaling": {"factor": 4.0}}, "v_mix": True}
    delta = {"heads": s["d_heads"], "kv_heads": s["d_kv_heads"], "dim": s["d_dim"], "vdim": s["d_vdim"], "conv": s["conv"]}
    latent = {"heads": s["l_heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5, "rot": {"base": 10000.0, "dims": 64}}
    kinds = {"A": ("attention", attn), "D": ("delta", delta), "L": ("latent_attention", latent)}
    return {"architecture": "Zivulix", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": kinds[c][0], "mixer": kinds[c][1], "mlp": {"kind": "dense", "ff": s["dense_ff"]}} for c in s["order"]]}


BILURAX_SIZES = {
    # the same widths, feed-forward sizes, expert counts and layer-run counts as MABIDRA_SIZES (6 layer runs for 5 layers / 3 for 2, the first
    # layer dense, the others mixtures of experts, the span `loop` running twice); every mixer is chunked soft-max attention over the grouped
    # heads of Mabidra's attention layers.  The chunk is as long as the benchmark's context, and `ctx` puts the decoded token at a chunk's last
    # position, so that a decode step reads as many keys as Mabidra's attention does.  The closest existing model at equal size is Mabidra with
    # sigmoid attention in every layer (its experts have two matrices where these have three).
    "2k-wide": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, chunk=2048, dense_ff=8192, experts=32, top=4, groups=4, keep=2, ff=1024, vocab=32768, n_layers=5,
                    loop=(1, 2, 2), ctx=2047, rank=64),
    "v3-layer": dict(width=7168, heads=64, kv_heads=8, dim=128, vdim=128, chunk=4096, dense_ff=18432, experts=32, top=8, groups=4, keep=2, ff=2048, vocab=32768, n_layers=2,
                     loop=(1, 2, 2), ctx=4095, rank=128),
}


def make_bilurax_config(s):
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "softcap": 30.0, "mask": {"size": s["chunk"]}}
    moe = {"kind": "moe", "expert": {"ff": s["ff"], "limit": 7.0}, "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": s["groups"], "keep": s["keep"]}, "scale": 2.0}}
    layers = [{"type": "attention", "mixer": attn, "mlp": {"kind": "dense", "ff": s["dense_ff"]} if i == 0 else moe} for i in range(s["n_layers"])]
    return {"architecture": "Bilurax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "logit_softcap": 50.0, "layers": layers,
            "loop": {"start": s["loop"][0], "stop": s["loop"][1], "times": s["loop"][2]}}


def make_mabidra_attn_config(s):
    """Mabidra at the sizes of a Bilurax size entry: sigmoid attention in every layer, the same dense and expert feed-forward sizes, the same loop"""
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "bias_max": 1024, "q_temp": {"coef": 0.1, "every": 512}}
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}
    layers = [{"type": "attention", "mixer": attn, "mlp": {"kind": "dense", "ff": s["dense_ff"]} if i == 0 else moe} for i in range(s["n_layers"])]
    return {"architecture": "Mabidra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5, "groups": 4}, "embedding": {"scale": 1.0}, "layers": layers,
            "loop": {"start": s["loop"][0], "stop": s["loop"][1], "times": s["loop"][2]}}


RUNUNEX_SIZES = {
    # the same widths, expert sizes and counts as BILURAX_SIZES with every feed-forward a mixture plus a shared expert; P: chunked attention over the
    # grouped heads of Mabidra's attention layers side by side with a Mamba-2 state space of twice the width (heads of 64 channels, state 128),
    # D: differential attention with as many query and key columns.  The chunk is as long as the benchmark's context, and `ctx` puts the decoded
    # token at a chunk's last position.  The closest existing model at equal size is Mabidra: a sigmoid-attention layer without feed-forward
    # followed by a gated-linear-attention layer (as many state values) for P, a sigmoid-attention layer for D, the same routed experts (of two
    # matrices where these have three), no shared expert.
    "2k-wide": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, chunk=2048, s_heads=64, s_vdim=64, state=128, groups=4, conv=4, norm_groups=4, d_dim=64, experts=32, top=4, ff=1024,
                    shared_ff=2048, vocab=32768, order="PDPDP", ctx=2047, rank=64),
    "v3-layer": dict(width=7168, heads=64, kv_heads=8, dim=128, vdim=128, chunk=4096, s_heads=224, s_vdim=64, state=128, groups=8, conv=4, norm_groups=8, d_dim=64, experts=32, top=8, ff=2048,
                     shared_ff=2048, vocab=32768, order="PD", ctx=4095, rank=128),
}


def make_rununex_config(s):
    left = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "mask": {"size": s["chunk"]}}
    right = {"heads": s["s_heads"], "vdim": s["s_vdim"], "state": s["state"], "groups": s["groups"], "conv": s["conv"], "norm_groups": s["norm_groups"]}
    diff = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["d_dim"], "vdim": s["vdim"], "scale": s["d_dim"] ** -0.5, "mask": {"size": s["chunk"]}, "conv": s["conv"], "diff": 0.4,
            "rot": {"base": 500000.0, "dims": s["d_dim"], "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    kinds = {"P": ("parallel", {"left": left, "right": right, "left_scale": 0.7, "right_scale": 1.2}), "D": ("attention", diff)}
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}, "shared": {"ff": s["shared_ff"]}}
    return {"architecture": "Rununex", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 4.0}, "residual_mult": 0.5, "logit_scale": 0.5,
            "layers": [{"type": kinds[c][0], "mixer": kinds[c][1], "mlp": moe} for c in s["order"]]}


LIPADRA_SIZES = {
    # the same widths and expert sizes as RUNUNEX_SIZES; R: retention, M: the selective scan with twice the width in channels and 16 states each, A:
    # chunked attention over the grouped heads of Mabidra's attention layers; every feed-forward a mixture with a quarter as many identity experts
    # as experts, plus a shared expert.  The chunk is as long as the benchmark's context, and `ctx` puts the decoded token at a chunk's last
    # position.  The closest existing model at equal size is Mabidra: gated linear attention of the same heads for R and of as many channels for M,
    # sigmoid attention for A, the same routed experts (of two matrices where these have three), no shared expert, no identity experts.
    "2k-wide": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, chunk=2048, r_heads=16, r_dim=128, r_vdim=128, inner=4096, state=16, dt_rank=128, conv=4, experts=32, identity=8, top=4, groups=4,
                    keep=2, ff=1024, shared_ff=2048, vocab=32768, order="RMARM", ctx=2047, rank=64),
    "v3-layer": dict(width=7168, heads=64, kv_heads=8, dim=128, vdim=128, chunk=4096, r_heads=56, r_dim=128, r_vdim=128, inner=14336, state=16, dt_rank=448, conv=4, experts=32, identity=8, top=8,
                     groups=4, keep=2, ff=2048, shared_ff=2048, vocab=32768, order="RMA", ctx=4095, rank=128),
}


def make_lipadra_config(s):
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "mask": {"size": s["chunk"]},
            "rot": {"base": 10000.0, "dims": s["dim"] // 2}}
    ret = {"heads": s["r_heads"], "dim": s["r_dim"], "vdim": s["r_vdim"], "decay": [1.0 - 2.0 ** (-4.0 - 6.0 * h / s["r_heads"]) for h in range(s["r_heads"])],
           "rot": {"base": 10000.0, "dims": s["r_dim"]}}
    scan = {"inner": s["inner"], "state": s["state"], "dt_rank": s["dt_rank"], "conv": s["conv"]}
    kinds = {"A": ("attention", attn), "R": ("retention", ret), "M": ("mamba1", scan)}
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "shared": {"ff": s["shared_ff"]},
           "router": {"experts": s["experts"], "identity": s["identity"], "top": s["top"], "groups": {"count": s["groups"], "keep": s["keep"]}, "scale": 2.0}}
    return {"architecture": "Lipadra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "postln_alpha": 3.0,
            "layers": [{"type": kinds[c][0], "mixer": kinds[c][1], "mlp": moe} for c in s["order"]]}


def settle_lipadra(model):
    """the parameters whose usual range is not that of a projection or of a norm weight: small biases and corrections, negative state rates"""
    for pname, p in model.named_parameters():
        last = pname.rsplit(".", 1)[-1]
        if last in ("b_in", "conv_b", "correction"):
            p.data.sub_(1.0)
        elif last == "dt_bias":
            p.data.sub_(3.0)
        elif last == "a":
            p.data.copy_(-torch.arange(1, p.shape[1] + 1, device=p.device, dtype=torch.float32).expand_as(p))
        elif pname.endswith("router.weight"):      # as a bf16 checkpoint ships it
            p.data.copy_(p.data.bfloat16().float())
    for layer in model.owned.values():
        if layer.mlp is not None:
            layer.mlp.router.find_bf16()
    return model


def make_mabidra_recurrent_config(s):
    """Mabidra at the sizes of a Lipadra size entry: gated linear attention of the same heads for R and of as many channels for M, sigmoid attention
    for A, the same routed expert sizes"""
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "bias_max": 1024, "q_temp": {"coef": 0.1, "every": 512}}
    gla = lambda heads: {"heads": heads, "dim": s["r_dim"], "vdim": s["r_vdim"], "tau": 16.0}
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}
    kinds = {"A": ("attention", attn), "R": ("gla", gla(s["r_heads"])), "M": ("gla", gla(s["inner"] // s["r_vdim"]))}
    return {"architecture": "Mabidra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5, "groups": 4}, "embedding": {"scale": 1.0},
            "layers": [{"type": kinds[c][0], "mixer": kinds[c][1], "mlp": moe} for c in s["order"]]}


def make_mabidra_mixed_config(s):
    """Mabidra at the sizes of a Rununex size entry: per P a sigmoid-attention layer without feed-forward and a gated-linear-attention layer with as
    many state values, per D a sigmoid-attention layer, the same routed expert sizes"""
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "bias_max": 1024, "q_temp": {"coef": 0.1, "every": 512}}
    gla = {"heads": s["s_heads"] * s["s_vdim"] * s["state"] // (128 * 128), "dim": 128, "vdim": 128, "tau": 16.0}
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}
    layers = []
    for c in s["order"]:
        layers += [{"type": "attention", "mixer": attn, "mlp": None}, {"type": "gla", "mixer": gla, "mlp": moe}] if c == "P" else [{"type": "attention", "mixer": attn, "mlp": moe}]
    return {"architecture": "Mabidra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5, "groups": 4}, "embedding": {"scale": 1.0}, "layers": layers}


def make_mabidra_dense_config(s):
    """Mabidra at the sizes of a Zivulix size entry: sigmoid attention for A and L, gated linear attention for D, dense feed-forwards"""
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5, "bias_max": 1024, "q_temp": {"coef": 0.1, "every": 512}}
    gla = {"heads": s["d_heads"], "dim": s["d_dim"], "vdim": s["d_vdim"], "tau": 16.0}
    return {"architecture": "Mabidra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5, "groups": 4}, "embedding": {"scale": 1.0},
            "layers": [{"type": "gla" if c == "D" else "attention", "mixer": gla if c == "D" else attn, "mlp": {"kind": "dense", "ff": s["dense_ff"]}} for c in s["order"]]}


def random_model(cfg_dict, dtype=torch.bfloat16, device="cuda", size=None):
    if cfg_dict["architecture"] == "Lipadra":
        from ..models.configuration_lipadra import LipadraConfig
        from ..models.modeling_lipadra import LipadraForCausalLM
        model = LipadraForCausalLM(LipadraConfig.from_dict(cfg_dict), dtype=dtype, device=device)
    elif cfg_dict["architecture"] == "Rununex":
        from ..models.configuration_rununex import RununexConfig
        from ..models.modeling_rununex import RununexForCausalLM
        model = RununexForCausalLM(RununexConfig.from_dict(cfg_dict), dtype=dtype, device=device)
    elif cfg_dict["architecture"] == "Bilurax":
        from ..models.configuration_bilurax import BiluraxConfig
        from ..models.modeling_bilurax import BiluraxForCausalLM
        model = BiluraxForCausalLM(BiluraxConfig.from_dict(cfg_dict), dtype=dtype, device=device)
    elif cfg_dict["architecture"] == "Zivulix":
        from ..models.configuration_zivulix import ZivulixConfig
        from ..models.modeling_zivulix import ZivulixForCausalLM
        model = ZivulixForCausalLM(ZivulixConfig.from_dict(cfg_dict), dtype=dtype, device=device)
    elif cfg_dict["architecture"] == "Mabidra":
        from ..models.configuration_mabidra import MabidraConfig
        from ..models.modeling_mabidra import MabidraForCausalLM
        from ..operators.attention import distance_bias_table
        model = MabidraForCausalLM(MabidraConfig.from_dict(cfg_dict), dtype=dtype, device=device)
        for layer in model.layers:
            if hasattr(layer.mix, "set_rank"):
                layer.mix.set_rank(size["rank"])
            else:
                layer.mix.bias_table = distance_bias_table(torch.randn(64, layer.mix.spec.heads, device=device), layer.mix.spec.bias_max)
    else:
        from ..models.configuration_lekapel import LekapelConfig
        from ..models.modeling_lekapel import LekapelForCausalLM
        model = LekapelForCausalLM(LekapelConfig.from_dict(cfg_dict), dtype=dtype, device=device)
    g = torch.Generator(device=device).manual_seed(1)
    for name, p in model.named_parameters():
        if p.dim() == 1:
            p.data.copy_(1 + 0.1 * torch.randn(p.shape, generator=g, device=device))
        else:
            p.data.copy_(torch.randn(p.shape, generator=g, device=device, dtype=torch.float32) * p.shape[-1] ** -0.5)
    if cfg_dict["architecture"] == "Lipadra":
        settle_lipadra(model)
    return model.eval()


def model_bytes(model):
    return sum(p.numel() * p.element_size() for p in model.parameters())


def progress(msg):
    print("[model_bench] " + msg, file=sys.stderr, flush=True)


class Flusher:
    def __init__(self, dev):
        self.buf = torch.empty(256 << 20, dtype=torch.uint8, device=dev)

    def __call__(self):
        self.buf.fill_(1)


def timed(fn, flush, iters=10, warmup=3):
    for _ in range(warmup):
        fn()
    ts = []
    for _ in range(iters):
        flush()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return statistics.median(ts)


def engine_leg(name, size, flush, steps, warmup, family="lekapel"):
    from .engine import Engine
    cfg = {"lekapel": make_config, "mabidra": make_mabidra_config, "zivulix": make_zivulix_config, "mabidra-dense": make_mabidra_dense_config,
           "bilurax": make_bilurax_config, "mabidra-attn": make_mabidra_attn_config, "rununex": make_rununex_config, "mabidra-mixed": make_mabidra_mixed_config,
           "lipadra": make_lipadra_config, "mabidra-recurrent": make_mabidra_recurrent_config}[family](size)
    model = random_model(cfg, size=size)
    if family == "zivulix":      # norm weights are zero-centred, decays and the value blend inside their usual ranges
        for pname, p in model.named_parameters():
            if pname.endswith("weight") or pname.endswith("vmix") or pname.endswith("dt_bias"):
                p.data.sub_(1.0)
            if pname.endswith("a_log"):
                p.data.sub_(3.0)
    if family == "rununex":      # step logits and decays inside their usual ranges, small biases
        for pname, p in model.named_parameters():
            if pname.rsplit(".", 1)[-1] in ("dt_bias", "conv_b", "sink", "r2"):
                p.data.sub_(1.0 if not pname.endswith("r2") else 0.9)
    prompt_len, chunk, ctx = 4096, 2048, min(4096, size["window"] * 2) if family == "lekapel" else size["ctx"]
    eng = Engine(model, max_tokens=8 * (ctx + 64) + prompt_len, max_slots=9, max_step_tokens=chunk)
    g = torch.Generator().manual_seed(0)
    tok = lambda n: torch.randint(0, size["vocab"], (n,), generator=g).tolist()
    out = {"size": name, "config": {k: v for k, v in size.items()}, "weights_GB": model_bytes(model) / 1e9}
    progress(f"{family} {name}: model built")

    def prefill():
        p = tok(prompt_len)
        for lo in range(0, prompt_len, chunk):
            eng.step([("p", p[lo:lo + chunk], [len(p[lo:lo + chunk]) - 1] if lo + chunk >= prompt_len else [])], ["p"] if lo + chunk >= prompt_len else [])
    ms = timed(prefill, flush, iters=max(3, steps // 4), warmup=max(1, warmup // 2))
    out["prefill"] = {"prompt_tokens": prompt_len, "portion": chunk, "ms": ms, "tok_s": prompt_len / ms * 1e3}
    progress(f"{family} {name}: prefill {ms:.1f} ms")
    for bs in (1, 8):
        ids = [("d", i) for i in range(bs)]
        for i in ids:                                     # fill each sequence's cache to ctx tokens
            p = tok(ctx)
            for lo in range(0, ctx, chunk):
                eng.step([(i, p[lo:lo + chunk], [])])
        nxt = tok(bs)
        ms = timed(lambda: eng.step([(i, [t], [0]) for i, t in zip(ids, nxt)]), flush, iters=steps, warmup=warmup)
        for i in ids:
            eng.cache.close(i)
        out[f"decode_bs{bs}"] = {"ctx": ctx, "ms_per_step": ms, "tok_s": bs / ms * 1e3}
        progress(f"{family} {name}: decode x{bs} {ms:.3f} ms")
    return out


def kernel_leg(flush, peak_gbs, have_main_lib):
    """Token-major kernels against the DeepSeek path's kernels at DeepSeek-V3 sizes (bf16)."""
    dev, bf = torch.device("cuda"), torch.bfloat16
    seq = native.seq_lib()
    S = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731
    D, NH, R, ROPE, NOPE, QL, PAGE = 7168, 128, 512, 64, 128, 1536, 64
    rows = []

    def row(kernel, what, ms, nbytes, peer=None):
        r = {"kernel": kernel, "case": what, "us": ms * 1e3, "GBps": nbytes / ms / 1e6, "frac_of_measured_hbm": nbytes / ms / 1e6 / peak_gbs}
        if peer:
            r["closest"] = peer
        rows.append(r)
        return r

    g = torch.Generator(device=dev).manual_seed(7)
    rn = lambda *s, dt=bf: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(dt)
    main = native.lib() if have_main_lib else None
    for T in (1, 8, 2048):
        # ---- fused residual sum + grouped norm + shift  vs  add_rmsnorm
        x, a, b = rn(T, D, dt=torch.float32), rn(T, D), rn(T, D)
        w, mu = rn(D), rn(D)
        xo, h, hs = torch.empty_like(x), torch.empty(T, D, dtype=bf, device=dev), torch.empty(T, D, dtype=bf, device=dev)
        meta = torch.tensor([[-1] + list(range(T - 1)), [-1] * T, [-1] * (T - 1) + [0]], dtype=torch.int32, device=dev)
        st = torch.zeros(2, D, device=dev)
        fn = lambda: native.check_seq(seq.ktb200_group_rmsnorm_shift(x.data_ptr(), a.data_ptr(), 30, b.data_ptr(), 30, 0.6, None, xo.data_ptr(), w.data_ptr(), 4, 1e-5, mu.data_ptr(),
                                                                     meta[0].data_ptr(), meta[1].data_ptr(), meta[2].data_ptr(), st.data_ptr(), h.data_ptr(), hs.data_ptr(), T, D, 30, S()))
        ours = timed(fn, flush)
        peer = None
        if main is not None:
            r16, d16, o16 = rn(T, D), rn(T, D), torch.empty(T, D, dtype=bf, device=dev)
            ms = timed(lambda: native.check(main.ktb200_add_rmsnorm(r16.data_ptr(), d16.data_ptr(), w.data_ptr(), 1e-6, o16.data_ptr(), T, D, S())), flush)
            peer = {"kernel": "add_rmsnorm_kernel", "us": ms * 1e3, "GBps": T * D * 8 / ms / 1e6, "frac_of_measured_hbm": T * D * 8 / ms / 1e6 / peak_gbs}
        row("group_norm_shift_kernel", f"T={T} width={D}", ours, T * D * (4 + 2 + 2 + 4 + 2 + 2), peer)
    # ---- paged latent attention, decode, ctx 4096: ours (window 4096, sink) vs the tcgen05 MLA decode kernel
    for B, ctx in ((1, 4096), (8, 4096), (1, 32768)):
        pages = (ctx + PAGE - 1) // PAGE
        cache = rn(B * pages + 1, PAGE, R + ROPE)
        ptab = torch.arange(B * pages, dtype=torch.int32, device=dev).reshape(B, pages)
        q, q_abs, lat = rn(B, NH, NOPE + ROPE), rn(B, NH, R), torch.empty(B, NH, R, dtype=bf, device=dev)
        pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
        slot = torch.arange(B, dtype=torch.int32, device=dev)
        inv = torch.arange(ROPE // 2, dtype=torch.float64, device=dev).mul(-2.0 / ROPE).exp2()
        sink = torch.zeros(NH, device=dev)
        splits = max(1, min(32, ctx // 128, 296 // (B * NH // 8)))
        ws = torch.empty(max(1, seq.ktb200_latent_window_attn_workspace(B, NH, R, splits) // 4), device=dev)
        fn = lambda: native.check_seq(seq.ktb200_latent_window_attn(q.data_ptr(), q_abs.data_ptr(), NH, NOPE, ROPE, R, ROPE, 0, inv.data_ptr(), 0.07, sink.data_ptr(), ctx, pos.data_ptr(),
                                                                    slot.data_ptr(), ptab.data_ptr(), pages, PAGE, cache.data_ptr(), lat.data_ptr(), B, splits, ws.data_ptr(), 30, S()))
        ours = timed(fn, flush)
        nbytes = B * ctx * (R + ROPE) * 2
        peer = None
        if main is not None:
            qn, qp, o = rn(B, NH, R), rn(B, NH, ROPE), torch.empty(B, NH, R, dtype=bf, device=dev)
            kl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
            wsb = main.ktb200_mla_workspace_bytes(B, NH, 0)
            mws = torch.zeros(max(wsb, 16), dtype=torch.uint8, device=dev)
            mp = native.MlaParams(B, NH, PAGE, pages, 0, 0.07, qn.data_ptr(), qp.data_ptr(), cache.data_ptr(), ptab.data_ptr(), kl.data_ptr(), o.data_ptr(), None, mws.data_ptr(), wsb,
                                  (B * pages + 1) * PAGE)
            ms = timed(lambda: native.check(main.ktb200_mla_decode(C.byref(mp), S())), flush)
            peer = {"kernel": "mla_decode_tc_kernel", "us": ms * 1e3, "GBps": nbytes / ms / 1e6, "frac_of_measured_hbm": nbytes / ms / 1e6 / peak_gbs}
        row("latent_window_attn_kernel (+merge)", f"decode B={B} ctx={ctx} heads={NH} splits={splits}", ours, nbytes, peer)
        q_rot = rn(B, NH, ROPE)
        wsb = seq.ktb200_latent_window_attn_tc_workspace(B, NH, ctx, ctx)
        tws = torch.empty(wsb // 4, device=dev)
        fn = lambda: native.check_seq(seq.ktb200_latent_window_attn_tc(q_abs.data_ptr(), q_rot.data_ptr(), NH, 0.07, sink.data_ptr(), ctx, pos.data_ptr(), slot.data_ptr(),
                                                                       ptab.data_ptr(), pages, PAGE, cache.data_ptr(), (B * pages + 1) * PAGE, lat.data_ptr(), B, ctx, tws.data_ptr(), wsb, S()))
        row("mla_decode_tc_kernel<split P> (+merge with sink)", f"decode B={B} ctx={ctx} heads={NH}", timed(fn, flush), nbytes, peer)
    # ---- a prompt portion: 2048 tokens of one sequence at positions 2048..4095, window 4096 (work is FLOP-shaped: per token
    #      and head a (576 + 512)-long multiply-add per visible key)
    T, ctx = 2048, 4096
    pages = ctx // PAGE
    cache = rn(pages + 1, PAGE, R + ROPE)
    ptab = torch.arange(pages, dtype=torch.int32, device=dev).reshape(1, pages)
    q, q_abs, q_rot, lat = rn(T, NH, NOPE + ROPE), rn(T, NH, R), rn(T, NH, ROPE), torch.empty(T, NH, R, dtype=bf, device=dev)
    pos = torch.arange(ctx - T, ctx, dtype=torch.int32, device=dev)
    slot = torch.zeros(T, dtype=torch.int32, device=dev)
    inv = torch.arange(ROPE // 2, dtype=torch.float64, device=dev).mul(-2.0 / ROPE).exp2()
    sink = torch.zeros(NH, device=dev)
    flops = float(sum(range(ctx - T + 1, ctx + 1))) * NH * (R + ROPE + R) * 2
    wsb = seq.ktb200_latent_window_attn_tc_workspace(T, NH, ctx, ctx)
    tws = torch.empty(wsb // 4, device=dev)
    f_tc = lambda: native.check_seq(seq.ktb200_latent_window_attn_tc(q_abs.data_ptr(), q_rot.data_ptr(), NH, 0.07, sink.data_ptr(), ctx, pos.data_ptr(), slot.data_ptr(), ptab.data_ptr(),
                                                                     pages, PAGE, cache.data_ptr(), (pages + 1) * PAGE, lat.data_ptr(), T, ctx, tws.data_ptr(), wsb, S()))
    f_cc = lambda: native.check_seq(seq.ktb200_latent_window_attn(q.data_ptr(), q_abs.data_ptr(), NH, NOPE, ROPE, R, ROPE, 0, inv.data_ptr(), 0.07, sink.data_ptr(), ctx, pos.data_ptr(),
                                                                  slot.data_ptr(), ptab.data_ptr(), pages, PAGE, cache.data_ptr(), lat.data_ptr(), T, 1, None, 30, S()))
    for name, f, it in (("mla_decode_tc_kernel<split P> (+merge with sink)", f_tc, 5), ("latent_window_attn_kernel", f_cc, 2)):
        ms = timed(f, flush, iters=it, warmup=1)
        rows.append({"kernel": name, "case": f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={NH}", "us": ms * 1e3, "TFLOPs": flops / ms / 1e9})
    # ---- dense experts per pair (the fallback for rows too long for the by-expert kernels) : bytes = pairs * 3 * ff * width * 2
    E, top, ff = 32, 8, 2048
    Wg, Wu, Wd = rn(E, ff, D), rn(E, ff, D), rn(E, D, ff)
    for T in (1, 8):
        x = rn(T, D)
        ids = torch.stack([torch.randperm(E, generator=g, device=dev)[:top] for _ in range(T)]).to(torch.int64)
        wts = torch.rand(T, top, generator=g, device=dev)
        act, out = torch.empty(T * top, ff, dtype=bf, device=dev), torch.empty(T, D, device=dev)
        f1 = lambda: native.check_seq(seq.ktb200_experts_gate_up(x.data_ptr(), ids.data_ptr(), top, Wg.shape[0], Wg.data_ptr(), Wu.data_ptr(), act.data_ptr(), T, D, ff, 0, 0.0, None, 30, S()))
        f2 = lambda: native.check_seq(seq.ktb200_experts_down(act.data_ptr(), ids.data_ptr(), wts.data_ptr(), top, Wd.shape[0], Wd.data_ptr(), out.data_ptr(), T, D, ff, 30, S()))
        uniq = len(set(ids.flatten().tolist()))                            # every chosen expert is read from HBM at least once
        row("experts_gate_up_kernel", f"T={T} top={top} width={D} ff={ff} bf16", timed(f1, flush), uniq * 2 * ff * D * 2,
            {"kernel": "moe_block_kernel (Q4_K/Q6_K, whole block)", "frac_of_measured_hbm": 0.55, "note": "committed measurement of the DeepSeek path, one token"})
        row("experts_down_kernel", f"T={T} top={top} width={D} ff={ff} bf16", timed(f2, flush), uniq * ff * D * 2)
    # ---- the same by expert (what decode steps run): an expert's rows cross HBM once per two or four pairs routed to it
    for T in (1, 8, 16):
        x = rn(T, D)
        ids = torch.stack([torch.randperm(E, generator=g, device=dev)[:top] for _ in range(T)]).to(torch.int64)
        wts = torch.rand(T, top, generator=g, device=dev)
        act, out, pair_rows = torch.empty(T * top, ff, dtype=bf, device=dev), torch.empty(T, D, device=dev), torch.empty(T * top, D, device=dev)
        f1 = lambda: native.check_seq(seq.ktb200_experts_gate_up_by_expert(x.data_ptr(), ids.data_ptr(), top, E, Wg.data_ptr(), Wu.data_ptr(), act.data_ptr(), T, D, ff, 0, 0, 0.0, None, 30, S()))
        f2 = lambda: native.check_seq(seq.ktb200_experts_down_by_expert(act.data_ptr(), ids.data_ptr(), wts.data_ptr(), top, E, Wd.data_ptr(), pair_rows.data_ptr(), out.data_ptr(),
                                                                        T, D, ff, 0, 30, S()))
        uniq = len(set(ids.flatten().tolist()))
        row("experts_gate_up_by_expert_kernel", f"T={T} top={top} width={D} ff={ff} bf16", timed(f1, flush), uniq * 2 * ff * D * 2,
            {"kernel": "moe_block_kernel (Q4_K/Q6_K, whole block)", "frac_of_measured_hbm": 0.55, "note": "committed measurement of the DeepSeek path, one token"})
        row("experts_down_by_expert_kernel (+combine)", f"T={T} top={top} width={D} ff={ff} bf16", timed(f2, flush), uniq * ff * D * 2)
    return rows


def mabidra_kernel_leg(flush, peak_gbs, peak_tflops):
    """The kernels of the Mabidra operators at real layer sizes (bf16), each beside the like kernel of the Lekapel path."""
    dev, bf = torch.device("cuda"), torch.bfloat16
    seq = native.seq_lib()
    S = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731
    rows = []
    g = torch.Generator(device=dev).manual_seed(7)
    rn = lambda *s, dt=bf: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(dt)

    def row(kernel, what, ms, nbytes=None, flops=None, peer=None):
        r = {"kernel": kernel, "case": what, "us": ms * 1e3}
        progress(f"{kernel} {what}: {ms * 1e3:.1f} us")
        if nbytes is not None:
            r.update(GBps=nbytes / ms / 1e6, frac_of_measured_hbm=nbytes / ms / 1e6 / peak_gbs)
        if flops is not None:
            r.update(TFLOPs=flops / ms / 1e9, frac_of_measured_bf16=flops / ms / 1e9 / peak_tflops)
        if peer:
            r["closest"] = peer
        rows.append(r)

    D = 7168
    for T in (1, 8, 2048):      # residual sum + two grouped norms  vs  residual sum + grouped norm + token shift
        x, y, w1, w2 = rn(T, D, dt=torch.float32), rn(T, D), rn(D), rn(D)
        xo, h = torch.empty_like(x), torch.empty(T, D, dtype=bf, device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_group_rmsnorm_sandwich(x.data_ptr(), y.data_ptr(), 30, w1.data_ptr(), None, xo.data_ptr(), w2.data_ptr(), h.data_ptr(), 4,
                                                                                1e-5, 0.0, T, D, 30, S())), flush)
        a, b, mu, hs = rn(T, D), rn(T, D), rn(D), torch.empty(T, D, dtype=bf, device=dev)
        meta = torch.tensor([[-1] + list(range(T - 1)), [-1] * T, [-1] * (T - 1) + [0]], dtype=torch.int32, device=dev)
        st = torch.zeros(2, D, device=dev)
        ms = timed(lambda: native.check_seq(seq.ktb200_group_rmsnorm_shift(x.data_ptr(), a.data_ptr(), 30, b.data_ptr(), 30, 0.6, None, xo.data_ptr(), w1.data_ptr(), 4, 1e-5, mu.data_ptr(),
                                                                           meta[0].data_ptr(), meta[1].data_ptr(), meta[2].data_ptr(), st.data_ptr(), h.data_ptr(), hs.data_ptr(), T, D, 30,
                                                                           S())), flush)
        pb = T * D * (4 + 2 + 2 + 4 + 2 + 2)
        row("sandwich_norm_kernel", f"T={T} width={D}", ours, nbytes=T * D * (4 + 2 + 4 + 2),
            peer={"kernel": "group_norm_shift_kernel", "us": ms * 1e3, "frac_of_measured_hbm": pb / ms / 1e6 / peak_gbs})

    # ---- attention over the paged cache: 64 query heads on 8 key/value heads of 128 + 128 values; the Lekapel kernel beside it reads
    #      one latent row of 512 + 64 values per key for 128 heads (its tcgen05 path), the same bytes per key within 2x
    H, G, d, dv, PAGE = 64, 8, 128, 128, 64
    cw = G * (d + dv)
    bias, hb = rn(H, 1026, dt=torch.float32), rn(H, dt=torch.float32)

    def lekapel_attn(B, ctx, pos, slot, ptab, pages, T):
        R, ROPE, NH = 512, 64, 128
        cache = rn(B * pages + 1, PAGE, R + ROPE)
        q_abs, q_rot, lat = rn(T, NH, R), rn(T, NH, ROPE), torch.empty(T, NH, R, dtype=bf, device=dev)
        sink = torch.zeros(NH, device=dev)
        wsb = seq.ktb200_latent_window_attn_tc_workspace(T, NH, ctx, ctx)
        tws = torch.empty(wsb // 4, device=dev)
        return lambda: native.check_seq(seq.ktb200_latent_window_attn_tc(q_abs.data_ptr(), q_rot.data_ptr(), NH, 0.07, sink.data_ptr(), ctx, pos.data_ptr(), slot.data_ptr(),
                                                                         ptab.data_ptr(), pages, PAGE, cache.data_ptr(), (B * pages + 1) * PAGE, lat.data_ptr(), T, ctx, tws.data_ptr(),
                                                                         wsb, S()))

    from ..operators.attention import KSigmoidBiasAttention
    from ..models.configuration_mabidra import SigmoidAttentionSpec
    spec = SigmoidAttentionSpec(H, G, d, dv, d ** -0.5, 1024.0, 0.1, 512)
    picker = KSigmoidBiasAttention.pick_splits
    for B, ctx in ((1, 4096), (8, 4096), (1, 32768)):
        pages = (ctx + PAGE - 1) // PAGE
        cache = rn(B * pages + 1, PAGE, cw)
        ptab = torch.arange(B * pages, dtype=torch.int32, device=dev).reshape(B, pages)
        q, gate, out = rn(B, H, d), rn(B, H), torch.empty(B, H * dv, dtype=bf, device=dev)
        pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
        slot = torch.arange(B, dtype=torch.int32, device=dev)
        holder = type("X", (), {"spec": spec})()
        seqs = torch.tensor([list(range(B)), [1] * B, [-1] * B, [-1] * B], dtype=torch.int32, device=dev)
        ours = {}
        for tc in (1, 0):
            splits = picker(holder, B, ctx, B, bool(tc))
            ws = torch.empty(max(1, seq.ktb200_sigmoid_bias_attn_workspace(B, H, dv, splits) // 4), device=dev)
            fn = lambda: native.check_seq(seq.ktb200_sigmoid_bias_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, bias.data_ptr(), bias.shape[1], hb.data_ptr(), pos.data_ptr(), slot.data_ptr(),
                                                                       seqs.data_ptr(), B, B, ptab.data_ptr(), pages, PAGE, cache.data_ptr(), gate.data_ptr(), H, out.data_ptr(), B, splits,
                                                                       ws.data_ptr(), 30, tc, S()))
            ours[tc] = (timed(fn, flush), splits)
        ms = timed(lekapel_attn(B, ctx, pos, slot, ptab, pages, B), flush)
        lb = B * ctx * 576 * 2
        peer = {"kernel": "mla_decode_tc_kernel<split P> (+merge)", "case": "128 heads, latent 512 + 64", "us": ms * 1e3, "frac_of_measured_hbm": lb / ms / 1e6 / peak_gbs}
        row("sigmoid_attn_mma_kernel (+merge)", f"decode B={B} ctx={ctx} heads={H}/{G} splits={ours[1][1]}", ours[1][0], nbytes=B * ctx * cw * 2, peer=peer)
        row("sigmoid_attn_kernel (+merge), CUDA cores", f"decode B={B} ctx={ctx} heads={H}/{G} splits={ours[0][1]}", ours[0][0], nbytes=B * ctx * cw * 2, peer=peer)
    T, ctx = 2048, 4096
    pages = ctx // PAGE
    cache = rn(pages + 1, PAGE, cw)
    ptab = torch.arange(pages, dtype=torch.int32, device=dev).reshape(1, pages)
    q, gate, out = rn(T, H, d), rn(T, H), torch.empty(T, H * dv, dtype=bf, device=dev)
    pos = torch.arange(ctx - T, ctx, dtype=torch.int32, device=dev)
    slot = torch.zeros(T, dtype=torch.int32, device=dev)
    keys = float(sum(range(ctx - T + 1, ctx + 1)))
    seqs = torch.tensor([[0], [T], [-1], [-1]], dtype=torch.int32, device=dev)
    fn = lambda tc: native.check_seq(seq.ktb200_sigmoid_bias_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, bias.data_ptr(), bias.shape[1], hb.data_ptr(), pos.data_ptr(), slot.data_ptr(),
                                                                  seqs.data_ptr(), 1, 1, ptab.data_ptr(), pages, PAGE, cache.data_ptr(), gate.data_ptr(), H, out.data_ptr(), T, 1, None, 30,
                                                                  tc, S()))
    ours = timed(lambda: fn(1), flush, iters=5, warmup=2)
    slow = timed(lambda: fn(0), flush, iters=2, warmup=1)
    ms = timed(lekapel_attn(1, ctx, pos, slot, ptab, pages, T), flush, iters=3, warmup=1)
    lf = keys * 128 * (576 + 512) * 2
    row("sigmoid_attn_kernel, CUDA cores", f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={H}/{G}", slow, flops=keys * H * (d + dv) * 2)
    row("sigmoid_attn_mma_kernel", f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={H}/{G}", ours, flops=keys * H * (d + dv) * 2,
        peer={"kernel": "mla_decode_tc_kernel<split P>", "case": "128 heads, latent 512 + 64", "us": ms * 1e3, "TFLOPs": lf / ms / 1e9, "frac_of_measured_bf16": lf / ms / 1e9 / peak_tflops})

    # ---- gated linear attention: decode reads and writes the fp32 state once (bytes); a prompt portion is a chain of T dependent steps
    GH, gd, gdv = 56, 128, 128
    n_in = 2 * GH * gd + 2 * GH * gdv
    for B, T in ((1, 1), (8, 1), (1, 2048)):
        proj, z, zb = rn(B * T, n_in), rn(B * T, GH * gd), rn(GH * gd)
        state, o = torch.zeros(2 * B, GH * gd * gdv, device=dev), torch.empty(B * T, GH * gdv, device=dev)
        seqs = torch.tensor([[i * T for i in range(B)], [T] * B, [2 * i for i in range(B)], [2 * i + 1 for i in range(B)]], dtype=torch.int32, device=dev)
        fn = lambda: native.check_seq(seq.ktb200_gla_scan(proj.data_ptr(), n_in, 0, GH * gd, 2 * GH * gd, z.data_ptr(), GH * gd, zb.data_ptr(), 16.0, GH, gd, gdv, seqs.data_ptr(), B, B,
                                                          B * T, state.data_ptr(), o.data_ptr(), 30, S()))
        ms = timed(fn, flush, iters=5 if T > 1 else 10)
        if T == 1:
            row("gla_scan_kernel", f"decode B={B} heads={GH} dim={gd} vdim={gdv}", ms, nbytes=B * GH * gd * gdv * 8,
                peer={"note": "no recurrent mixer in the Lekapel path; its decode attention reads the cache rows once, as this reads the state once"})
        else:
            row("gla_scan_kernel", f"prompt portion T={T} heads={GH} dim={gd} vdim={gdv}", ms, flops=float(T) * GH * gd * gdv * 4,
                peer={"note": "fp32 CUDA-core recurrence (state and decays are fp32 by design): %.2f us per token step" % (ms * 1e3 / T)})
        og, gt, nw = torch.empty(B * T, GH * gdv, dtype=bf, device=dev), rn(B * T, GH * gdv), rn(gdv)
        ms = timed(lambda: native.check_seq(seq.ktb200_gla_out(o.data_ptr(), nw.data_ptr(), 1e-5, gt.data_ptr(), GH * gdv, og.data_ptr(), B * T, GH, gdv, 30, S())), flush)
        row("gla_out_kernel", f"T={B * T} heads={GH} vdim={gdv}", ms, nbytes=B * T * GH * gdv * (4 + 2 + 2))
    # ---- activation
    for T, ff in ((8, 18432), (2048, 18432)):
        zz, oo, pq, cf = rn(T, ff), torch.empty(T, ff, dtype=bf, device=dev), torch.tensor([0.3, -0.2], device=dev), torch.tensor([0.3, -0.2, 0.1, 0.0], device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_xielu(zz.data_ptr(), oo.data_ptr(), pq.data_ptr(), zz.numel(), 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_poly_norm(zz.data_ptr(), oo.data_ptr(), cf.data_ptr(), 1e-5, T, ff, 30, S())), flush)
        row("xielu_kernel", f"T={T} ff={ff}", ours, nbytes=T * ff * 4, peer={"kernel": "poly_norm_kernel", "us": ms * 1e3, "frac_of_measured_hbm": T * ff * 4 / ms / 1e6 / peak_gbs})
    # ---- experts without a gate matrix, by expert, beside the gated ones (same kernels, two thirds of the bytes)
    E, top, ff = 32, 8, 2048
    Wg, Wu, Wd = rn(E, ff, D), rn(E, ff, D), rn(E, D, ff)
    for T in (1, 8, 16):
        x = rn(T, D)
        ids = torch.stack([torch.randperm(E, generator=g, device=dev)[:top] for _ in range(T)]).to(torch.int64)
        act = torch.empty(T * top, ff, dtype=bf, device=dev)
        uniq = len(set(ids.flatten().tolist()))
        ours = timed(lambda: native.check_seq(seq.ktb200_experts_gate_up_by_expert(x.data_ptr(), ids.data_ptr(), top, E, None, Wu.data_ptr(), act.data_ptr(), T, D, ff, 0, 0, 0.0, None, 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_experts_gate_up_by_expert(x.data_ptr(), ids.data_ptr(), top, E, Wg.data_ptr(), Wu.data_ptr(), act.data_ptr(), T, D, ff, 0, 0, 0.0, None, 30, S())), flush)
        row("experts_gate_up_by_expert_kernel (no gate, relu^2)", f"T={T} top={top} width={D} ff={ff} bf16", ours, nbytes=uniq * ff * D * 2,
            peer={"kernel": "experts_gate_up_by_expert_kernel (gated)", "us": ms * 1e3, "frac_of_measured_hbm": uniq * 2 * ff * D * 2 / ms / 1e6 / peak_gbs})
    return rows


def zivulix_kernel_leg(flush, peak_gbs, peak_tflops):
    """The kernels of the Zivulix operators at real layer sizes (bf16), each beside the like kernel of the Mabidra path."""
    dev, bf = torch.device("cuda"), torch.bfloat16
    seq = native.seq_lib()
    S = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731
    rows = []
    g = torch.Generator(device=dev).manual_seed(7)
    rn = lambda *s, dt=bf: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(dt)

    def row(kernel, what, ms, nbytes=None, flops=None, peer=None):
        r = {"kernel": kernel, "case": what, "us": ms * 1e3}
        progress(f"{kernel} {what}: {ms * 1e3:.1f} us")
        if nbytes is not None:
            r.update(GBps=nbytes / ms / 1e6, frac_of_measured_hbm=nbytes / ms / 1e6 / peak_gbs)
        if flops is not None:
            r.update(TFLOPs=flops / ms / 1e9, frac_of_measured_bf16=flops / ms / 1e9 / peak_tflops)
        if peer:
            r["closest"] = peer
        rows.append(r)

    def peer_of(kernel, ms, nbytes=None, flops=None):
        r = {"kernel": kernel, "us": ms * 1e3}
        if nbytes is not None:
            r["frac_of_measured_hbm"] = nbytes / ms / 1e6 / peak_gbs
        if flops is not None:
            r.update(TFLOPs=flops / ms / 1e9, frac_of_measured_bf16=flops / ms / 1e9 / peak_tflops)
        return r

    D = 7168
    for T in (1, 8, 2048):      # residual sum + norm of the added term, the sum rounded for the next GEMM  vs  residual sum + two grouped norms
        x, y, w1, w2 = rn(T, D, dt=torch.float32), rn(T, D), rn(D), rn(D)
        xo, h = torch.empty_like(x), torch.empty(T, D, dtype=bf, device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_group_rmsnorm_sandwich(x.data_ptr(), y.data_ptr(), 30, w1.data_ptr(), None, xo.data_ptr(), None, h.data_ptr(), 1, 1e-6, 1.0,
                                                                                T, D, 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_group_rmsnorm_sandwich(x.data_ptr(), y.data_ptr(), 30, w1.data_ptr(), None, xo.data_ptr(), w2.data_ptr(), h.data_ptr(), 4, 1e-5,
                                                                              0.0, T, D, 30, S())), flush)
        nb = T * D * (4 + 2 + 4 + 2)
        row("sandwich_norm_kernel (zero-centred weights, plain h)", f"T={T} width={D}", ours, nbytes=nb, peer=peer_of("sandwich_norm_kernel (two grouped norms)", ms, nb))

    # ---- attention: 64 query heads on 8 key/value heads of 128 + 128 values, as the Mabidra attention beside it
    H, G, d, dv, PAGE = 64, 8, 128, 128, 64
    cw, n_in = G * (d + dv), (64 + 8) * 128 + 8 * 128
    inv = torch.arange(d // 4, dtype=torch.float64, device=dev).mul(-4.0 / d).exp2() / 4.0
    lam = torch.tensor([0.3], device=dev)
    for T in (8, 2048):         # rotation + unit rms + value blend + cache write  vs  per-head norms + temperature + cache write
        pages = (T + PAGE - 1) // PAGE
        proj, vo, cache, qo = rn(T, n_in), rn(T, G * dv), rn(pages + 1, PAGE, cw), torch.empty(T, H, d, dtype=bf, device=dev)
        ptab = torch.arange(pages, dtype=torch.int32, device=dev).reshape(1, pages)
        pos, slot = torch.arange(T, dtype=torch.int32, device=dev), torch.zeros(T, dtype=torch.int32, device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_rope_norm_cache_write(proj.data_ptr(), n_in, 0, H * d, (H + G) * d, H, G, d, dv, d // 2, 1, inv.data_ptr(), 1, None, None, 0, 1e-6,
                                                                               vo.data_ptr(), G * dv, lam.data_ptr(), pos.data_ptr(), slot.data_ptr(), ptab.data_ptr(), pages, PAGE,
                                                                               cache.data_ptr(), qo.data_ptr(), T, 30, S())), flush)
        qw, kw = rn(d), rn(d)
        ms = timed(lambda: native.check_seq(seq.ktb200_qk_norm_cache_write(proj.data_ptr(), n_in, H, G, d, dv, qw.data_ptr(), kw.data_ptr(), 1e-5, 0.1, 512, pos.data_ptr(),
                                                                           slot.data_ptr(), ptab.data_ptr(), pages, PAGE, cache.data_ptr(), qo.data_ptr(), T, 30, S())), flush)
        nb = T * (n_in + H * d + cw) * 2
        row("rope_norm_cache_write_kernel", f"T={T} heads={H}/{G} dim={d}", ours, nbytes=nb + T * G * dv * 2, peer=peer_of("qk_norm_cache_write_kernel", ms, nb))

    bias, hb = rn(H, 1026, dt=torch.float32), rn(H, dt=torch.float32)
    from ..models.configuration_mabidra import SigmoidAttentionSpec
    from ..models.configuration_zivulix import CappedWindowAttentionSpec
    from ..operators.attention import KCappedWindowAttention, KSigmoidBiasAttention
    for B, ctx in ((1, 4096), (8, 4096), (1, 32768)):
        pages = (ctx + PAGE - 1) // PAGE
        cache = rn(B * pages + 1, PAGE, cw)
        ptab = torch.arange(B * pages, dtype=torch.int32, device=dev).reshape(B, pages)
        q, gate, out = rn(B, H, d), rn(B, H), torch.empty(B, H * dv, dtype=bf, device=dev)
        pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
        slot = torch.arange(B, dtype=torch.int32, device=dev)
        seqs = torch.tensor([list(range(B)), [1] * B, [-1] * B, [-1] * B], dtype=torch.int32, device=dev)
        mine = type("X", (), {"spec": CappedWindowAttentionSpec(H, G, d, dv, d ** -0.5, 30.0, ctx, None, True, True)})()
        theirs = type("X", (), {"spec": SigmoidAttentionSpec(H, G, d, dv, d ** -0.5, 1024.0, 0.1, 512)})()
        sp = KSigmoidBiasAttention.pick_splits(theirs, B, ctx, B, True)
        ws = torch.empty(max(1, seq.ktb200_sigmoid_bias_attn_workspace(B, H, dv, sp) // 4), device=dev)
        ms = timed(lambda: native.check_seq(seq.ktb200_sigmoid_bias_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, bias.data_ptr(), bias.shape[1], hb.data_ptr(), pos.data_ptr(), slot.data_ptr(),
                                                                         seqs.data_ptr(), B, B, ptab.data_ptr(), pages, PAGE, cache.data_ptr(), gate.data_ptr(), H, out.data_ptr(), B, sp,
                                                                         ws.data_ptr(), 30, 1, S())), flush)
        nb = B * ctx * cw * 2
        peer = peer_of("sigmoid_attn_mma_kernel (+merge)", ms, nb)
        for tc in (1, 0):
            splits = KCappedWindowAttention.pick_splits(mine, B, ctx, B, bool(tc))
            ws2 = torch.empty(max(1, seq.ktb200_window_softmax_attn_workspace(B, H, dv, splits) // 4), device=dev)
            fn = lambda: native.check_seq(seq.ktb200_window_softmax_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, None, 30.0, ctx, 0, pos.data_ptr(), slot.data_ptr(), seqs.data_ptr(), B, B,
                                                                         ptab.data_ptr(), pages, PAGE, cache.data_ptr(), out.data_ptr(), B, splits, ws2.data_ptr(), 30, tc, S()))
            row("window_softmax_attn_mma_kernel (+merge)" if tc else "window_softmax_attn_kernel (+merge), CUDA cores", f"decode B={B} ctx={ctx} heads={H}/{G} splits={splits}",
                timed(fn, flush), nbytes=nb, peer=peer)
    T, ctx = 2048, 4096
    pages = ctx // PAGE
    cache = rn(pages + 1, PAGE, cw)
    ptab = torch.arange(pages, dtype=torch.int32, device=dev).reshape(1, pages)
    q, gate, out = rn(T, H, d), rn(T, H), torch.empty(T, H * dv, dtype=bf, device=dev)
    pos = torch.arange(ctx - T, ctx, dtype=torch.int32, device=dev)
    slot = torch.zeros(T, dtype=torch.int32, device=dev)
    keys = float(sum(range(ctx - T + 1, ctx + 1)))
    seqs = torch.tensor([[0], [T], [-1], [-1]], dtype=torch.int32, device=dev)
    fl = keys * H * (d + dv) * 2
    ms = timed(lambda: native.check_seq(seq.ktb200_sigmoid_bias_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, bias.data_ptr(), bias.shape[1], hb.data_ptr(), pos.data_ptr(), slot.data_ptr(),
                                                                     seqs.data_ptr(), 1, 1, ptab.data_ptr(), pages, PAGE, cache.data_ptr(), gate.data_ptr(), H, out.data_ptr(), T, 1, None, 30,
                                                                     1, S())), flush, iters=5, warmup=2)
    peer = peer_of("sigmoid_attn_mma_kernel", ms, flops=fl)
    fn = lambda tc, win: native.check_seq(seq.ktb200_window_softmax_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, None, 30.0, win, 0, pos.data_ptr(), slot.data_ptr(), seqs.data_ptr(), 1, 1,
                                                                         ptab.data_ptr(), pages, PAGE, cache.data_ptr(), out.data_ptr(), T, 1, None, 30, tc, S()))
    row("window_softmax_attn_mma_kernel", f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={H}/{G}, every earlier key in sight", timed(lambda: fn(1, ctx), flush, iters=5, warmup=2),
        flops=fl, peer=peer)
    row("window_softmax_attn_mma_kernel", f"the same, window 1024", timed(lambda: fn(1, 1024), flush, iters=5, warmup=2), flops=float(T) * 1024 * H * (d + dv) * 2)
    row("window_softmax_attn_kernel, CUDA cores", f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={H}/{G}", timed(lambda: fn(0, ctx), flush, iters=2, warmup=1), flops=fl)

    # ---- the gated delta rule: decode reads and writes the fp32 state once (bytes); a prompt portion is a chain of T dependent steps
    DH, DG, dd, ddv, taps = 56, 28, 128, 128, 4
    C_ = 2 * DG * dd + DH * ddv
    n_in = C_ + DH * ddv + 2 * DH
    n_in = (n_in + 7) // 8 * 8
    sw = DH * dd * ddv + (taps - 1) * C_
    GH, gd, gdv = 56, 128, 128
    g_in = 2 * GH * gd + 2 * GH * gdv
    for B, T in ((1, 1), (8, 1), (1, 2048)):
        proj, cwt = rn(B * T, n_in), rn(C_, taps)
        al, dtb = rn(DH, dt=torch.float32) - 3.0, rn(DH, dt=torch.float32)
        state = torch.zeros(2 * B, sw, device=dev)
        f32 = lambda *s: torch.empty(*s, device=dev)
        qn, kn, vv, be, de, o = f32(B * T, DG * dd), f32(B * T, DG * dd), f32(B * T, DH * ddv), f32(B * T, DH), f32(B * T, DH), f32(B * T, DH * ddv)
        seqs = torch.tensor([[i * T for i in range(B)], [T] * B, [2 * i for i in range(B)], [2 * i + 1 for i in range(B)]], dtype=torch.int32, device=dev)
        seq_of = torch.arange(B, dtype=torch.int32, device=dev).repeat_interleave(T)
        prep = lambda: native.check_seq(seq.ktb200_delta_prep(proj.data_ptr(), n_in, 0, C_ + DH * ddv, C_ + DH * ddv + DH, cwt.data_ptr(), taps, al.data_ptr(), dtb.data_ptr(), DH, DG, dd,
                                                              ddv, 1e-6, seq_of.data_ptr(), seqs.data_ptr(), B, state.data_ptr(), sw, qn.data_ptr(), kn.data_ptr(), vv.data_ptr(),
                                                              be.data_ptr(), de.data_ptr(), B * T, 30, S()))
        scan = lambda: native.check_seq(seq.ktb200_delta_scan(qn.data_ptr(), kn.data_ptr(), vv.data_ptr(), be.data_ptr(), de.data_ptr(), DH, DG, dd, ddv, seqs.data_ptr(), B, B,
                                                              state.data_ptr(), sw, o.data_ptr(), S()))
        prep()
        gproj, z, zb = rn(B * T, g_in), rn(B * T, GH * gd), rn(GH * gd)
        gstate, go = torch.zeros(2 * B, GH * gd * gdv, device=dev), torch.empty(B * T, GH * gdv, device=dev)
        gla = lambda: native.check_seq(seq.ktb200_gla_scan(gproj.data_ptr(), g_in, 0, GH * gd, 2 * GH * gd, z.data_ptr(), GH * gd, zb.data_ptr(), 16.0, GH, gd, gdv, seqs.data_ptr(), B, B,
                                                           B * T, gstate.data_ptr(), go.data_ptr(), 30, S()))
        it = 5 if T > 1 else 10
        ms_prep, ms_scan, ms_gla = timed(prep, flush, iters=it), timed(scan, flush, iters=it), timed(gla, flush, iters=it)
        row("delta_prep_kernel", f"B={B} T={T} heads={DH}/{DG} taps={taps}", ms_prep, nbytes=B * T * (C_ * 2 + C_ * 4 + 2 * DH * 4) + B * (taps - 1) * C_ * 8)
        if T == 1:
            nb = B * DH * dd * ddv * 8
            row("delta_scan_kernel", f"decode B={B} heads={DH}/{DG} dim={dd} vdim={ddv}", ms_scan, nbytes=nb, peer=peer_of("gla_scan_kernel", ms_gla, B * GH * gd * gdv * 8))
        else:
            fl = float(T) * DH * dd * ddv * 6
            row("delta_scan_kernel", f"prompt portion T={T} heads={DH}/{DG} dim={dd} vdim={ddv} ({ms_scan * 1e3 / T:.2f} us per token step)", ms_scan, flops=fl,
                peer=dict(peer_of("gla_scan_kernel", ms_gla, flops=float(T) * GH * gd * gdv * 4), us_per_token_step=ms_gla * 1e3 / T))
    # ---- activation
    for T, ff in ((8, 18432), (2048, 18432)):
        gu, oo, zz, pq = rn(T, 2 * ff), torch.empty(T, ff, dtype=bf, device=dev), rn(T, ff), torch.tensor([0.3, -0.2], device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_gated_act_mul(gu.data_ptr(), gu.data_ptr() + 2 * ff, 2 * ff, oo.data_ptr(), T, ff, 1, 0.0, None, 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_xielu(zz.data_ptr(), oo.data_ptr(), pq.data_ptr(), zz.numel(), 30, S())), flush)
        row("gated_act_mul_kernel (gelu_tanh)", f"T={T} ff={ff}", ours, nbytes=T * ff * 6, peer=peer_of("xielu_kernel", ms, T * ff * 4))
    return rows


def bilurax_kernel_leg(flush, peak_gbs, peak_tflops):
    """The kernels of the Bilurax operators at real layer sizes (bf16), each beside the like kernel of the closest existing path."""
    dev, bf = torch.device("cuda"), torch.bfloat16
    seq = native.seq_lib()
    S = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731
    rows = []
    g = torch.Generator(device=dev).manual_seed(7)
    rn = lambda *s, dt=bf: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(dt)

    def peer_of(kernel, ms, nbytes=None, flops=None):
        r = {"kernel": kernel, "us": ms * 1e3}
        if nbytes is not None:
            r["frac_of_measured_hbm"] = nbytes / ms / 1e6 / peak_gbs
        if flops is not None:
            r.update(TFLOPs=flops / ms / 1e9, frac_of_measured_bf16=flops / ms / 1e9 / peak_tflops)
        return r

    def row(kernel, what, ms, nbytes=None, flops=None, peer=None):
        r = dict(peer_of(kernel, ms, nbytes, flops), case=what)
        if nbytes is not None:
            r["GBps"] = nbytes / ms / 1e6
        progress(f"{kernel} {what}: {ms * 1e3:.1f} us")
        if peer:
            r["closest"] = peer
        rows.append(r)

    D = 7168
    from ..operators.norm import KGroupRMSNormShift
    for T in (1, 8, 2048):      # a pass opening: x + y + x0 + step, norm, shift  vs  Lekapel's x + m (a + b), norm in 4 groups, shift
        x, y, x0, step = rn(T, D, dt=torch.float32), rn(T, D), rn(T, D, dt=torch.float32), rn(D, dt=torch.float32)
        state = torch.zeros(2, D, device=dev)
        meta = torch.zeros(5, T, dtype=torch.int32, device=dev)
        meta[2] = torch.arange(-1, T - 1, dtype=torch.int32, device=dev)
        meta[3], meta[4] = -1, -1
        batch = type("B", (), {"prev_idx": meta[2], "rd_row": meta[3], "wr_row": meta[4]})()
        mine, theirs = KGroupRMSNormShift(D, 1, 1e-6, True), KGroupRMSNormShift(D, 4, 1e-5, True)
        ours = timed(lambda: mine(x, y, x0, 1.0, batch, state, want_h=False, row_add=step), flush)
        ms = timed(lambda: theirs(x, y, y, 0.6, batch, state, want_h=True), flush)
        row("group_norm_shift_kernel (two addends of which one fp32, a row vector, shifted output only)", f"T={T} width={D}", ours, nbytes=T * D * (4 + 2 + 4 + 4 + 2),
            peer=peer_of("group_norm_shift_kernel (two bf16 addends, 4 groups, both outputs)", ms, T * D * (4 + 2 + 2 + 4 + 2 + 2)))

    # ---- attention: 64 query heads on 8 key/value heads of 128 + 128 values
    H, G, d, dv, PAGE = 64, 8, 128, 128, 64
    cw, n_in = G * (d + dv), (64 + 8) * 128 + 8 * 128
    inv = torch.arange(d // 4, dtype=torch.float64, device=dev).mul(-4.0 / d).exp2() / 4.0
    lam = torch.tensor([0.3], device=dev)
    for T in (8, 2048):         # row-wide weighted q / k norms + value unit rms + cache write  vs  rotation + per-head unit rms + value blend + cache write
        pages = (T + PAGE - 1) // PAGE
        proj, vo, cache, qo = rn(T, n_in), rn(T, G * dv), rn(pages + 1, PAGE, cw), torch.empty(T, H, d, dtype=bf, device=dev)
        qw, kw = rn(H * d), rn(G * d)
        ptab = torch.arange(pages, dtype=torch.int32, device=dev).reshape(1, pages)
        pos, slot = torch.arange(T, dtype=torch.int32, device=dev), torch.zeros(T, dtype=torch.int32, device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_rope_norm_cache_write(proj.data_ptr(), n_in, 0, H * d, (H + G) * d, H, G, d, dv, 0, 0, None, 2, qw.data_ptr(), kw.data_ptr(), 1,
                                                                               1e-6, None, 0, None, pos.data_ptr(), slot.data_ptr(), ptab.data_ptr(), pages, PAGE, cache.data_ptr(),
                                                                               qo.data_ptr(), T, 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_rope_norm_cache_write(proj.data_ptr(), n_in, 0, H * d, (H + G) * d, H, G, d, dv, d // 2, 1, inv.data_ptr(), 1, None, None, 0, 1e-6,
                                                                             vo.data_ptr(), G * dv, lam.data_ptr(), pos.data_ptr(), slot.data_ptr(), ptab.data_ptr(), pages, PAGE,
                                                                             cache.data_ptr(), qo.data_ptr(), T, 30, S())), flush)
        nb = T * (n_in + H * d + cw) * 2
        row("rope_norm_cache_write_kernel (row-wide q/k norms, unit-rms values)", f"T={T} heads={H}/{G} dim={d}", ours, nbytes=nb,
            peer=peer_of("rope_norm_cache_write_kernel (rotation, per-head unit rms, value blend)", ms, nb + T * G * dv * 2))

    from ..operators.attention import softmax_attention_splits
    temp = 0.5 + torch.rand(H, device=dev)
    for B, ctx in ((1, 4096), (8, 4096), (1, 32768)):      # the chunk mask with a head temperature  vs  the window mask of the same kernel
        pages = (ctx + PAGE - 1) // PAGE
        cache = rn(B * pages + 1, PAGE, cw)
        ptab = torch.arange(B * pages, dtype=torch.int32, device=dev).reshape(B, pages)
        q, out = rn(B, H, d), torch.empty(B, H * dv, dtype=bf, device=dev)
        pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
        slot = torch.arange(B, dtype=torch.int32, device=dev)
        seqs = torch.tensor([list(range(B)), [1] * B, [-1] * B, [-1] * B], dtype=torch.int32, device=dev)
        nb = B * ctx * cw * 2
        for tc in (1, 0):
            splits = softmax_attention_splits(H, G, ctx, B, B, bool(tc))
            ws2 = torch.empty(max(1, seq.ktb200_window_softmax_attn_workspace(B, H, dv, splits) // 4), device=dev)
            fn = lambda hs, win, ch: native.check_seq(seq.ktb200_window_softmax_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, hs, 30.0, win, ch, pos.data_ptr(), slot.data_ptr(),
                                                                                     seqs.data_ptr(), B, B, ptab.data_ptr(), pages, PAGE, cache.data_ptr(), out.data_ptr(), B, splits,
                                                                                     ws2.data_ptr(), 30, tc, S()))
            ms = timed(lambda: fn(None, ctx, 0), flush)
            name = "window_softmax_attn_mma_kernel (+merge)" if tc else "window_softmax_attn_kernel (+merge), CUDA cores"
            row(name + ", chunk mask, head temperature", f"decode B={B} last position of a chunk of {ctx} heads={H}/{G} splits={splits}",
                timed(lambda: fn(temp.data_ptr(), 0, ctx), flush), nbytes=nb, peer=peer_of(name + ", window mask", ms, nb))
    T, ctx = 2048, 4096
    pages = ctx // PAGE
    cache = rn(pages + 1, PAGE, cw)
    ptab = torch.arange(pages, dtype=torch.int32, device=dev).reshape(1, pages)
    q, out = rn(T, H, d), torch.empty(T, H * dv, dtype=bf, device=dev)
    pos = torch.arange(ctx - T, ctx, dtype=torch.int32, device=dev)
    slot = torch.zeros(T, dtype=torch.int32, device=dev)
    seqs = torch.tensor([[0], [T], [-1], [-1]], dtype=torch.int32, device=dev)
    fn = lambda hs, win, ch: native.check_seq(seq.ktb200_window_softmax_attn(q.data_ptr(), H, G, d, dv, d ** -0.5, hs, 30.0, win, ch, pos.data_ptr(), slot.data_ptr(), seqs.data_ptr(), 1, 1,
                                                                             ptab.data_ptr(), pages, PAGE, cache.data_ptr(), out.data_ptr(), T, 1, None, 30, 1, S()))
    fl = float(sum(range(ctx - T + 1, ctx + 1))) * H * (d + dv) * 2
    ms = timed(lambda: fn(None, ctx, 0), flush, iters=5, warmup=2)
    row("window_softmax_attn_mma_kernel, chunk mask, head temperature", f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={H}/{G}, one chunk of {ctx}",
        timed(lambda: fn(temp.data_ptr(), 0, ctx), flush, iters=5, warmup=2), flops=fl, peer=peer_of("window_softmax_attn_mma_kernel, window mask", ms, flops=fl))
    fl = 2 * float(sum(range(1, 1025))) * H * (d + dv) * 2
    ms = timed(lambda: fn(None, 1024, 0), flush, iters=5, warmup=2)
    row("window_softmax_attn_mma_kernel, chunk mask, head temperature", f"the same, chunks of 1024 (half the keys of a window of 1024)",
        timed(lambda: fn(temp.data_ptr(), 0, 1024), flush, iters=5, warmup=2), flops=fl, peer=peer_of("window_softmax_attn_mma_kernel, window of 1024", ms, flops=float(T) * 1024 * H * (d + dv) * 2))

    # ---- router: 256 experts in 8 groups of which 4 are kept, 8 choices (DeepSeek-V3's shape)  vs  soft-max over all, 8 largest
    from ..operators.gate import KGroupedSigmoidGate, KSoftmaxTopKGate
    E, top = 256, 8
    mine, theirs = KGroupedSigmoidGate(D, E, top, 8, 4, 2.0), KSoftmaxTopKGate(D, E, top)
    mine.weight.data.copy_(rn(E, D, dt=torch.float32) * D ** -0.5)
    theirs.weight.data.copy_(mine.weight.data)
    mine.correction.data.copy_(rn(E, dt=torch.float32) * 0.1)
    for T in (1, 8, 2048):
        x = rn(T, D)
        ours, ms = timed(lambda: mine(x), flush), timed(lambda: theirs(x), flush)
        nb = E * D * 4 + T * D * 2
        small = T < mine.gemm_min_tokens
        row("gate_kernel (sigmoid, correction, groups)" if small else "fp32 GEMM + gate_select_kernel", f"T={T} experts={E} width={D} top={top}", ours, nbytes=nb,
            peer=peer_of("gate_kernel (soft-max, greedy)" if small else "fp32 GEMM + torch soft-max and top-k", ms, nb))

    # ---- experts: the clamped sigmoid form beside silu(gate) * up in the same kernels
    E, top, ff = 32, 8, 2048
    Wg, Wu = rn(E, ff, D) * D ** -0.5, rn(E, ff, D) * D ** -0.5
    for T in (1, 8):
        x, act = rn(T, D), torch.empty(T * top, ff, dtype=bf, device=dev)
        ids = torch.stack([torch.randperm(E, generator=g, device=dev)[:top] for _ in range(T)])
        uniq = int(ids.unique().numel())
        fn = lambda kind, lim: native.check_seq(seq.ktb200_experts_gate_up_by_expert(x.data_ptr(), ids.data_ptr(), top, E, Wg.data_ptr(), Wu.data_ptr(), act.data_ptr(), T, D, ff, 0, kind,
                                                                                     lim, None, 30, S()))
        ours, ms = timed(lambda: fn(2, 7.0), flush), timed(lambda: fn(0, 0.0), flush)
        nb = uniq * 2 * ff * D * 2
        row("experts_gate_up_by_expert_kernel (clamped sigmoid form)", f"T={T} top={top} width={D} ff={ff} bf16", ours, nbytes=nb,
            peer=peer_of("experts_gate_up_by_expert_kernel (silu)", ms, nb))
    # ---- elementwise: expert activation over grouped-GEMM outputs, relu squared, capped logits
    for P in (64, 2048 * 8):
        gg, uu, oo = rn(P, ff), rn(P, ff), torch.empty(P, ff, dtype=bf, device=dev)
        gu = rn(P, 2 * ff)
        ours = timed(lambda: native.check_seq(seq.ktb200_gated_act_mul(gg.data_ptr(), uu.data_ptr(), ff, oo.data_ptr(), P, ff, 2, 7.0, None, 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_gated_act_mul(gu.data_ptr(), gu.data_ptr() + 2 * ff, 2 * ff, oo.data_ptr(), P, ff, 1, 0.0, None, 30, S())), flush)
        row("gated_act_mul_kernel (clamped sigmoid form, separate gate and up rows)", f"pairs={P} ff={ff}", ours, nbytes=P * ff * 6,
            peer=peer_of("gated_act_mul_kernel (gelu_tanh, stacked rows)", ms, P * ff * 6))
    for T, F_ in ((8, 18432), (2048, 18432)):
        zz, oo, pq = rn(T, F_), torch.empty(T, F_, dtype=bf, device=dev), torch.tensor([0.3, -0.2], device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_relu_squared(zz.data_ptr(), oo.data_ptr(), zz.numel(), 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_xielu(zz.data_ptr(), oo.data_ptr(), pq.data_ptr(), zz.numel(), 30, S())), flush)
        row("relu_squared_kernel", f"T={T} ff={F_}", ours, nbytes=T * F_ * 4, peer=peer_of("xielu_kernel", ms, T * F_ * 4))
    for T, V in ((8, 32768), (2048, 32768)):
        zz, of, oo, pq = rn(T, V), torch.empty(T, V, device=dev), torch.empty(T, V, dtype=bf, device=dev), torch.tensor([0.3, -0.2], device=dev)
        ours = timed(lambda: native.check_seq(seq.ktb200_softcap(zz.data_ptr(), of.data_ptr(), zz.numel(), 30.0, 30, S())), flush)
        ms = timed(lambda: native.check_seq(seq.ktb200_xielu(zz.data_ptr(), oo.data_ptr(), pq.data_ptr(), zz.numel(), 30, S())), flush)
        row("softcap_kernel (bf16 in, fp32 out)", f"T={T} vocab={V}", ours, nbytes=T * V * 6, peer=peer_of("xielu_kernel", ms, T * V * 4))
    return rows


def rununex_kernel_leg(flush, peak_gbs, peak_tflops):
    """The kernels of the Rununex operators at real layer sizes (bf16), each beside the like kernel of the closest existing path."""
    dev, bf = torch.device("cuda"), torch.bfloat16
    seq = native.seq_lib()
    S = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731
    rows = []
    g = torch.Generator(device=dev).manual_seed(7)
    rn = lambda *s, dt=bf: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(dt)

    def peer_of(kernel, ms, nbytes=None, flops=None):
        r = {"kernel": kernel, "us": ms * 1e3}
        if nbytes is not None:
            r["frac_of_measured_hbm"] = nbytes / ms / 1e6 / peak_gbs
        if flops is not None:
            r.update(TFLOPs=flops / ms / 1e9, frac_of_measured_bf16=flops / ms / 1e9 / peak_tflops)
        return r

    def row(kernel, what, ms, nbytes=None, flops=None, peer=None, **more):
        r = dict(peer_of(kernel, ms, nbytes, flops), case=what, **more)
        if nbytes is not None:
            r["GBps"] = nbytes / ms / 1e6
        progress(f"{kernel} {what}: {ms * 1e3:.1f} us" + (f" (closest {peer['us']:.1f})" if peer else ""))
        if peer:
            r["closest"] = peer
        rows.append(r)

    class Batch:      # one sequence per entry of `lens`, each ending at position `ctx` - 1, on `pages` identity pages of 64 tokens
        def __init__(self, lens, ctx):
            T, B = sum(lens), len(lens)
            i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
            starts = [sum(lens[:i]) for i in range(B)]
            self.pos = torch.cat([torch.arange(ctx - n, ctx, dtype=torch.int32, device=dev) for n in lens])
            self.slot = torch.arange(B, dtype=torch.int32, device=dev).repeat_interleave(i32(lens).long())
            self.seq_of = self.slot
            self.seqs = i32([starts, lens, [2 * i for i in range(B)], [2 * i + 1 for i in range(B)]])
            self.n_seqs, self.n_tokens, self.max_kv = B, T, ctx
            self.page_size, self.max_pages_per_seq = 64, (ctx + 63) // 64
            self.page_table = torch.arange(B * self.max_pages_per_seq, dtype=torch.int32, device=dev).reshape(B, -1)

        def cache(self, width):
            return rn(self.n_seqs * self.max_pages_per_seq + 1, 64, width)

    D = 7168
    from ..operators.norm import KGroupRMSNormShift, KLayerNorm
    for _ in range(50):         # the first launches of a process also pay for what the host sets up
        KLayerNorm(D, 1e-6)(rn(1, D, dt=torch.float32))
    for T in (1, 8, 2048):      # x + m (a + b), layer norm  vs  the same sum with an RMS norm
        x, a, b = rn(T, D, dt=torch.float32), rn(T, D, dt=torch.float32), rn(T, D)
        mine, theirs = KLayerNorm(D, 1e-6), KGroupRMSNormShift(D, 1, 1e-6, False)
        nb = T * D * (4 + 4 + 2 + 4 + 2)
        row("residual_layernorm_kernel", f"T={T} width={D}", timed(lambda: mine(x, a, b, 0.5), flush), nbytes=nb,
            peer=peer_of("group_norm_shift_kernel (no shift)", timed(lambda: theirs(x, a, b, 0.5), flush), nb))

    # ---- cache write: 64 / 8 heads.  Filter + rotation of two maps of 64  vs  rotation + unit rms + value blend of heads of 128 (as many columns)
    from ..operators.attention import paged_softmax_attention, qkv_prep
    from ..models.configuration_lekapel import RotarySpec
    H, G, d, dv, taps = 64, 8, 128, 128, 4
    n_q, n_k, n_v, cw = H * d, G * d, G * dv, G * (d + dv)
    n_in = n_q + n_k + n_v
    rot = RotarySpec(500000.0, 64, factor=8.0, low=1.0, high=4.0, original=8192)
    inv, lam = rot.inv_freq(dev), torch.tensor([0.3], device=dev)
    for T in (8, 2048):
        bt = Batch([1] * 8 if T == 8 else [T], 4096)
        proj, cwt, vo, kv = rn(T, n_in), rn(n_in, taps), rn(T, n_v), bt.cache(cw)
        state = torch.zeros(2 * bt.n_seqs, (taps - 1) * n_in, device=dev)
        qo = torch.empty(T, H, d, dtype=bf, device=dev)
        nb = T * (n_in + n_q + cw) * 2
        nb_conv = nb + (bt.n_seqs * (taps - 1) * n_in * 8)
        theirs = lambda: native.check_seq(seq.ktb200_rope_norm_cache_write(proj.data_ptr(), n_in, 0, n_q, n_q + n_k, H, G, d, dv, d // 2, 0, inv.data_ptr(), 1, None, None, 0, 1e-6,
                                                                           vo.data_ptr(), n_v, lam.data_ptr(), bt.pos.data_ptr(), bt.slot.data_ptr(), bt.page_table.data_ptr(),
                                                                           bt.max_pages_per_seq, 64, kv.data_ptr(), qo.data_ptr(), T, 30, S()))
        peer = peer_of("rope_norm_cache_write_kernel (rotation, per-head unit rms, value blend)", timed(theirs, flush), nb + T * n_v * 2)
        row("conv_rope_cache_write_kernel (4 taps, two maps of 64, rotation)", f"T={T} heads={H}/{G}",
            timed(lambda: qkv_prep(proj, bt, bt, kv, H, G, 64, dv, (0, n_q, n_q + n_k), maps=2, rot=rot, inv_freq=inv, conv_w=cwt, state=state), flush), nbytes=nb_conv, peer=peer)
        row("rope_norm_cache_write_kernel (unit rms)", f"T={T} heads={H}/{G} dim={d}",
            timed(lambda: qkv_prep(proj, bt, bt, kv, H, G, d, dv, (0, n_q, n_q + n_k), qk_norm=1, eps=1e-6), flush), nbytes=nb, peer=peer)

    # ---- attention: distance bias + sink + gate, and differential maps  vs  the plain chunk mask of the same kernel over as many key columns
    r1, r2, sink = 0.3 + torch.rand(H, device=dev), 0.02 + 0.1 * torch.rand(H, device=dev), torch.rand(H, device=dev)

    def attn_rows(bt, chunk, what, nbytes=None, flops=None, iters=10, tcs=(True, False)):
        T = bt.n_tokens
        kv, q, gate, proj_gate = bt.cache(cw), rn(T, H, d), None, rn(T, n_in + H * dv)
        gate = proj_gate[:, n_in:]
        for tc in tcs:
            plain = timed(lambda: paged_softmax_attention(q, kv, bt, bt, H, G, d, dv, d ** -0.5, chunk=chunk, tensor_cores=tc), flush, iters=iters)
            nm = "window_softmax_attn_mma_kernel" if tc else "window_softmax_attn_kernel, CUDA cores"
            peer = peer_of(nm + ", chunk mask", plain, nbytes, flops)
            row(nm + ", distance bias, sink, gate", what,
                timed(lambda: paged_softmax_attention(q, kv, bt, bt, H, G, d, dv, d ** -0.5, chunk=chunk, tensor_cores=tc, dist_bias=(r1, r2), sink=sink, gate=gate), flush, iters=iters),
                nbytes, flops, peer)
            # (two maps of 64: the same query and key columns, twice the value products)
            row(nm + ", two maps of 64", what,
                timed(lambda: paged_softmax_attention(q, kv, bt, bt, H, G, 64, dv, 0.125, chunk=chunk, tensor_cores=tc, maps=2, lam=lam, rms_eps=1e-6, out_scale=0.6), flush, iters=iters),
                nbytes, flops * (d + 2 * dv) / (d + dv) if flops else None, peer)

    for B, ctx in ((1, 4096), (8, 4096), (1, 32768)):
        attn_rows(Batch([1] * B, ctx), ctx, f"decode B={B} last position of a chunk of {ctx} heads={H}/{G}", nbytes=B * ctx * cw * 2)
    T, ctx = 2048, 4096
    attn_rows(Batch([T], ctx), ctx, f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={H}/{G}, one chunk of {ctx}", flops=float(sum(range(ctx - T + 1, ctx + 1))) * H * (d + dv) * 2,
              iters=5, tcs=(True,))
    attn_rows(Batch([T], ctx), 1024, "the same, chunks of 1024", flops=2 * float(sum(range(1, 1025))) * H * (d + dv) * 2, iters=5, tcs=(True,))

    # ---- state space: 112 heads of 64 channels, state 128, 4 groups (as many state values as 56 heads of 128 x 128)  vs  gated linear attention
    P, sv, N, J = 112, 64, 128, 4
    inner, C_ = P * sv, P * sv + 2 * J * N
    s_in = (inner + C_ + P + 7) // 8 * 8
    sw = inner * N + (taps - 1) * C_
    GH, gd = 56, 128
    g_in = 4 * GH * gd
    cwt, cb, dtb, al, ds = rn(C_, taps), rn(C_), rn(P, dt=torch.float32) - 2.0, rn(P, dt=torch.float32), rn(P, dt=torch.float32)
    nw = rn(inner)
    for B, T in ((1, 1), (8, 1), (1, 2048)):
        bt = Batch([T] * B, max(T, 64))
        n = B * T
        proj, state = rn(n, s_in), torch.zeros(2 * B, sw, device=dev)
        xbc, y, oo = torch.empty(n, C_, dtype=bf, device=dev), torch.empty(n, inner, device=dev), torch.empty(n, inner, dtype=bf, device=dev)
        a = native.SsdParams(proj=proj.data_ptr(), proj_stride=s_in, xbc_off=inner, dt_off=inner + C_, conv_w=cwt.data_ptr(), conv_b=cb.data_ptr(), taps=taps, dt_bias=dtb.data_ptr(),
                             a_log=al.data_ptr(), d_skip=ds.data_ptr(), heads=P, groups=J, state_size=N, vdim=sv, seq_of=bt.seq_of.data_ptr(), seqs=bt.seqs.data_ptr(), seqs_stride=B, n_seqs=B,
                             state=state.data_ptr(), state_stride=sw)
        gproj, z, zb = rn(n, g_in), rn(n, GH * gd), rn(GH * gd)
        gstate, go = torch.zeros(2 * B, GH * gd * gd, device=dev), torch.empty(n, GH * gd, device=dev)
        gla = lambda: native.check_seq(seq.ktb200_gla_scan(gproj.data_ptr(), g_in, 0, GH * gd, 2 * GH * gd, z.data_ptr(), GH * gd, zb.data_ptr(), 16.0, GH, gd, gd, bt.seqs.data_ptr(), B, B, n,
                                                           gstate.data_ptr(), go.data_ptr(), 30, S()))
        it = 5 if T > 1 else 10
        ms_gla = timed(gla, flush, iters=it)
        if T == 1:
            nb = B * (inner * N * 8 + (taps - 1) * C_ * 8)
            row("ssd_step_kernel (filter and recurrence)", f"decode B={B} heads={P} x {sv} state={N}", timed(lambda: native.check_seq(seq.ktb200_ssd_step(C.byref(a), y.data_ptr(), 30, S())), flush),
                nbytes=nb, peer=peer_of("gla_scan_kernel", ms_gla, B * GH * gd * gd * 8))
        else:
            conv = lambda: native.check_seq(seq.ktb200_ssd_conv(C.byref(a), xbc.data_ptr(), n, 30, S()))
            DH, DG = 56, 28
            dC = 2 * DG * 128 + DH * 128
            d_in = dC + DH * 128 + 2 * DH
            dproj, dcw, dstate = rn(n, d_in), rn(dC, taps), torch.zeros(2, DH * 128 * 128 + (taps - 1) * dC, device=dev)
            f32 = lambda *s: torch.empty(*s, device=dev)
            qn, kn, vv, be, de = f32(n, DG * 128), f32(n, DG * 128), f32(n, DH * 128), f32(n, DH), f32(n, DH)
            al2, db2 = rn(DH, dt=torch.float32) - 3.0, rn(DH, dt=torch.float32)
            dprep = lambda: native.check_seq(seq.ktb200_delta_prep(dproj.data_ptr(), d_in, 0, dC + DH * 128, dC + DH * 128 + DH, dcw.data_ptr(), taps, al2.data_ptr(), db2.data_ptr(), DH, DG,
                                                                   128, 128, 1e-6, bt.seq_of.data_ptr(), bt.seqs.data_ptr(), B, dstate.data_ptr(), dstate.shape[1], qn.data_ptr(), kn.data_ptr(),
                                                                   vv.data_ptr(), be.data_ptr(), de.data_ptr(), n, 30, S()))
            row("conv_silu_kernel", f"T={T} channels={C_} taps={taps}", timed(conv, flush, iters=it), nbytes=n * C_ * 4,
                peer=peer_of("delta_prep_kernel", timed(dprep, flush, iters=it), n * dC * 6))
            conv()
            for tc, name in ((1, "ssd_chunk_kernel"), (0, "ssd_scan_kernel, CUDA cores")):
                ms = timed(lambda: native.check_seq(seq.ktb200_ssd_scan(C.byref(a), xbc.data_ptr(), y.data_ptr(), 30, tc, S())), flush, iters=it)
                row(name, f"prompt portion T={T} heads={P} x {sv} state={N}", ms, flops=float(T) * P * sv * N * 4, us_per_token_step=ms * 1e3 / T,
                    peer=dict(peer_of("gla_scan_kernel", ms_gla, flops=float(T) * GH * gd * gd * 4), us_per_token_step=ms_gla * 1e3 / T))
        gw = rn(gd)
        ms = timed(lambda: native.check_seq(seq.ktb200_gla_out(go.data_ptr(), gw.data_ptr(), 1e-6, gproj.data_ptr(), g_in, oo.data_ptr(), n, GH, gd, 30, S())), flush)
        row("gated_group_norm_kernel", f"T={n} width={inner} groups=8",
            timed(lambda: native.check_seq(seq.ktb200_gated_group_norm(y.data_ptr(), proj.data_ptr(), s_in, nw.data_ptr(), 8, 1e-6, 0.9, oo.data_ptr(), inner, n, inner, 30, S())), flush),
            nbytes=n * inner * 8, peer=peer_of("gla_out_kernel", ms, n * GH * gd * 8))

    # ---- router: plain sigmoid top 8 of 256  vs  soft-max over all, 8 largest
    from ..operators.gate import KSigmoidTopKGate, KSoftmaxTopKGate
    E, top = 256, 8
    mine, theirs = KSigmoidTopKGate(D, E, top), KSoftmaxTopKGate(D, E, top)
    mine.weight.data.copy_(rn(E, D, dt=torch.float32) * D ** -0.5)
    theirs.weight.data.copy_(mine.weight.data)
    for T in (1, 8, 2048):
        x = rn(T, D)
        ours, ms = timed(lambda: mine(x), flush), timed(lambda: theirs(x), flush)
        nb = E * D * 4 + T * D * 2
        small = T < mine.gemm_min_tokens
        row("gate_kernel (sigmoid, greedy)" if small else "fp32 GEMM + gate_select_kernel", f"T={T} experts={E} width={D} top={top}", ours, nbytes=nb,
            peer=peer_of("gate_kernel (soft-max, greedy)" if small else "fp32 GEMM + torch soft-max and top-k", ms, nb))

    # ---- experts: weights on the input beside weights on the output in the same kernels
    E, top, ff = 32, 8, 2048
    from ..operators.experts import KExpertsDense
    ex = KExpertsDense(D, ff, E)
    for p in ex.parameters():
        p.data.copy_(rn(*p.shape) * p.shape[-1] ** -0.5)
    for T in (1, 8, 2048):
        x = rn(T, D)
        ids = torch.stack([torch.randperm(E, generator=g, device=dev)[:top] for _ in range(T)])
        w = torch.rand(T, top, generator=g, device=dev)
        uniq = int(ids.unique().numel())
        kw = dict(nbytes=uniq * 3 * ff * D * 2) if T < 48 else dict(flops=float(T) * top * 3 * ff * D * 2)
        ms = timed(lambda: ex(x, ids, w), flush)
        row("experts, weight on the input (whole call)", f"T={T} top={top} of {E} width={D} ff={ff}", timed(lambda: ex(x, ids, w, on_input=True), flush),
            peer=peer_of("experts, weight on the output (whole call)", ms, **kw), **kw)
    return rows


class KernelRows:
    """rows of a kernel leg: times beside the like kernel of the closest path, as fractions of the measured peaks"""

    def __init__(self, peak_gbs, peak_tf):
        self.peak_gbs, self.peak_tf, self.rows = peak_gbs, peak_tf, []

    def measure(self, kernel, ms, nbytes=None, flops=None):
        r = {"kernel": kernel, "us": ms * 1e3}
        if nbytes is not None:
            r["GBps"], r["frac_of_measured_hbm"] = nbytes / ms / 1e6, nbytes / ms / 1e6 / self.peak_gbs
        if flops is not None:
            r["TFLOPs"], r["frac_of_measured_bf16"] = flops / ms / 1e9, flops / ms / 1e9 / self.peak_tf
        return r

    def add(self, kernel, case, ms, nbytes=None, flops=None, peer=None, **extra):
        r = dict(self.measure(kernel, ms, nbytes, flops), case=case, **extra)
        progress(f"{kernel} {case}: {ms * 1e3:.1f} us" + (f" (closest {peer['us']:.1f})" if peer else ""))
        if peer:
            r["closest"] = peer
        self.rows.append(r)


class KernelBatch:
    """one sequence per entry of `lens`, each ending at position `ctx` - 1, on identity pages of 64 tokens"""

    def __init__(self, lens, ctx, dev):
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
        B, starts = len(lens), [sum(lens[:i]) for i in range(len(lens))]
        self.pos = torch.cat([torch.arange(ctx - n, ctx, dtype=torch.int32, device=dev) for n in lens])
        self.slot = torch.arange(B, dtype=torch.int32, device=dev).repeat_interleave(i32(lens).long())
        self.seq_of = self.slot
        self.seqs = i32([starts, lens, [2 * i for i in range(B)], [2 * i + 1 for i in range(B)]])
        self.n_seqs, self.n_tokens, self.max_kv = B, sum(lens), ctx
        self.page_size, self.max_pages_per_seq = 64, (ctx + 63) // 64
        self.page_table = torch.arange(B * self.max_pages_per_seq, dtype=torch.int32, device=dev).reshape(B, -1)

    def cache(self, width, fill):
        return fill(self.n_seqs * self.max_pages_per_seq + 1, 64, width)


def lipadra_kernel_leg(flush, peak_gbs, peak_tf):
    """Lipadra's kernels beside their like kernels at DeepSeek-V3 widths (bf16)"""
    dev, bf = torch.device("cuda"), torch.bfloat16
    seq, S = native.seq_lib(), lambda: torch.cuda.current_stream().cuda_stream
    K = KernelRows(peak_gbs, peak_tf)
    g = torch.Generator(device=dev).manual_seed(7)
    rn = lambda *s, dt=bf: torch.randn(*s, generator=g, device=dev, dtype=torch.float32).to(dt)
    f32, ok = torch.float32, native.check_seq
    from ..operators.attention import paged_softmax_attention, qkv_prep
    from ..operators.experts import KExpertsDense
    from ..operators.gate import KGroupedSigmoidGate, KGroupedSoftmaxGate
    from ..operators.norm import KLayerNorm, KSumRMSNorm
    from ..models.configuration_lekapel import RotarySpec
    D, top = 7168, 8
    for _ in range(50):         # the first launches of a process also pay for what the host sets up
        KLayerNorm(D, 1e-6)(rn(1, D, dt=f32))
    for T in (1, 8, 2048):      # the sum with identity experts and a gated addend, RMS norm  vs  the sum of two addends, layer norm
        x, a, b, bs, dot = rn(T, D, dt=f32), rn(T, D, dt=f32), rn(T, D), torch.rand(T, device=dev), rn(D)
        ids, iw = torch.randint(0, 40, (T, top), device=dev), torch.rand(T, top, device=dev)
        mine, theirs, nb = KSumRMSNorm(D, 1e-6), KLayerNorm(D, 1e-6), T * D * (4 + 4 + 2 + 4 + 2)
        peer = K.measure("residual_layernorm_kernel", timed(lambda: theirs(x, a, b, 0.5), flush), nb)
        K.add("sum_rmsnorm_kernel (identity experts, gated addend)", f"T={T} width={D}", timed(lambda: mine(x, 3.0, a, b, bs, (ids, iw, 32)), flush), nb, peer=peer)
        K.add("sum_rmsnorm_kernel (one addend, gate dot)", f"T={T} width={D}", timed(lambda: mine(x, 3.0, a=b, dot=dot), flush), T * D * (4 + 2 + 4 + 2),
              peer=K.measure("residual_layernorm_kernel (one addend)", timed(lambda: theirs(x, b, None, 0.5), flush), T * D * (4 + 2 + 4 + 2)))

    # ---- attention: 64 / 8 heads of 128; weighted norms ahead of half a rotation; one added to the denominator
    H, G, d, dv = 64, 8, 128, 128
    n_q, n_k, n_v, cw = H * d, G * d, G * dv, G * (d + dv)
    n_in = n_q + n_k + n_v
    rot = RotarySpec(10000.0, 64, layout="halves")
    inv, qw, kw, zero = rot.inv_freq(dev), rn(d), rn(d), torch.zeros(H, device=dev)
    for T in (8, 2048):
        bt = KernelBatch([1] * 8 if T == 8 else [T], 4096, dev)
        proj, kv, nb = rn(T, n_in), bt.cache(cw, rn), T * (n_in + n_q + cw) * 2
        prep = lambda **o: timed(lambda: qkv_prep(proj, bt, bt, kv, H, G, d, dv, (0, n_q, n_q + n_k), eps=1e-6, rot=rot, inv_freq=inv, **o), flush)
        K.add("rope_norm_cache_write_kernel (weighted norm, then rotation)", f"T={T} heads={H}/{G} dim={d}", prep(qk_norm=3, q_weight=qw, k_weight=kw), nb,
              peer=K.measure("rope_norm_cache_write_kernel (rotation, then unit rms)", prep(qk_norm=1), nb))
    cases = [(KernelBatch([1] * B, ctx, dev), ctx, f"decode B={B} last position of a chunk of {ctx} heads={H}/{G}", B * ctx * cw * 2, None) for B, ctx in ((1, 4096), (8, 4096), (1, 32768))]
    T, ctx = 2048, 4096
    cases += [(KernelBatch([T], ctx, dev), ctx, f"prompt portion T={T} positions {ctx - T}..{ctx - 1} heads={H}/{G}, one chunk of {ctx}", None, float(sum(range(ctx - T + 1, ctx + 1))) * H * (d + dv) * 2),
              (KernelBatch([T], ctx, dev), 1024, "the same, chunks of 1024", None, 2 * float(sum(range(1, 1025))) * H * (d + dv) * 2)]
    for bt, chunk, case, nb, fl in cases:
        kv, q = bt.cache(cw, rn), rn(bt.n_tokens, H, d)
        run_ = lambda **o: timed(lambda: paged_softmax_attention(q, kv, bt, bt, H, G, d, dv, d ** -0.5, chunk=chunk, **o), flush, iters=5 if fl else 10)
        K.add("window_softmax_attn_mma_kernel (+merge), one in the denominator", case, run_(sink=zero), nb, fl, peer=K.measure("the same kernel, plain soft-max", run_(), nb, fl))

    # ---- retention: 56 heads of 128 x 128  vs  Mamba-2 (112 heads of 64, state 128: as many state values) and gated linear attention of the same heads
    RH, P, sv, N, J, taps = 56, 112, 64, 128, 4, 4
    r_in, inner2 = 4 * RH * d, P * sv
    C_ = inner2 + 2 * J * N
    s_in, sw = (inner2 + C_ + P + 7) // 8 * 8, inner2 * N + (taps - 1) * C_
    rrot = RotarySpec(10000.0, 128, layout="halves")
    rinv, decays = rrot.inv_freq(dev), [1.0 - 2.0 ** (-4.0 - 6.0 * h / RH) for h in range(RH)]
    dec, low, l2 = torch.tensor(decays, device=dev), torch.zeros(RH, device=dev), torch.tensor(decays, device=dev).log2()
    scw, scb, dtb, al, ds = rn(C_, taps), rn(C_), rn(P, dt=f32) - 2.0, rn(P, dt=f32), rn(P, dt=f32)
    for B, T in ((1, 1), (8, 1), (1, 2048), (1, 8192)):
        bt = KernelBatch([T] * B, max(T, 64), dev)
        n, it = B * T, 5 if T > 1 else 10
        proj, state, out, o = rn(n, r_in), torch.zeros(2 * B, RH * d * dv, device=dev), torch.empty(n, RH * dv, dtype=bf, device=dev), torch.empty(n, RH * dv, device=dev)
        turn = torch.empty(n, 64, 2, device=dev)
        table = lambda: ok(seq.ktb200_turn_table(bt.pos.data_ptr(), rinv.data_ptr(), 64, turn.data_ptr(), n, S()))
        K.add("turn_table_kernel (once per step)", f"T={n} pairs=64", timed(table, flush), n * 64 * 8)
        a = native.RetentionParams(proj=proj.data_ptr(), proj_stride=r_in, q_off=0, k_off=RH * d, v_off=2 * RH * d, g_off=3 * RH * d, heads=RH, dim=d, vdim=dv, rot_dims=128, rot_layout=1,
                                   turn=turn.data_ptr(), k_scale=d ** -0.5, decay=dec.data_ptr(), decay_low=low.data_ptr(), log2_decay=l2.data_ptr(), eps=1e-6, seqs=bt.seqs.data_ptr(),
                                   seqs_stride=B, n_seqs=B, state=state.data_ptr(), state_stride=state.stride(0))
        z, zb, gw = rn(n, RH * d), rn(RH * d), rn(d)
        gla = lambda: ok(seq.ktb200_gla_scan(proj.data_ptr(), r_in, 0, RH * d, 2 * RH * d, z.data_ptr(), RH * d, zb.data_ptr(), 16.0, RH, d, dv, bt.seqs.data_ptr(), B, B, n, state.data_ptr(),
                                             o.data_ptr(), 30, S()))
        gout = lambda: ok(seq.ktb200_gla_out(o.data_ptr(), gw.data_ptr(), 1e-6, proj[:, 3 * RH * d:].data_ptr(), r_in, out.data_ptr(), n, RH, dv, 30, S()))
        sproj, sstate = rn(n, s_in), torch.zeros(2 * B, sw, device=dev)
        xbc, y = torch.empty(n, C_, dtype=bf, device=dev), torch.empty(n, inner2, device=dev)
        sa = native.SsdParams(proj=sproj.data_ptr(), proj_stride=s_in, xbc_off=inner2, dt_off=inner2 + C_, conv_w=scw.data_ptr(), conv_b=scb.data_ptr(), taps=taps, dt_bias=dtb.data_ptr(),
                              a_log=al.data_ptr(), d_skip=ds.data_ptr(), heads=P, groups=J, state_size=N, vdim=sv, seq_of=bt.seq_of.data_ptr(), seqs=bt.seqs.data_ptr(), seqs_stride=B, n_seqs=B,
                              state=sstate.data_ptr(), state_stride=sw)
        if T == 1:
            nb = B * RH * d * dv * 8
            both = lambda: (gla(), gout())
            K.add("retention_step_kernel (rotation, recurrence, norm, gate)", f"decode B={B} heads={RH} of {d} x {dv}", timed(lambda: ok(seq.ktb200_retention_step(C.byref(a), out.data_ptr(), 30, S())), flush),
                  nb, peer=K.measure("gla_scan_kernel + gla_out_kernel", timed(both, flush), nb),
                  like=K.measure("ssd_step_kernel", timed(lambda: ok(seq.ktb200_ssd_step(C.byref(sa), y.data_ptr(), 30, S())), flush), B * (inner2 * N + (taps - 1) * C_) * 8))
        else:
            fl = float(T) * RH * d * dv * 4
            ws = torch.empty(seq.ktb200_retention_chunk_workspace(RH, d, dv, n, B), dtype=torch.uint8, device=dev)
            ok(seq.ktb200_ssd_conv(C.byref(sa), xbc.data_ptr(), n, 30, S()))
            ssd = timed(lambda: ok(seq.ktb200_ssd_scan(C.byref(sa), xbc.data_ptr(), y.data_ptr(), 30, 1, S())), flush, iters=it)
            ms = timed(lambda: ok(seq.ktb200_retention_chunk(C.byref(a), out.data_ptr(), n, ws.data_ptr(), ws.numel(), 30, S())), flush, iters=it)
            K.add("retention_chunk_state + carry + chunk_out kernels", f"prompt portion T={T} heads={RH} of {d} x {dv}", ms, flops=fl, peer=K.measure("ssd_chunk_kernel", ssd, flops=float(T) * inner2 * N * 4),
                  frac_of_hbm_floor=n * RH * (3 * d + 2 * dv) * 2 / ms / 1e6 / peak_gbs)
            if T == 2048:
                K.add("retention_scan_kernel, CUDA cores", f"prompt portion T={T} heads={RH} of {d} x {dv}", timed(lambda: ok(seq.ktb200_retention_scan(C.byref(a), o.data_ptr(), 30, S())), flush, iters=it),
                      flops=fl, peer=K.measure("gla_scan_kernel", timed(gla, flush, iters=it), flops=fl))

    # ---- selective scan: 14336 channels of 16 states; its floor is the exponentials (one per channel, state and token: 16 a clock and SM)
    I, N1 = 14336, 16
    R_ = 448
    bcw = R_ + 2 * N1
    cwt, cb = rn(I, taps), rn(I)
    bias, A, Dk = rn(I, dt=f32) - 3.0, -torch.arange(1, N1 + 1, device=dev, dtype=f32).repeat(I, 1).contiguous(), rn(I, dt=f32)
    props = torch.cuda.get_device_properties(0)
    ex_per_s = props.multi_processor_count * 16 * 1.965e9
    for B, T in ((1, 1), (8, 1), (32, 1), (1, 2048), (8, 256)):      # (32 sequences hold as many state bytes as eight of the state-space layer's)
        bt = KernelBatch([T] * B, max(T, 64), dev)
        n, it = B * T, 5 if T > 1 else 10
        proj, p, step, x, y = rn(n, 2 * I), rn(n, bcw), rn(n, I), torch.empty(n, I, dtype=bf, device=dev), torch.empty(n, I, dtype=bf, device=dev)
        state = torch.zeros(2 * B, I * (N1 + taps - 1), device=dev)
        conv = lambda: ok(seq.ktb200_conv_silu(proj.data_ptr(), 2 * I, cwt.data_ptr(), cb.data_ptr(), taps, I, bt.seq_of.data_ptr(), bt.seqs.data_ptr(), B, state.data_ptr(), state.stride(0), I * N1,
                                               x.data_ptr(), n, B, 30, S()))
        nbc = n * I * 4 + B * (taps - 1) * I * 8
        K.add("conv_silu_kernel", f"T={n} ({B} portions) channels={I} taps={taps}", timed(conv, flush, iters=it), nbc)
        conv()
        a = native.SelectiveScanParams(x=x.data_ptr(), dt_logit=step.data_ptr(), b=p[:, R_:].data_ptr(), c=p[:, R_ + N1:].data_ptr(), z=proj[:, I:].data_ptr(), dt_stride=I, bc_stride=bcw, z_stride=2 * I,
                                       dt_bias=bias.data_ptr(), a=A.data_ptr(), d_skip=Dk.data_ptr(), inner=I, state_size=N1, seqs=bt.seqs.data_ptr(), seqs_stride=B, n_seqs=B, state=state.data_ptr(),
                                       state_stride=state.stride(0))
        ms = timed(lambda: ok(seq.ktb200_selective_scan(C.byref(a), y.data_ptr(), n, 30, S())), flush, iters=it)
        sproj, sstate = rn(n, s_in), torch.zeros(2 * B, sw, device=dev)
        xbc, sy = torch.empty(n, C_, dtype=bf, device=dev), torch.empty(n, inner2, device=dev)
        sa = native.SsdParams(proj=sproj.data_ptr(), proj_stride=s_in, xbc_off=inner2, dt_off=inner2 + C_, conv_w=scw.data_ptr(), conv_b=scb.data_ptr(), taps=taps, dt_bias=dtb.data_ptr(),
                              a_log=al.data_ptr(), d_skip=ds.data_ptr(), heads=P, groups=J, state_size=N, vdim=sv, seq_of=bt.seq_of.data_ptr(), seqs=bt.seqs.data_ptr(), seqs_stride=B, n_seqs=B,
                              state=sstate.data_ptr(), state_stride=sw)
        nb = n * (I * 8 + 4 * N1) + B * I * N1 * 8
        if T == 1:
            peer = K.measure("ssd_step_kernel", timed(lambda: ok(seq.ktb200_ssd_step(C.byref(sa), sy.data_ptr(), 30, S())), flush), B * (inner2 * N + (taps - 1) * C_) * 8)
        else:
            ok(seq.ktb200_ssd_conv(C.byref(sa), xbc.data_ptr(), n, 30, S()))
            peer = K.measure("ssd_chunk_kernel", timed(lambda: ok(seq.ktb200_ssd_scan(C.byref(sa), xbc.data_ptr(), sy.data_ptr(), 30, 1, S())), flush, iters=it),
                             n * (C_ * 2 + inner2 * 4) + B * inner2 * N * 8)
        K.add("selective_scan_kernel", f"{B} x {T} tokens, {I} channels of {N1}", ms, nb, peer=peer, frac_of_exponentials=n * I * N1 / ms * 1e3 / ex_per_s)

    # ---- router: grouped soft-max top 8 of 256 + 64  vs  grouped sigmoid
    E = 320
    mine, theirs = KGroupedSoftmaxGate(D, E, top, 8, 4, 2.0), KGroupedSigmoidGate(D, E, top, 8, 4, 2.0)
    mine.weight.data.copy_((rn(E, D, dt=f32) * D ** -0.5).bfloat16().float())
    theirs.weight.data.copy_(mine.weight.data)
    mine.bf16_min_tokens = 1
    for T in (1, 8, 2048):
        x, nb = rn(T, D), E * D * 4 + T * D * 2
        peer = K.measure("grouped sigmoid: " + ("gate_kernel" if T < mine.gemm_min_tokens else "fp32 GEMM + gate_select_kernel"), timed(lambda: theirs(x), flush), nb)
        mine.weight_bf16 = None
        K.add("gate_kernel (soft-max, biased group max)" if T < mine.gemm_min_tokens else "fp32 GEMM + gate_select_kernel", f"T={T} outputs={E} width={D} top={top}", timed(lambda: mine(x), flush),
              nb, peer=peer)
        mine.find_bf16()
        K.add("bf16 GEMM with fp32 sums + gate_select_kernel", f"T={T} outputs={E} width={D} top={top}", timed(lambda: mine(x), flush), E * D * 2 + T * D * 2, peer=peer)

    # ---- experts: a fifth of the choices identity experts  vs  every choice an expert
    E, ff = 32, 2048
    ex = KExpertsDense(D, ff, E)
    for p_ in ex.parameters():
        p_.data.copy_(rn(*p_.shape) * p_.shape[-1] ** -0.5)
    for T in (1, 8, 2048):
        x, w = rn(T, D), torch.rand(T, top, generator=g, device=dev)
        draw = lambda n: torch.stack([torch.randperm(n, generator=g, device=dev)[:top] for _ in range(T)])
        ids, all_ids = draw(40), draw(E)
        cost = lambda i: dict(nbytes=int(i[i < E].unique().numel()) * 3 * ff * D * 2) if T < 48 else dict(flops=float((i < E).sum()) * 3 * ff * D * 2)
        K.add("experts, a fifth of the choices identities (whole call)", f"T={T} top={top} of 32 + 8 width={D} ff={ff}", timed(lambda: ex(x, ids, w), flush), **cost(ids),
              peer=K.measure("experts, every choice an expert (whole call)", timed(lambda: ex(x, all_ids, w), flush), **cost(all_ids)))
    return K.rows


# family -> (sizes, kernel leg, the closest existing model: its family name in engine_leg and its sizes)
FAMILIES = {"mabidra": (MABIDRA_SIZES, mabidra_kernel_leg, "lekapel", SIZES), "zivulix": (ZIVULIX_SIZES, zivulix_kernel_leg, "mabidra-dense", ZIVULIX_SIZES),
            "bilurax": (BILURAX_SIZES, bilurax_kernel_leg, "mabidra-attn", BILURAX_SIZES), "rununex": (RUNUNEX_SIZES, rununex_kernel_leg, "mabidra-mixed", RUNUNEX_SIZES),
            "lipadra": (LIPADRA_SIZES, lipadra_kernel_leg, "mabidra-recurrent", LIPADRA_SIZES)}


def run_family(args, family):
    """one JSON line: the family's kernels, then per size the model and the closest existing model, in one process"""
    sizes, leg, closest, closest_sizes = FAMILIES[family]
    torch.cuda.set_device(0)
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        m = json.load(open(os.path.join(root, "MEASURED_PEAKS.json")))
        peak, tf, src = float(m["hbm_gbs"]), float(m["bf16_tflops"]), "measured (MEASURED_PEAKS.json hbm_gbs, bf16_tflops)"
    except Exception:
        peak, tf, src = 6650.0, 1590.0, "fallback"
    flush = Flusher("cuda")
    n0 = native.seq_lib().ktb200_launch_count()
    out = {"bench": family, "dtype": "bf16", "data": "synthetic (random weights and tokens)", "hbm_peak_GBps": peak, "bf16_peak_TFLOPs": tf, "peak_source": src,
           "timing": "CUDA events, median, 256 MB L2 flush between timed calls", "kernels": [] if getattr(args, "no_kernels", False) else leg(flush, peak, tf),
           "models": [], "closest_models": []}
    for name in (args.sizes.split(",") if getattr(args, "sizes", None) else sizes):
        out["models"].append(engine_leg(name, sizes[name], flush, args.steps, args.warmup, family=family))
        torch.cuda.empty_cache()
        out["closest_models"].append(engine_leg(name, closest_sizes[name], flush, args.steps, args.warmup, family=closest))
        torch.cuda.empty_cache()
    out["gpu_launches"] = int(native.seq_lib().ktb200_launch_count() - n0)
    print(json.dumps(out))


def run(args):
    """`bench.py --model lekapel | mabidra | zivulix | bilurax | rununex | lipadra`: prints one JSON line."""
    if args.model in FAMILIES:
        return run_family(args, args.model)
    torch.cuda.set_device(0)
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        peak, src = float(json.load(open(os.path.join(root, "MEASURED_PEAKS.json")))["hbm_gbs"]), "measured (MEASURED_PEAKS.json hbm_gbs)"
    except Exception:
        peak, src = 6650.0, "fallback"
    flush = Flusher("cuda")
    have_main = os.path.exists(native.LIB_PATH)
    n0 = native.seq_lib().ktb200_launch_count()
    out = {"bench": "lekapel", "dtype": "bf16", "data": "synthetic (random weights and tokens)", "hbm_peak_GBps": peak, "peak_source": src,
           "timing": "CUDA events, median, 256 MB L2 flush between timed calls", "kernels": kernel_leg(flush, peak, have_main), "models": []}
    for name in (args.sizes.split(",") if getattr(args, "sizes", None) else SIZES):
        out["models"].append(engine_leg(name, SIZES[name], flush, args.steps, args.warmup))
        torch.cuda.empty_cache()
    out["gpu_launches"] = int(native.seq_lib().ktb200_launch_count() - n0)
    print(json.dumps(out))
