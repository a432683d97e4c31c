"""Small random Rununex checkpoints for the tests: a config dict, a tensor dict in the checkpoint's naming, and a writer."""
import json
import os

import torch


def left(heads=4, kv_heads=2, dim=6, vdim=5, scale=None, chunk=7):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5, "mask": {"size": chunk}}


def right(heads=4, vdim=6, state=5, groups=2, conv=3, norm_groups=3):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def parallel(l=None, r=None, left_scale=0.6, right_scale=1.3):
    return {"type": "parallel", "mixer": {"left": l or left(), "right": r or right(), "left_scale": left_scale, "right_scale": right_scale}}


def diff(heads=4, kv_heads=2, dim=6, vdim=5, scale=None, chunk=9, conv=4, diff=0.3, dims=None, base=300.0, scaling=(4.0, 1.0, 4.0, 40)):
    """scaling: (factor, low, high, original) or None"""
    rot = {"base": base, "dims": dims if dims is not None else dim // 2 * 2}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5, "mask": {"size": chunk},
                                           "conv": conv, "diff": diff, "rot": rot}}


def moe(ff=10, experts=6, top=2, shared=14):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}


def config(layers, vocab=50, width=24, eps=1e-5, embed_scale=3.0, residual_mult=0.8, logit_scale=0.6):
    """layers: [(mixer description from parallel() / diff(), feed-forward from moe() or None)]"""
    return {"architecture": "Rununex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "residual_mult": residual_mult,
            "logit_scale": logit_scale, "layers": [{"type": m["type"], "mixer": m["mixer"], "mlp": f} for m, f in layers]}


def left_weights(rn, lin, p, m, D):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {p + "q": lin(H * d, D, 2.0), p + "k": lin(G * d, D, 2.0), p + "v": lin(G * dv, D), p + "g": lin(H * dv, D, 1.5), p + "o": lin(D, H * dv),
            p + "r1": 0.4 + 0.4 * rn(H).abs(), p + "r2": 0.05 + 0.5 * rn(H).abs(), p + "sink": rn(H, k=0.7)}


def right_weights(rn, lin, p, m, D):
    P, dv, N, J, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    inner, C = P * dv, P * dv + 2 * J * N
    return {p + "in": lin(inner + C + P, D, 1.5), p + "conv": rn(C, taps, k=0.6), p + "conv.b": rn(C, k=0.3), p + "dt_bias": rn(P) - 1.0, p + "A_log": rn(P, k=0.7), p + "D": rn(P),
            p + "norm": 1.0 + 0.3 * rn(inner), p + "o": lin(D, inner)}


def diff_weights(rn, lin, p, m, D):
    H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    w = {p + "q": lin(2 * H * d, D, 2.0), p + "k": lin(2 * G * d, D, 2.0), p + "v": lin(G * dv, D), p + "o": lin(D, H * dv)}
    for n, c in (("q", 2 * H * d), ("k", 2 * G * d), ("v", G * dv)):
        w[p + n + ".conv"] = rn(c, taps, k=0.6)
    for n in ("lq1", "lk1", "lq2", "lk2"):
        w[p + n] = rn(d, k=0.4 / d ** 0.25)
    return w


def weights(cfg, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    D = cfg["width"]
    rn = lambda *s, k=1.0: torch.randn(*s, generator=g) * k
    lin = lambda o, i, s=1.0: rn(o, i, k=s / i ** 0.5)
    nw = lambda n: 1.0 + 0.3 * rn(n)
    w = {"embed": rn(cfg["vocab"], D, k=0.5), "final.norm": nw(D), "head": lin(cfg["vocab"], D, 2.0)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        w[p + "norm1"] = nw(D)
        if l["type"] == "parallel":
            w.update(left_weights(rn, lin, p + "mix.left.", m["left"], D))
            w.update(right_weights(rn, lin, p + "mix.right.", m["right"], D))
        else:
            w.update(diff_weights(rn, lin, p + "mix.", m, D))
        f = l["mlp"]
        if f is None:
            continue
        w[p + "norm2"] = nw(D)
        E, ff, sf = f["router"]["experts"], f["expert"]["ff"], f["shared"]["ff"]
        w[p + "mlp.router"] = lin(E, D, 3.0)
        for e, n in [(f"e{e}", ff) for e in range(E)] + [("shared", sf)]:
            w[p + f"mlp.{e}.gate"], w[p + f"mlp.{e}.up"], w[p + f"mlp.{e}.down"] = lin(n, D, 2.0), lin(n, D, 2.0), lin(D, n)
    return {k: v.to(dtype).contiguous() for k, v in w.items()}


def save(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(w, os.path.join(path, "model.safetensors"))
    return str(path)
