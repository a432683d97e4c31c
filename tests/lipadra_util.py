"""Small random Lipadra checkpoints for the tests: a config dict, a tensor dict in the checkpoint's naming, and a writer."""
import json
import os

import torch


def attention(heads=4, kv_heads=2, dim=6, vdim=5, scale=None, chunk=7, dims=4, base=300.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5, "mask": {"size": chunk}, "rot": {"base": base, "dims": dims}}
    return {"type": "attention", "mixer": m}


def retention(heads=3, dim=6, vdim=5, decay=None, dims=None, base=500.0):
    if decay is None:
        decay = [1.0 - 0.3 / (1.0 + 2.7 * i) for i in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": dims if dims is not None else dim // 2 * 2}}}


def scan(inner=14, state=5, dt_rank=3, conv=4):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}


def moe(ff=10, experts=7, identity=2, top=2, groups=(3, 1), scale=1.7, shared=14):
    """(groups go by their largest score: they only bear on the choice when more outputs are chosen than groups are kept)"""
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups[0], "keep": groups[1]}, "scale": scale},
            "shared": {"ff": shared} if shared else None}


def config(layers, vocab=50, width=24, eps=1e-5, alpha=5.0):
    """layers: (mixer description, feed-forward from moe() or None), or the index of the layer whose tensors (and description) are used again"""
    out = []
    for l in layers:
        if isinstance(l, int):
            out.append(dict(out[l], weights_of=l))
        else:
            out.append({"type": l[0]["type"], "mixer": l[0]["mixer"], "mlp": l[1]})
    return {"architecture": "Lipadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": out}


def attention_weights(rn, lin, p, m, D):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {p + "q": lin(H * d, D, 2.0), p + "k": lin(G * d, D, 2.0), p + "v": lin(G * dv, D), p + "o": lin(D, H * dv), p + "q.b": rn(H * d, k=0.3), p + "k.b": rn(G * d, k=0.3),
            p + "v.b": rn(G * dv, k=0.3), p + "q.norm": 1.3 + 0.4 * rn(d), p + "k.norm": 1.1 + 0.4 * rn(d)}


def retention_weights(rn, lin, p, m, D):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    return {p + "q": lin(H * d, D, 1.5), p + "k": lin(H * d, D, 1.5), p + "v": lin(H * dv, D), p + "g": lin(H * dv, D, 1.5), p + "o": lin(D, H * dv)}


def scan_weights(rn, lin, p, m, D):
    I, N, R, taps = m["inner"], m["state"], m["dt_rank"], m["conv"]
    return {p + "in": lin(2 * I, D, 1.5), p + "conv": rn(I, taps, k=0.6), p + "conv.b": rn(I, k=0.3), p + "x": lin(R + 2 * N, I, 1.5), p + "dt": lin(I, R, 1.0), p + "dt.b": rn(I) - 1.0,
            p + "A_log": rn(I, N, k=0.8), p + "D": rn(I), p + "o": lin(D, I)}


WEIGHTS = {"attention": attention_weights, "retention": retention_weights, "mamba1": scan_weights}


def moe_weights(rn, lin, p, f, D):
    r = f["router"]
    n = r["experts"] + r["identity"]
    w = {p + "router": lin(n, D, 1.5), p + "correction": rn(n, k=0.5 / n) - 0.4}      # negative choice scores are common
    parts = [(f"e{e}", f["expert"]["ff"]) for e in range(r["experts"])]
    if f["shared"]:
        parts.append(("shared", f["shared"]["ff"]))
        w[p + "shared.sg"] = lin(1, D, 2.0)
    for e, n in parts:
        w[p + e + ".gate"], w[p + e + ".up"], w[p + e + ".down"] = lin(n, D, 1.5), lin(n, D, 1.5), lin(D, n)
    return w


def weights(cfg, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    D = cfg["width"]
    rn = lambda *s, k=1.0: torch.randn(*s, generator=g) * k
    lin = lambda o, i, s=1.0: rn(o, i, k=s / i ** 0.5)
    nw = lambda n: 1.0 + 0.3 * rn(n)
    w = {"embed": rn(cfg["vocab"], D), "final.norm": nw(D)}
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p = f"l{i}."
        w[p + "norm1"] = nw(D)
        w.update(WEIGHTS[l["type"]](rn, lin, p + "mix.", l["mixer"], D))
        if l["mlp"] is not None:
            w[p + "norm2"] = nw(D)
            w.update(moe_weights(rn, lin, p + "mlp.", l["mlp"], D))
    return {k: v.to(dtype).contiguous() for k, v in w.items()}


def save(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(w, os.path.join(path, "model.safetensors"))
    return str(path)
