"""TEST-ONLY plain restatement of the Rununex decoder, one function per mechanism, float64 (or float32) torch on the CPU.

Nothing here is imported by the product path and nothing of the product path is imported here.  Every function works on one
sequence `[tokens, features]`; `Model.forward` runs a token range over explicit Python state (tensors of cached key and value rows, one
state matrix per head, the last inputs of every short convolution), with no paging and no batching, token by token where a recurrence
is involved.

Notation: `T` tokens, `D` model width, `H` query heads, `G` key/value heads, `d` query/key size and `dv` value size per head (of one
map), `C` the chunk length of an attention mask, `P` state-space heads of `dv` channels, `N` their state size, `J` their groups,
`E` experts, `n` the experts a token uses.
"""
from __future__ import annotations

import math

import torch

from .lekapel_oracle import read_safetensors  # noqa: F401  (the same file format)


def layer_norm(x, w, eps):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * w over the last axis"""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
    """x over its last axis divided by sqrt(mean(x^2) + eps)"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def short_conv(u, before, w, bias=None):
    """u [T, channels], before [taps - 1, channels] (the inputs just ahead of u, oldest first; zeros at a sequence's start), w [channels,
    taps] whose last column meets the current token.  Returns (filtered rows, the last taps - 1 inputs)."""
    taps = w.shape[1]
    rows = torch.cat([before, u], 0)
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * rows[t + j]
    if bias is not None:
        y = y + bias
    return y, rows[rows.shape[0] - (taps - 1):].clone()


def scaled_frequencies(base, dims, scaling=None):
    """base^(-2 i / dims) for i < dims / 2; with `scaling` = {factor, low, high, original}: slow turns (wavelength above original / low) are
    divided by factor, fast ones (below original / high) kept, and those between interpolated linearly in original / wavelength."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            length = 2.0 * math.pi / f
            if length > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif length >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate_interleaved(x, pos, freqs):
    """x [T, heads, n]: columns 2 i and 2 i + 1 of every head turn together by the angle pos * freqs[i]; the columns behind them pass."""
    out = x.clone()
    for t in range(x.shape[0]):
        for i, f in enumerate(freqs):
            a = float(pos[t]) * f
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            out[t, :, 2 * i] = u * c - v * s
            out[t, :, 2 * i + 1] = v * c + u * s
    return out


def seen_keys(i, kpos, chunk):
    """indices of the keys that the query at position i sees: j <= i in the chunk of i"""
    return [n for n in range(len(kpos)) if int(kpos[n]) <= i and (chunk is None or int(kpos[n]) // chunk == i // chunk)]


def softmax_attention(q, k, v, qpos, kpos, scale, chunk, r1=None, r2=None, sink=None):
    """q [T, H, d], k [N, G, d], v [N, G, dv]; query head h reads key/value head h // (H / G).  score = scale q.k, less
    r1_h ln(1 + r2_h (i - j)) when r1, r2 are given; with `sink` the denominator also counts exp(sink_h), which has no value."""
    T, H, _ = q.shape
    G, dv = k.shape[1], v.shape[2]
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for t in range(T):
        i = int(qpos[t])
        seen = seen_keys(i, kpos, chunk)
        for h in range(H):
            g = h // (H // G)
            s = (k[seen, g] @ q[t, h]) * scale
            if r1 is not None:
                dist = (i - kpos[seen]).to(q.dtype)
                s = s - r1[h] * torch.log(1.0 + r2[h] * dist)
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            den = e.sum() if sink is None else e.sum() + torch.exp(sink[h] - top)
            out[t, h] = (e / den) @ v[seen, g]
    return out


def biased_sink_mixer(h, pos, cache, W, m, eps):
    """h [T, D]; cache = (K [N, G, d], V [N, G, dv], positions [N]).  Unit-rms queries and keys head by head (no weight), no rotation, the
    logarithmic distance bias, the chunk mask, the sink, an element-wise sigmoid output gate read from h."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = rms((h @ W["q"].T).reshape(T, H, d), eps)
    k = rms((h @ W["k"].T).reshape(T, G, d), eps)
    v = (h @ W["v"].T).reshape(T, G, dv)
    K, V, P = torch.cat([cache[0], k]), torch.cat([cache[1], v]), torch.cat([cache[2], pos])
    o = softmax_attention(q, K, V, pos, P, m["scale"], m["mask"]["size"], W["r1"], W["r2"], W["sink"])
    o = o.reshape(T, H * dv) * torch.sigmoid(h @ W["g"].T)
    return o @ W["o"].T, (K, V, P)


def state_space_scan(x, B, Cm, dt, a_log, D, S):
    """x [T, P, dv], B and Cm [T, J, N], dt [T, P] (positive), S [P, N, dv].  Head p uses group p // (P / J):
    S <- exp(-exp(a_log_p) dt) S + dt B x^T ;  y = S^T C + D_p x.  Returns (y, the last S)."""
    T, P, _ = x.shape
    J = B.shape[1]
    S = S.clone()
    y = torch.zeros_like(x)
    for t in range(T):
        for p in range(P):
            j = p // (P // J)
            S[p] = torch.exp(-torch.exp(a_log[p]) * dt[t, p]) * S[p] + dt[t, p] * torch.outer(B[t, j], x[t, p])
            y[t, p] = S[p].T @ Cm[t, j] + D[p] * x[t, p]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    """u = y silu(z) is cut into `groups` equal parts, each part scaled to unit rms, and the row multiplied by w"""
    T, n = y.shape
    u = (y * silu(z)).reshape(T, groups, n // groups)
    return rms(u, eps).reshape(T, n) * w


def state_space_mixer(h, state, W, m, eps):
    """h [T, D]; state = (S [P, N, dv], the last taps - 1 convolution inputs).  W['in'] makes [z | x | B | C | dt]."""
    P, dv, N, J = m["heads"], m["vdim"], m["state"], m["groups"]
    T, inner = h.shape[0], m["heads"] * m["vdim"]
    u = h @ W["in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * J * N], u[:, 2 * inner + 2 * J * N:]
    c, tail = short_conv(xbc, state[1], W["conv"], W["conv.b"])
    c = silu(c)
    x, B, Cm = c[:, :inner].reshape(T, P, dv), c[:, inner:inner + J * N].reshape(T, J, N), c[:, inner + J * N:].reshape(T, J, N)
    dt = torch.log1p(torch.exp(dt + W["dt_bias"]))
    y, S = state_space_scan(x, B, Cm, dt, W["A_log"], W["D"], state[0])
    return gated_group_norm(y.reshape(T, inner), z, W["norm"], m["norm_groups"], eps) @ W["o"].T, (S, tail)


def parallel_mixer(h, pos, state, W, m, eps):
    """left_scale * attention + right_scale * state space, both of the same h; state = {'kv', 'ssm'}"""
    part = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    left, kv = biased_sink_mixer(h, pos, state["kv"], part("left."), m["left"], eps)
    right, ssm = state_space_mixer(h, state["ssm"], part("right."), m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right, {"kv": kv, "ssm": ssm}


def difference_strength(W, diff):
    """the one number by which the second map's output is taken off the first's"""
    return torch.exp((W["lq1"] * W["lk1"]).sum()) - torch.exp((W["lq2"] * W["lk2"]).sum()) + diff


def differential_mixer(h, pos, state, W, m, eps):
    """h [T, D]; state = {'kv': (K [N, 2 G, d], V, positions), 'conv': {'q', 'k', 'v'}}.  Every head has two maps (rows [map 1, map 2] head by
    head), each a soft-max attention of its own over the same values: o = unit rms of (a1 - lambda a2), times 1 - diff."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, conv, u = h.shape[0], {}, {}
    for n in "qkv":
        u[n], conv[n] = short_conv(h @ W[n].T, state["conv"][n], W[n + ".conv"])
    freqs = scaled_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
    q = rotate_interleaved(u["q"].reshape(T, 2 * H, d), pos, freqs).reshape(T, H, 2, d)
    k = rotate_interleaved(u["k"].reshape(T, 2 * G, d), pos, freqs)
    v = u["v"].reshape(T, G, dv)
    K, V, P = torch.cat([state["kv"][0], k]), torch.cat([state["kv"][1], v]), torch.cat([state["kv"][2], pos])
    Km = K.reshape(-1, G, 2, d)
    a = [softmax_attention(q[:, :, i], Km[:, :, i], V, pos, P, m["scale"], m["mask"]["size"]) for i in (0, 1)]
    o = rms(a[0] - difference_strength(W, m["diff"]) * a[1], eps) * (1.0 - m["diff"])
    return o.reshape(T, H * dv) @ W["o"].T, {"kv": (K, V, P), "conv": conv}


def sigmoid_router(h, router, top):
    """(ids [T, n], weights [T, n]): the n largest of sigmoid(W h), which are also the weights as they are"""
    s = torch.sigmoid(h @ router.T)
    ids = torch.zeros(h.shape[0], top, dtype=torch.long)
    for t in range(h.shape[0]):
        ids[t] = torch.tensor(sorted(range(router.shape[0]), key=lambda e: (-float(s[t, e]), e))[:top])
    return ids, torch.gather(s, 1, ids)


def gated_expert(x, gate, up, down):
    return down @ (silu(gate @ x) * (up @ x))


def moe_mlp(h, W, f):
    """an expert sees its weight times h, and its output counts as it is; the shared expert sees h"""
    ids, wts = sigmoid_router(h, W["router"], f["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        out[t] = gated_expert(h[t], W["shared.gate"], W["shared.up"], W["shared.down"])
        for j in range(ids.shape[1]):
            e = int(ids[t, j])
            out[t] += gated_expert(wts[t, j] * h[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"])
    return out


class Model:
    def __init__(self, config, tensors, dtype=torch.float64):
        self.c, self.dtype = config, dtype
        self.W = {k: v.to(dtype) for k, v in tensors.items()}

    def sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.W.items() if k.startswith(prefix)}

    def new_state(self):
        z = lambda *s: torch.zeros(*s, dtype=self.dtype)
        st = {"pos": 0, "layers": []}
        for l in self.c["layers"]:
            m = l["mixer"]
            if l["type"] == "parallel":
                a, r = m["left"], m["right"]
                inner = r["heads"] * r["vdim"]
                st["layers"].append({"kv": (z(0, a["kv_heads"], a["dim"]), z(0, a["kv_heads"], a["vdim"]), torch.zeros(0, dtype=torch.long)),
                                     "ssm": (z(r["heads"], r["state"], r["vdim"]), z(r["conv"] - 1, inner + 2 * r["groups"] * r["state"]))})
            else:
                G, b = m["kv_heads"], m["conv"] - 1
                st["layers"].append({"kv": (z(0, 2 * G, m["dim"]), z(0, G, m["vdim"]), torch.zeros(0, dtype=torch.long)),
                                     "conv": {"q": z(b, m["heads"] * 2 * m["dim"]), "k": z(b, G * 2 * m["dim"]), "v": z(b, G * m["vdim"])}})
        return st

    def forward(self, tokens, state, trace=None):
        """logits [len(tokens), vocab] of the next tokens of ONE sequence; `state` is advanced"""
        c, W = self.c, self.W
        eps, mult = c["norm"]["eps"], c["residual_mult"]
        pos = torch.arange(state["pos"], state["pos"] + len(tokens))
        x = W["embed"][torch.tensor(tokens)] * c["embedding"]["scale"]
        for i, l in enumerate(c["layers"]):
            p = f"l{i}."
            mixer = {"parallel": parallel_mixer, "attention": differential_mixer}[l["type"]]
            y, state["layers"][i] = mixer(layer_norm(x, W[p + "norm1"], eps), pos, state["layers"][i], self.sub(p + "mix."), l["mixer"], eps)
            x = x + mult * y
            if l["mlp"] is not None:
                x = x + mult * moe_mlp(layer_norm(x, W[p + "norm2"], eps), self.sub(p + "mlp."), l["mlp"])
            if trace is not None:
                trace.append(x.clone())
        state["pos"] += len(tokens)
        return layer_norm(x, W["final.norm"], eps) @ W["head"].T * c["logit_scale"]
