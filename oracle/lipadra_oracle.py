"""TEST-ONLY plain restatement of the Lipadra decoder, one function per mechanism, float64 (or float32) torch on the CPU.

Nothing here is imported by the product path and nothing of the product path is imported here.  Every function works on one
sequence `[tokens, features]`; `Model.forward` runs a token range over explicit Python state (tensors of cached key and value rows, one
state matrix per head or channel, the last inputs of a short convolution), with no paging and no batching, token by token where a
recurrence is involved.

Notation: `T` tokens, `D` model width, `H` query heads, `G` key/value heads, `d` query/key size and `dv` value size per head, `C` the
chunk length of the attention mask, `I` channels of the selective scan, `N` their state size, `R` the rank of the step projection, `E`
experts with tensors, `J` identity experts, `n` the choices per token.
"""
from __future__ import annotations

import math

import torch

from .lekapel_oracle import read_safetensors  # noqa: F401  (the same file format)


def rms(x, eps):
    """x over its last axis divided by sqrt(mean(x^2) + eps)"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def short_conv(u, before, w, bias):
    """u [T, I], before [taps - 1, I] (the inputs just ahead of u, oldest first; zeros at a sequence's start), w [I, taps] whose last
    column meets the current token.  Returns (filtered rows + bias, the last taps - 1 inputs)."""
    taps = w.shape[1]
    rows = torch.cat([before, u], 0)
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * rows[t + j]
    return y + bias, rows[rows.shape[0] - (taps - 1):].clone()


def selective_scan(x, dt, A, B, Cm, D, S):
    """x and dt [T, I], A and S [I, N], B and Cm [T, N]:  S <- exp(dt A) S + (dt x) B ;  y = S C + D x.  Returns (y, the last S)."""
    S = S.clone()
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ Cm[t] + D * x[t]
    return y, S


def selective_scan_mixer(h, state, W, m):
    """h [T, D]; state = (S [I, N], the last taps - 1 convolution inputs)"""
    I, N, R = m["inner"], m["state"], m["dt_rank"]
    u = h @ W["in"].T
    x, z = u[:, :I], u[:, I:]
    x, tail = short_conv(x, state[1], W["conv"], W["conv.b"])
    x = silu(x)
    p = x @ W["x"].T
    dt = softplus(p[:, :R] @ W["dt"].T + W["dt.b"])
    y, S = selective_scan(x, dt, -torch.exp(W["A_log"]), p[:, R:R + N], p[:, R + N:], W["D"], state[0])
    return (y * silu(z)) @ W["o"].T, (S, tail)


def rotated_halves(x, pos, base, dims):
    """x [T, heads, n]: columns i and i + dims / 2 of every head turn together by pos * base^(-2 i / dims), i < dims / 2; the columns
    from `dims` on pass."""
    out = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = float(pos[t]) * float(base) ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def seen_keys(i, kpos, chunk):
    """indices of the keys that the query at position i sees: j <= i in the chunk of i"""
    return [n for n in range(len(kpos)) if int(kpos[n]) <= i and (chunk is None or int(kpos[n]) // chunk == i // chunk)]


def plus_one_attention(q, k, v, qpos, kpos, scale, chunk):
    """q [T, H, d], k [N, G, d], v [N, G, dv]; query head h reads key/value head h // (H / G).  Weights e^s / (1 + sum e^s)."""
    T, H, _ = q.shape
    G, dv = k.shape[1], v.shape[2]
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for t in range(T):
        i = int(qpos[t])
        seen = seen_keys(i, kpos, chunk)
        for h in range(H):
            g = h // (H // G)
            s = (k[seen, g] @ q[t, h]) * scale
            top = torch.clamp(s.max(), min=0.0)
            e = torch.exp(s - top)
            out[t, h] = (e / (e.sum() + torch.exp(-top))) @ v[seen, g]
    return out


def attention_mixer(h, pos, cache, W, m, eps):
    """h [T, D]; cache = (K [N, G, d], V [N, G, dv], positions [N]).  Biased projections; queries and keys to unit rms head by head times a
    weight of d numbers, then the rotation; the chunk mask; the plus-one soft-max."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = rms((h @ W["q"].T + W["q.b"]).reshape(T, H, d), eps) * W["q.norm"]
    k = rms((h @ W["k"].T + W["k.b"]).reshape(T, G, d), eps) * W["k.norm"]
    v = (h @ W["v"].T + W["v.b"]).reshape(T, G, dv)
    q, k = (rotated_halves(x, pos, m["rot"]["base"], m["rot"]["dims"]) for x in (q, k))
    K, V, P = torch.cat([cache[0], k]), torch.cat([cache[1], v]), torch.cat([cache[2], pos])
    o = plus_one_attention(q, K, V, pos, P, m["scale"], m["mask"]["size"])
    return o.reshape(T, H * dv) @ W["o"].T, (K, V, P)


def retention(q, k, v, decay, S):
    """q and k [T, H, d], v [T, H, dv], S [H, d, dv]:  S <- decay_h S + k v^T ;  o = S^T q.  Returns (o, the last S)."""
    S = S.clone()
    o = torch.zeros_like(v)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            S[h] = decay[h] * S[h] + torch.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def retention_mixer(h, pos, S, W, m, eps):
    """h [T, D]; S [H, d, dv]"""
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    rot = lambda n: rotated_halves((h @ W[n].T).reshape(T, H, d), pos, m["rot"]["base"], m["rot"]["dims"])
    o, S = retention(rot("q"), rot("k") * d ** -0.5, (h @ W["v"].T).reshape(T, H, dv), m["decay"], S)
    return (rms(o, eps).reshape(T, H * dv) * silu(h @ W["g"].T)) @ W["o"].T, S


def grouped_softmax_router(h, router, correction, top, groups, keep, scale):
    """(ids [T, n], weights [T, n]).  s = softmax(W h) over every output; the choice goes by s + correction among the outputs of the `keep`
    groups (of neighbours) whose largest choice score is largest; a weight is scale times s of the chosen one."""
    s = torch.softmax(h @ router.T, -1)
    c = s + correction
    E = router.shape[0]
    size = E // groups
    ids = torch.zeros(h.shape[0], top, dtype=torch.long)
    for t in range(h.shape[0]):
        best = sorted(range(groups), key=lambda g: (-float(c[t, g * size:(g + 1) * size].max()), g))[:keep]
        pool = [e for e in range(E) if e // size in best]
        ids[t] = torch.tensor(sorted(pool, key=lambda e: (-float(c[t, e]), e))[:top])
    return ids, scale * torch.gather(s, 1, ids)


def gated_expert(x, gate, up, down):
    return down @ (silu(gate @ x) * (up @ x))


def moe_mlp(h, W, f):
    """experts with tensors, then identity experts (whose output is their input); the shared expert times a sigmoid read from h"""
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    ids, wts = grouped_softmax_router(h, W["router"], W["correction"], r["top"], g["count"], g["keep"], r["scale"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            e = int(ids[t, j])
            y = gated_expert(h[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"]) if e < r["experts"] else h[t]
            out[t] += wts[t, j] * y
        if f.get("shared"):
            out[t] += torch.sigmoid(W["shared.sg"][0] @ h[t]) * gated_expert(h[t], W["shared.gate"], W["shared.up"], W["shared.down"])
    return out


class Model:
    def __init__(self, config, tensors, dtype=torch.float64):
        self.c, self.dtype = config, dtype
        self.W = {k: v.to(dtype) for k, v in tensors.items()}

    def sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.W.items() if k.startswith(prefix)}

    def owner(self, i):
        """the layer whose tensors layer i uses"""
        j = self.c["layers"][i].get("weights_of")
        return i if j is None else self.owner(j)

    def new_state(self):
        z = lambda *s: torch.zeros(*s, dtype=self.dtype)
        st = {"pos": 0, "layers": []}
        for l in self.c["layers"]:
            m = l["mixer"]
            if l["type"] == "attention":
                st["layers"].append((z(0, m["kv_heads"], m["dim"]), z(0, m["kv_heads"], m["vdim"]), torch.zeros(0, dtype=torch.long)))
            elif l["type"] == "retention":
                st["layers"].append(z(m["heads"], m["dim"], m["vdim"]))
            else:
                st["layers"].append((z(m["inner"], m["state"]), z(m["conv"] - 1, m["inner"])))
        return st

    def forward(self, tokens, state, trace=None):
        """logits [len(tokens), vocab] of the next tokens of ONE sequence; `state` is advanced"""
        c, W = self.c, self.W
        eps, alpha = c["norm"]["eps"], c["postln_alpha"]
        pos = torch.arange(state["pos"], state["pos"] + len(tokens))
        x = W["embed"][torch.tensor(tokens)]
        for i, l in enumerate(c["layers"]):
            p, m, st = f"l{self.owner(i)}.", l["mixer"], state["layers"]
            mix = self.sub(p + "mix.")
            if l["type"] == "attention":
                y, st[i] = attention_mixer(x, pos, st[i], mix, m, eps)
            elif l["type"] == "retention":
                y, st[i] = retention_mixer(x, pos, st[i], mix, m, eps)
            else:
                y, st[i] = selective_scan_mixer(x, st[i], mix, m)
            x = rms(alpha * x + y, eps) * W[p + "norm1"]
            if l["mlp"] is not None:
                x = rms(alpha * x + moe_mlp(x, self.sub(p + "mlp."), l["mlp"]), eps) * W[p + "norm2"]
            if trace is not None:
                trace.append(x.clone())
        state["pos"] += len(tokens)
        return rms(x, eps) * W["final.norm"] @ W["embed"].T
