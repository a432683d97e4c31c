"""Rununex through the framework (registry, loader, paged state cache, scheduler, engine, CUDA operators) against the plain
restatement in oracle/rununex_oracle.py, on small random checkpoints made here.  CPU tests cover the host logic."""
import json
import math
import random

import pytest
import torch

import rununex_util as U
from oracle import rununex_oracle as O

gpu = pytest.mark.gpu
F32_TOL, BF16_TOL = 3e-4, 6e-2


def rel(a, b):
    a, b = a.detach().double().cpu(), b.detach().double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


def rel_rows(a, b, q=0.8):
    """the q-quantile of the per-row errors, for bf16 runs of whole models"""
    a, b = a.detach().double().cpu(), b.detach().double().cpu()
    return float(((a - b).abs().amax(-1) / b.abs().max()).quantile(q))


class DictLoader:
    def __init__(self, w):
        self.w = w

    def load_tensor(self, key, device="cpu"):
        return self.w[key].to(device)


def part(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


MIXED = [(U.parallel(), U.moe()), (U.diff(), U.moe(ff=7, experts=9, top=1, shared=5)), (U.parallel(U.left(heads=6, kv_heads=1, dim=4, vdim=7, chunk=16), U.right(heads=6, vdim=5, state=8, groups=1, conv=2, norm_groups=1), 1.0, 0.7), None),
         (U.diff(heads=3, kv_heads=3, dim=4, vdim=6, chunk=5, conv=2, diff=0.6, dims=2, scaling=None), U.moe(ff=12, experts=4, top=3, shared=9))]


def serve(tmp_path, cfg, dtype, seed=0, **engine_kw):
    from ktransformers_b200.models import load_model
    from ktransformers_b200.util.engine import Engine
    w = U.weights(cfg, seed, torch.bfloat16 if dtype == "bfloat16" else torch.float32)
    path = U.save(tmp_path / f"ckpt{seed}", cfg, w)
    torch.backends.cuda.matmul.allow_tf32 = False
    model = load_model(path, dtype)
    return Engine(model, **engine_kw), O.Model(cfg, w, torch.float64)


def oracle_logits(om, tokens):
    return om.forward(tokens, om.new_state()).float()


def run_steps(eng, steps):
    """steps: list of lists of (id, tokens, last); every position's logits are asked for; returns {id: [n, V]}"""
    out = {}
    for step in steps:
        lg = eng.step([(i, t, list(range(len(t)))) for i, t, _ in step], [i for i, _, last in step if last]).cpu()
        k = 0
        for i, t, _ in step:
            out.setdefault(i, []).append(lg[k:k + len(t)])
            k += len(t)
    return {i: torch.cat(v) for i, v in out.items()}


def cut(seq_id, tokens, sizes):
    """portions of the given sizes (repeating the last) as single-entry steps"""
    steps, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(k, len(sizes) - 1)], len(tokens) - at)
        steps.append([(seq_id, tokens[at:at + n], at + n == len(tokens))])
        at, k = at + n, k + 1
    return steps


def toks(n, vocab=50, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# ------------------------------------------------------------------------------------------------ host logic (CPU)
def test_config_reads_sizes_and_constants_per_layer():
    from ktransformers_b200.models.configuration_rununex import RununexConfig
    cfg = U.config(MIXED, vocab=77, width=40, eps=2e-4, embed_scale=5.5, residual_mult=0.25, logit_scale=1.75)
    c = RununexConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.norm_eps, c.embedding_scale, c.residual_mult, c.logit_scale) == (77, 40, 2e-4, 5.5, 0.25, 1.75)
    p, a = c.layers[0].mixer, c.layers[3].mixer
    assert (p.left.heads, p.left.kv_heads, p.left.dim, p.left.vdim, p.left.chunk, p.left_scale, p.right_scale) == (4, 2, 6, 5, 7, 0.6, 1.3)
    assert (p.right.heads, p.right.vdim, p.right.state_size, p.right.groups, p.right.conv, p.right.norm_groups, p.right.inner, p.right.channels) == (4, 6, 5, 2, 3, 3, 24, 44)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.conv, a.diff, a.rot.dims, a.rot.original) == (3, 3, 4, 6, 5, 2, 0.6, 2, None)
    b = c.layers[1].mixer.rot
    assert (b.base, b.factor, b.low, b.high, b.original, b.layout) == (300.0, 4.0, 1.0, 4.0, 40.0, "interleaved")
    f = c.layers[1].mlp
    assert (f.ff, f.experts, f.top, f.shared_ff) == (7, 9, 1, 5) and c.layers[2].mlp is None
    assert c.cache_row_widths() == [2 * 11, 2 * 17, 1 * 11, 3 * 14] and c.chunks() == [7, 9, 16, 5]
    assert c.state_widths() == [24 * 5 + 2 * 44, 3 * (8 * 6 + 4 * 6 + 2 * 5), 30 * 8 + 1 * 46, 1 * (6 * 4 + 6 * 4 + 3 * 6)]
    with pytest.raises(ValueError):
        RununexConfig.from_dict(dict(cfg, layers=[dict(cfg["layers"][0], type="conv")]))
    with pytest.raises(ValueError):
        RununexConfig.from_dict(dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "dense", "ff": 3})]))


def test_registry_picks_the_class_by_config():
    from ktransformers_b200.models import architecture_of, model_class
    assert model_class(architecture_of(U.config(MIXED))).__name__ == "RununexForCausalLM"


@pytest.mark.parametrize("base,dims,scaling", [(300.0, 12, (4.0, 1.0, 4.0, 40)), (10000.0, 64, (8.0, 1.5, 5.0, 700)), (50.0, 6, (3.0, 0.5, 2.0, 20)), (777.0, 10, None)])
def test_scaled_rotation_frequencies(base, dims, scaling):
    from ktransformers_b200.models.configuration_rununex import _rotary
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    got = _rotary(rot, dims).inv_freq("cpu")
    want = torch.tensor(O.scaled_frequencies(base, dims, rot.get("scaling")), dtype=torch.float64)
    assert rel(got, want) < 1e-12
    if scaling:      # kept, mixed and divided frequencies all occur
        plain = torch.tensor(O.scaled_frequencies(base, dims), dtype=torch.float64)
        ratio = plain / want
        assert (ratio < 1 + 1e-9).any() and (ratio > scaling[0] - 1e-9).any() and ((ratio > 1 + 1e-6) & (ratio < scaling[0] - 1e-6)).any()


def test_oracle_portions_equal_whole_prompt_and_the_attention_is_what_it_says():
    cfg = U.config(MIXED)
    om = O.Model(cfg, U.weights(cfg, 3, torch.float32))
    t = toks(23, seed=1)
    whole = om.forward(t, om.new_state())
    st = om.new_state()
    parts = torch.cat([om.forward(t[a:b], st) for a, b in ((0, 6), (6, 7), (7, 9), (9, 23))])
    assert rel(parts, whole) < 1e-9
    # bias, sink and chunk against a matrix form
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(11, 4, 3, generator=g).double(), torch.randn(11, 2, 3, generator=g).double(), torch.randn(11, 2, 2, generator=g).double()
    r1, r2, sink, pos = torch.rand(4, generator=g).double(), torch.rand(4, generator=g).double(), torch.randn(4, generator=g).double(), torch.arange(11)
    got = O.softmax_attention(q, k, v, pos, pos, 0.7, 4, r1, r2, sink)
    dist = (pos[:, None] - pos[None, :]).clamp_min(0).double()
    s = torch.einsum("thd,nhd->htn", q, k.repeat_interleave(2, 1)) * 0.7 - r1[:, None, None] * torch.log1p(r2[:, None, None] * dist)
    ok = (pos[None, :] <= pos[:, None]) & (pos[None, :] // 4 == pos[:, None] // 4)
    e = torch.exp(s) * ok
    want = torch.einsum("htn,nhv->thv", e / (e.sum(-1, keepdim=True) + torch.exp(sink)[:, None, None]), v.repeat_interleave(2, 1))
    assert rel(got, want) < 1e-12


def test_oracle_state_space_against_the_closed_form():
    """y_t = sum_s<=t exp(sum of log decays in (s, t]) dt_s (C_t . B_s) x_s + D x_t"""
    g = torch.Generator().manual_seed(1)
    T, P, J, N, dv = 9, 4, 2, 3, 2
    x, B, C = torch.randn(T, P, dv, generator=g).double(), torch.randn(T, J, N, generator=g).double(), torch.randn(T, J, N, generator=g).double()
    dt, al, D = torch.rand(T, P, generator=g).double(), torch.randn(P, generator=g).double(), torch.randn(P, generator=g).double()
    y, _ = O.state_space_scan(x, B, C, dt, al, D, torch.zeros(P, N, dv).double())
    la = torch.cumsum(-torch.exp(al) * dt, 0)
    for t in range(T):
        for p in range(P):
            want = D[p] * x[t, p] + sum(math.exp(la[t, p] - la[s, p]) * dt[s, p] * (C[t, p // 2] @ B[s, p // 2]) * x[s, p] for s in range(t + 1))
            assert rel(y[t, p], want) < 1e-10


# ------------------------------------------------------------------------------------------------ mechanisms alone (GPU)
@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("width,n", [(20, 5), (35, 7), (6, 3), (256, 9), (1024, 300), (7168, 3), (9000, 2), (12288, 301)])
def test_layer_norm_with_scaled_sum_and_row_pick(dtype, tol, width, n):
    from ktransformers_b200.operators.norm import KLayerNorm
    g = torch.Generator().manual_seed(width)
    x, a, b = torch.randn(n, width, generator=g) + 3.0, torch.randn(n, width, generator=g), torch.randn(n, width, generator=g).to(dtype)
    w = (1 + 0.3 * torch.randn(width, generator=g)).to(dtype)
    op = KLayerNorm(width, 1e-3, dtype=dtype)
    op.load(DictLoader({"n": w}), "n")
    xs = x.double() + 0.7 * (a.double() + b.double())
    x_out, h = op(x.cuda(), a.cuda(), b.cuda(), 0.7)
    assert rel(x_out, xs) < 1e-6 and rel(h, O.layer_norm(xs, w.double(), 1e-3)) < tol
    # picked rows, no kept sum, a constant on the normed row
    rows = torch.tensor([n - 1, 0, 1, 0])
    none, h = op(x.cuda(), None, b.cuda(), 0.7, rows=rows.cuda(), keep_x=False, h_scale=0.3)
    assert none is None and rel(h, 0.3 * O.layer_norm((x.double() + 0.7 * b.double())[rows], w.double(), 1e-3)) < tol
    # an embedding lookup: no residual yet; the sum alone
    x_out, h = op(None, b.cuda(), mult=4.5, rows=rows.cuda())
    assert rel(x_out, 4.5 * b.double()[rows]) < 1e-6 and rel(h, O.layer_norm(4.5 * b.double()[rows], w.double(), 1e-3)) < tol
    assert rel(op(x.cuda(), a.cuda(), None, 0.7, want_h=False)[0], x.double() + 0.7 * a.double()) < 1e-6
    # nothing to add: the stream itself comes back, and a norm that kept the mean would differ
    x0, h = op(x.cuda())
    assert rel(x0, x) == 0.0 and rel(h, O.layer_norm(x.double(), w.double(), 1e-3)) < tol
    assert rel(O.rms(x.double(), 1e-3) * w.double(), O.layer_norm(x.double(), w.double(), 1e-3)) > 0.1


@gpu
@pytest.mark.parametrize("experts,top", [(6, 2), (12, 1), (5, 5), (64, 8), (600, 3), (40, 33)])
@pytest.mark.parametrize("width,n", [(24, 7), (24, 130), (30, 5)])
def test_plain_sigmoid_router(experts, top, width, n):
    """decode-sized batches (one launch), prompt-sized ones (GEMM + selection), a width the GEMV kernel does not take, more experts or
    choices than the kernel selects from"""
    from ktransformers_b200.operators.gate import KSigmoidTopKGate
    g = torch.Generator().manual_seed(n + experts)
    W, x = torch.randn(experts, width, generator=g) * 0.6, torch.randn(n, width, generator=g)
    op = KSigmoidTopKGate(width, experts, top)
    op.load(DictLoader({"r": W}), "r")
    ids, wts = op(x.cuda())
    want_ids, want_w = O.sigmoid_router(x.double(), W.double(), top)
    assert ids.cpu().tolist() == want_ids.tolist() and rel(wts, want_w) < 1e-5


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("n,path", [(1, "pair"), (5, "pair"), (3, "expert"), (9, "expert"), (70, "grouped")])
def test_experts_weighted_on_their_input_on_every_path(dtype, tol, n, path):
    from ktransformers_b200.operators.experts import KExpertsDense
    g = torch.Generator().manual_seed(n)
    for width, ff, E, top in ((24, 16, 6, 2), (40, 9, 5, 3), (32, 8, 4, 1)):
        W = {}
        for e in range(E):
            W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"] = [(torch.randn(*s, generator=g) * k).to(dtype) for s, k in (((ff, width), 0.5), ((ff, width), 0.5), ((width, ff), 0.3))]
        op = KExpertsDense(width, ff, E, dtype=dtype)
        op.load(DictLoader(W), "")
        if path == "pair":
            op.by_expert_min_tokens = 10 ** 9
        x = torch.randn(n, width, generator=g).to(dtype)
        ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(n)])
        wts = 0.2 + 0.6 * torch.rand(n, top, generator=g)
        got = op(x.cuda(), ids.cuda(), wts.cuda(), on_input=True)
        Wd = {k: v.double() for k, v in W.items()}
        one = lambda t, j, w: O.gated_expert(w * x[t].double(), Wd[f"e{int(ids[t, j])}.gate"], Wd[f"e{int(ids[t, j])}.up"], Wd[f"e{int(ids[t, j])}.down"])
        want = torch.stack([sum(one(t, j, wts[t, j].double()) for j in range(top)) for t in range(n)])
        assert rel(got, want) < tol
        outside = torch.stack([sum(wts[t, j].double() * one(t, j, 1.0) for j in range(top)) for t in range(n)])
        assert rel(outside, want) > 0.1                                   # a weight on the output is another function
        assert rel(op(x.cuda(), ids.cuda(), wts.cuda()), outside) < tol


@gpu
@pytest.mark.parametrize("n", [3, 60])
def test_mixture_with_shared_expert(n):
    from ktransformers_b200.operators.experts import KSharedSigmoidMoE
    cfg = U.config([(U.diff(), U.moe(ff=11, experts=7, top=2, shared=19))], width=28)
    W = part(U.weights(cfg, 4, torch.float32), "l0.mlp.")
    op = KSharedSigmoidMoE(28, 11, 7, 2, 19, dtype=torch.float32)
    op.load(DictLoader(W), "")
    h = torch.randn(n, 28, generator=torch.Generator().manual_seed(0))
    routed, shared = op(h.cuda())
    want = O.moe_mlp(h.double(), {k: v.double() for k, v in W.items()}, cfg["layers"][0]["mlp"])
    assert rel(routed + shared, want) < 2e-5


def mixer_alone(desc, dtype, n, page_size, portions, seed=4, width=24, tweak=None, tensor_path=True):
    """one mixer ("left", "right" or "attention") over one sequence cut into `portions` (the last size repeats), against the restatement over
    the whole sequence"""
    from ktransformers_b200.models import configuration_rununex as cfgs
    from ktransformers_b200.models.custom_cache import PagedStateCache
    from ktransformers_b200.operators.attention import KBiasedSinkAttention, KDifferentialAttention
    from ktransformers_b200.operators.linear_attention import KStateSpace
    kind, m = desc
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s, k=1.0: torch.randn(*s, generator=g) * k
    lin = lambda o, i, s=1.0: rn(o, i, k=s / i ** 0.5)
    make, spec_cls, op_cls = {"left": (U.left_weights, cfgs.BiasedSinkAttentionSpec, KBiasedSinkAttention), "right": (U.right_weights, cfgs.StateSpaceSpec, KStateSpace),
                              "attention": (U.diff_weights, cfgs.DifferentialAttentionSpec, KDifferentialAttention)}[kind]
    W = make(rn, lin, "", m, width)
    h = rn(n, width)
    if tweak:
        tweak(W, h, m)
    W, h = {k: v.to(dtype) for k, v in W.items()}, h.to(dtype)
    spec = spec_cls.from_dict(m)
    op = op_cls(width, spec, 1e-5, dtype=dtype)
    op.use_tensor_cores = tensor_path
    op.load(DictLoader(W), "")
    layer = {"type": "parallel", "mixer": {"left": m if kind == "left" else U.left(), "right": m if kind == "right" else U.right()}} if kind != "attention" else {"type": kind, "mixer": m}
    st = O.Model({"layers": [layer]}, {}).new_state()["layers"][0]
    Wd, pos = {k: v.double() for k, v in W.items()}, torch.arange(n)
    if kind == "left":
        want, _ = O.biased_sink_mixer(h.double(), pos, st["kv"], Wd, m, 1e-5)
    elif kind == "right":
        want, _ = O.state_space_mixer(h.double(), st["ssm"], Wd, m, 1e-5)
    else:
        want, _ = O.differential_mixer(h.double(), pos, st, Wd, m, 1e-5)
    row = spec.cache_row_width() if kind != "right" else 0
    cache = PagedStateCache([row], [spec.state_width() if kind != "left" else 0], n + page_size, 2, "cuda", dtype=dtype, page_size=page_size)
    got, at, k = [], 0, 0
    while at < n:
        p = min(portions[min(k, len(portions) - 1)], n - at)
        batch = cache.build_batch([("s", [0] * p, [])])
        got.append(op(h[at:at + p].cuda().contiguous(), batch, cache, 0))
        cache.commit()
        at, k = at + p, k + 1
    return torch.cat(got), want


def D(**kw):
    return ("attention", U.diff(**kw)["mixer"])


def L(**kw):
    return ("left", U.left(**kw))


def R(**kw):
    return ("right", U.right(**kw))


ATTN_SHAPES = [L(), L(heads=6, kv_heads=6, dim=6, vdim=3, chunk=4), L(heads=9, kv_heads=1, dim=16, vdim=40, chunk=33), L(heads=20, kv_heads=2, dim=7, vdim=70, chunk=1000, scale=0.4),
               L(heads=1, kv_heads=1, dim=33, vdim=1, scale=0.9, chunk=64), L(heads=4, kv_heads=4, dim=130, vdim=130, chunk=1),
               D(), D(heads=6, kv_heads=6, dim=6, vdim=3, chunk=4, conv=1), D(heads=9, kv_heads=1, dim=16, vdim=40, chunk=33, conv=2, dims=8), D(heads=20, kv_heads=2, dim=7, vdim=70, chunk=1000, conv=3, dims=4, scaling=None),
               D(heads=1, kv_heads=1, dim=33, vdim=2, scale=0.4, chunk=64, conv=6, dims=32), D(heads=4, kv_heads=4, dim=130, vdim=130, chunk=2, diff=0.8), D(heads=2, kv_heads=1, dim=4, vdim=5, chunk=3, dims=0)]


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("desc", ATTN_SHAPES)
def test_attention_alone(dtype, tol, desc):
    width = 24 if desc[1]["dim"] < 100 else 48
    tol = tol * (3 if desc[0] == "attention" else 1)             # the norm of a difference of maps raises the rounding of both
    err = rel if dtype == torch.float32 else rel_rows
    got, want = mixer_alone(desc, dtype, 70, 8, [70], width=width)
    assert err(got, want) < tol
    assert err(got[:3], want[:3]) < tol                          # the first tokens: one, two, three visible keys
    got2, _ = mixer_alone(desc, dtype, 70, 8, [33, 1, 1, 2, 30, 3], width=width)
    assert err(got2, want) < tol and err(got2, got) < (2e-5 if dtype == torch.float32 else tol)


@gpu
def test_each_ingredient_of_the_biased_attention_matters():
    """the restatement without the bias, the sink, the gate or the unit-rms keys differs from the kernels' result"""
    desc = L(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20)
    got, want = mixer_alone(desc, torch.float32, 40, 8, [40])
    assert rel(got, want) < 3e-5

    def changed(**kw):
        def tweak(W, h, m):
            for k, f in kw.items():
                W[k] = f(W[k])
        return mixer_alone(desc, torch.float32, 40, 8, [40], tweak=tweak)
    for kw in (dict(r1=torch.zeros_like), dict(r2=lambda x: 2 * x), dict(sink=lambda x: x - 30.0), dict(g=torch.zeros_like), dict(r1=lambda x: x.flip(0)), dict(sink=lambda x: x.flip(0))):
        g2, w2 = changed(**kw)
        assert rel(g2, w2) < 3e-5 and rel(w2, want) > 1e-2
    g2, w2 = changed(k=lambda x: 5.0 * x)                        # normed keys: their length does not count
    assert rel(g2, w2) < 3e-5 and rel(w2, want) < 1e-4
    g2, w2 = changed(sink=lambda x: x + 60.0)                    # a sink far above every score: nothing is left, and nothing overflows
    assert torch.isfinite(g2).all() and float(g2.abs().max()) < 1e-9


@gpu
def test_each_ingredient_of_the_differential_attention_matters():
    desc = D(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20)
    got, want = mixer_alone(desc, torch.float32, 40, 8, [40])
    assert rel(got, want) < 5e-5

    def changed(d=desc, **kw):
        def tweak(W, h, m):
            for k, f in kw.items():
                W[k] = f(W[k])
        return mixer_alone(d, torch.float32, 40, 8, [40], tweak=tweak)
    identity = lambda x: torch.cat([torch.zeros_like(x[:, :-1]), torch.ones_like(x[:, -1:])], 1)
    swap = lambda x: x.reshape(-1, 2, 6, x.shape[1]).flip(1).reshape(x.shape)          # map 1 <-> map 2
    for kw in ({"lq1": torch.zeros_like}, {"lk2": lambda x: 2 * x}, {"q.conv": identity}, {"k.conv": identity}, {"v.conv": identity}, {"v.conv": lambda x: x.flip(1)}, {"q": swap}, {"k": swap}):
        g2, w2 = changed(**kw)
        assert rel(g2, w2) < 1e-4 and rel(w2, want) > 1e-2
    for d in (D(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20, scaling=None), D(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20, dims=4), D(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20, diff=0.5)):
        g2, w2 = changed(d)
        assert rel(g2, w2) < 1e-4 and rel(w2, want) > 1e-3


def standout(j):
    """Makes token j's key the one every query looks for: the first input column is one for every token and the queries read only it (all
    queries of a key/value head are one vector, in both maps), the keys do not read it, token j's row is solved so that its keys are those
    vectors, and every other row is made orthogonal to what the keys would need.  A filter in front of q and k is made to pass them."""
    def tweak(W, h, m):
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        maps = 2 if "lq1" in W else 1
        g = torch.Generator().manual_seed(99)
        c = torch.randn(G, maps * d, generator=g)
        c = c / (c.reshape(G, maps, d).square().mean(-1, keepdim=True).sqrt().expand(G, maps, d).reshape(G, maps * d))      # unit rms per row
        W["q"] = torch.zeros_like(W["q"])
        W["q"][:, 0] = c.repeat_interleave(H // G, 0).reshape(-1)
        W["k"][:, 0] = 0
        for n in ("q.conv", "k.conv"):
            if n in W:
                W[n] = torch.cat([torch.zeros_like(W[n][:, :-1]), torch.ones_like(W[n][:, -1:])], 1)
        if "r1" in W:
            W["r1"], W["sink"] = 0.3 * W["r1"], W["sink"] - 2.0
        if maps == 2:      # lambda = diff: a lambda near one would take the value that both maps find almost wholly away
            W["lq1"], W["lq2"] = torch.zeros_like(W["lq1"]), torch.zeros_like(W["lq2"])
        a = torch.stack([W["k"][i * d:(i + 1) * d].double().T @ c.reshape(-1, d)[i].double() for i in range(G * maps)], 1)
        basis = torch.linalg.qr(a).Q
        for i in range(h.shape[0]):
            h[i, 0] = 0.0
            if i == j:
                h[i] = torch.linalg.lstsq(W["k"].double(), c.reshape(-1, 1).double()).solution.reshape(-1).to(h.dtype)
            else:
                h[i] = (h[i].double() - basis @ (basis.T @ h[i].double())).to(h.dtype)
            h[i, 0] = 1.0
    return tweak


SHARP = dict(heads=4, kv_heads=2, dim=6)


@gpu
@pytest.mark.parametrize("make", [L, D])
@pytest.mark.parametrize("chunk", [1, 2, 7, 32, 33, 40])
@pytest.mark.parametrize("decode", [False, True])
def test_chunk_edge_with_a_key_that_stands_out(make, chunk, decode):
    """every query looks for token j's key, the second token of a chunk: the rows from j to the end of that chunk find it, the last row of the
    chunk before and the first of the chunk after do not.  Page size 4 puts the edges on and off page borders; a chunk one longer or
    shorter must differ."""
    kw = dict(SHARP, scale=4.0) if make is L else dict(SHARP, scale=4.0, dims=0)
    j = 2 * chunk + min(1, chunk - 1)
    n = 4 * chunk + 3
    got, want = mixer_alone(make(chunk=chunk, **kw), torch.float32, n, 4, [j + 1] + [1] * n if decode else [n], tweak=standout(j), width=40)
    assert rel(got, want) < 1e-4
    edges = (2 * chunk - 1, 2 * chunk, j, 3 * chunk - 1, 3 * chunk, 3 * chunk + 1)
    for r in edges:
        assert rel(got[r], want[r]) < 1e-4
    for other in (chunk + 1, max(1, chunk - 1)):
        if other != chunk:
            _, shifted = mixer_alone(make(chunk=other, **kw), torch.float32, n, 4, [n], tweak=standout(j), width=40)
            assert max(rel(shifted[r], want[r]) for r in edges) > 1e-2      # the test bites


@gpu
@pytest.mark.parametrize("make", [L, D])
def test_far_key_among_hundreds_and_the_split_path(make):
    """token 3's key is the one every query looks for; 600 tokens later (one chunk, pages of 16) each decoded token still finds it.  A
    single decoded token on a long range cuts the range into several parts."""
    from ktransformers_b200.operators.attention import softmax_attention_splits
    kw = dict(SHARP, scale=4.0, chunk=4096) if make is L else dict(SHARP, scale=4.0, chunk=4096, dims=0)
    assert softmax_attention_splits(4, 2, 600, 1) > 1
    got, want = mixer_alone(make(**kw), torch.float32, 600, 16, [590] + [1] * 10, tweak=standout(3), width=40)
    assert rel(got, want) < 1e-4 and rel(got[-10:], want[-10:]) < 1e-4
    _, blind = mixer_alone(make(**dict(kw, chunk=300)), torch.float32, 600, 16, [600], tweak=standout(3), width=40)
    assert rel(blind[-10:], want[-10:]) > 1e-2                   # the test bites
    got_b, _ = mixer_alone(make(**kw), torch.bfloat16, 600, 16, [590] + [1] * 10, tweak=standout(3), width=40)
    assert rel_rows(got_b, want, 0.9) < 6e-2 and rel(got_b[-10:], want[-10:]) < 6e-2


MMA_SHAPES = [L(heads=4, kv_heads=2, dim=16, vdim=16, chunk=40), L(heads=8, kv_heads=1, dim=32, vdim=48, chunk=33), L(heads=6, kv_heads=2, dim=64, vdim=32, chunk=1000), L(heads=20, kv_heads=1, dim=128, vdim=128, chunk=64),
              L(heads=3, kv_heads=3, dim=48, vdim=96, chunk=1), L(heads=40, kv_heads=2, dim=16, vdim=64, chunk=17),
              D(heads=4, kv_heads=2, dim=16, vdim=16, chunk=40), D(heads=8, kv_heads=1, dim=32, vdim=48, chunk=33, conv=3), D(heads=6, kv_heads=2, dim=64, vdim=128, chunk=1000, conv=2), D(heads=20, kv_heads=1, dim=128, vdim=128, chunk=64),
              D(heads=3, kv_heads=3, dim=48, vdim=16, chunk=1), D(heads=40, kv_heads=2, dim=16, vdim=64, chunk=17, dims=8), D(heads=9, kv_heads=1, dim=16, vdim=32, chunk=100, conv=1), D(heads=7, kv_heads=1, dim=16, vdim=128, chunk=70, conv=5)]


@gpu
@pytest.mark.parametrize("desc", MMA_SHAPES)
def test_tensor_core_attention_path(desc):
    """bf16 with head sizes that are multiples of 16: the tensor-core tiles against the restatement and against the CUDA-core kernel"""
    tol = 4e-2 if desc[0] == "left" else 8e-2
    for portions in ([150], [70, 3, 2, 40, 1, 34], [130] + [1] * 20):
        got, want = mixer_alone(desc, torch.bfloat16, 150, 16, portions, width=160)
        plain, _ = mixer_alone(desc, torch.bfloat16, 150, 16, portions, width=160, tensor_path=False)
        assert rel_rows(got, want, 0.95) < tol and rel_rows(got, plain, 0.95) < tol


@gpu
@pytest.mark.parametrize("make", [L, D])
@pytest.mark.parametrize("chunk", [1, 2, 31, 32, 33, 64, 65, 100])
@pytest.mark.parametrize("decode", [False, True])
def test_tensor_core_chunk_edges_inside_and_between_key_tiles(make, chunk, decode):
    """(the keys that are not looked for score zero up to bf16 rounding of their rows, times the scale: rows that average over such
    keys carry a few percent of noise, which the norm of a difference of two maps raises)"""
    noise = 0.1 if make is L else 0.2
    kw = dict(heads=4, kv_heads=2, dim=16, vdim=16, scale=2.0) if make is L else dict(heads=4, kv_heads=2, dim=16, vdim=16, scale=2.0, dims=0)
    j = 2 * chunk + min(1, chunk - 1)
    n = 4 * chunk + 3
    got, want = mixer_alone(make(chunk=chunk, **kw), torch.bfloat16, n, 16, [j + 1] + [1] * n if decode else [n], tweak=standout(j), width=96)
    edges = (2 * chunk - 1, 2 * chunk, j, 3 * chunk - 1, 3 * chunk, 3 * chunk + 1)
    for r in edges:
        assert rel(got[r], want[r]) < noise
    for other in (chunk + 1, max(1, chunk - 1)):
        if other != chunk:
            _, shifted = mixer_alone(make(chunk=other, **kw), torch.bfloat16, n, 16, [n], tweak=standout(j), width=96)
            assert max(rel(shifted[r], want[r]) for r in edges) > 2 * noise


@gpu
@pytest.mark.parametrize("make", [L, D])
def test_tensor_core_attention_far_key_and_split_edges(make):
    kw = dict(heads=8, kv_heads=2, dim=32, vdim=32, chunk=2048, scale=1.5)
    if make is D:
        kw["dims"] = 0
    got, want = mixer_alone(make(**kw), torch.bfloat16, 450, 64, [440] + [1] * 10, tweak=standout(5), width=160)
    assert rel_rows(got, want, 0.9) < 6e-2 and rel(got[-10:], want[-10:]) < 6e-2
    _, blind = mixer_alone(make(**dict(kw, chunk=200)), torch.bfloat16, 450, 64, [450], tweak=standout(5), width=160)
    assert rel(blind[-10:], want[-10:]) > 0.2


SSD_SHAPES = [R(), R(heads=1, vdim=1, state=1, groups=1, conv=1, norm_groups=1), R(heads=6, vdim=33, state=20, groups=3, conv=4, norm_groups=2), R(heads=2, vdim=64, state=128, groups=1, conv=2, norm_groups=1),
              R(heads=8, vdim=16, state=32, groups=8, conv=4, norm_groups=8), R(heads=4, vdim=130, state=37, groups=1, conv=5, norm_groups=4), R(heads=2, vdim=300, state=256, groups=2, conv=3, norm_groups=2)]


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("desc", SSD_SHAPES)
def test_state_space_alone(dtype, tol, desc):
    """whole, in portions down to one and two tokens (shorter than the filter; on, before and after the scan's staging edges), and decoded"""
    err = rel if dtype == torch.float32 else rel_rows
    whole, want = mixer_alone(desc, dtype, 150, 8, [150])
    assert err(whole, want) < tol and err(whole[:4], want[:4]) < tol
    for portions in ([33, 1, 1, 2, 31, 16, 3, 2], [64, 65, 1], [1], [2], [17, 15, 16]):
        got, _ = mixer_alone(desc, dtype, 150, 8, portions)
        assert err(got, want) < tol and err(got, whole) < (2e-5 if dtype == torch.float32 else tol)


@gpu
@pytest.mark.parametrize("P,J,N,dv", [(4, 2, 16, 8), (2, 1, 128, 64), (6, 3, 48, 40), (3, 1, 256, 72), (8, 8, 64, 16), (2, 2, 80, 128)])
@pytest.mark.parametrize("rate", [-6.0, 0.0, 3.0])
def test_chunked_scan_on_tensor_cores(P, J, N, dv, rate):
    """bf16 inputs, fp32 outputs and states of both scans against the restatement: portions that end on, before and after the 64-token chunk
    edge, one of them starting from a state; decays from almost one to almost zero (mixed with tokens that hardly step at all)"""
    import ctypes as C

    from ktransformers_b200 import native
    lib, lens = native.seq_lib(), [64, 65, 130, 1, 15, 128]
    g = torch.Generator().manual_seed(P * N + dv)
    T, inner, ch = sum(lens), P * dv, P * dv + 2 * J * N
    xbc, dtl = torch.randn(T, ch, generator=g).bfloat16(), (2.0 * torch.randn(T, P, generator=g)).bfloat16()
    dtl[::7] = -9.0
    dtb, al, D_ = torch.randn(P, generator=g), torch.full((P,), rate) + 0.3 * torch.randn(P, generator=g), torch.randn(P, generator=g)
    before = torch.randn(P, N, dv, generator=g)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    seqs = torch.tensor([starts, lens, [-1, 2, -1, -1, -1, -1], [7 + i for i in range(len(lens))]], dtype=torch.int32).cuda()
    outs = []
    for tc in (1, 0):
        assert lib.ktb200_ssd_scan_uses_tensor_cores(P, J, N, dv, 30) == 1
        state = torch.zeros(20, P * N * dv + 3)
        state[2, :P * N * dv] = before.reshape(-1)
        state, proj, xd, y = state.cuda(), dtl.cuda(), xbc.cuda(), torch.full((T, inner), float("nan"), device="cuda")
        dev = [t.cuda() for t in (dtb, al, D_)]
        w = torch.zeros(ch, 1, dtype=torch.bfloat16, device="cuda")
        a = native.SsdParams(proj=proj.data_ptr(), proj_stride=P, xbc_off=0, dt_off=0, conv_w=w.data_ptr(), conv_b=w.data_ptr(), taps=1, dt_bias=dev[0].data_ptr(), a_log=dev[1].data_ptr(),
                             d_skip=dev[2].data_ptr(), heads=P, groups=J, state_size=N, vdim=dv, seqs=seqs.data_ptr(), seqs_stride=len(lens), n_seqs=len(lens), state=state.data_ptr(),
                             state_stride=state.stride(0))
        native.check_seq(lib.ktb200_ssd_scan(C.byref(a), xd.data_ptr(), y.data_ptr(), 30, tc, torch.cuda.current_stream().cuda_stream))
        outs.append((y.cpu(), state.cpu()))
    dt = torch.nn.functional.softplus(dtl.double() + dtb.double(), threshold=1e9)
    for i, (lo, n) in enumerate(zip(starts, lens)):
        rows, xd = slice(lo, lo + n), xbc.double()
        S0 = before.double() if i == 1 else torch.zeros(P, N, dv, dtype=torch.float64)
        want, S = O.state_space_scan(xd[rows, :inner].reshape(n, P, dv), xd[rows, inner:inner + J * N].reshape(n, J, N), xd[rows, inner + J * N:].reshape(n, J, N), dt[rows], al.double(), D_.double(), S0)
        for (y, st), tol in zip(outs, (2e-4, 2e-5)):
            assert rel(y[rows], want.reshape(n, inner)) < tol
            assert rel(st[7 + i, :P * N * dv], S.reshape(-1)) < tol


@gpu
def test_each_ingredient_of_the_state_space_matters():
    desc = R(heads=4, vdim=6, state=5, groups=2, conv=3, norm_groups=3)
    _, want = mixer_alone(desc, torch.float32, 40, 8, [40])

    def changed(**kw):
        def tweak(W, h, m):
            for k, f in kw.items():
                W[k.replace("_b", ".b") if k == "conv_b" else k] = f(W[k.replace("_b", ".b") if k == "conv_b" else k])
        return mixer_alone(desc, torch.float32, 40, 8, [40], tweak=tweak)
    for kw in (dict(conv_b=torch.zeros_like), dict(dt_bias=lambda x: x + 1), dict(A_log=lambda x: x - 1), dict(D=torch.zeros_like), dict(norm=torch.ones_like), dict(conv=lambda x: x.flip(1))):
        got, w2 = changed(**kw)
        assert rel(got, w2) < 3e-5 and rel(w2, want) > 1e-2
    for other in (R(heads=4, vdim=6, state=5, groups=2, conv=3, norm_groups=1), R(heads=4, vdim=6, state=5, groups=2, conv=3, norm_groups=4)):
        got, w2 = mixer_alone(other, torch.float32, 40, 8, [40])
        assert rel(got, w2) < 3e-5 and rel(w2, want) > 1e-2
    got, w2 = changed(dt_bias=lambda x: x + 40.0)                 # large steps: the soft-plus is the identity there, decays vanish
    assert torch.isfinite(got).all() and rel(got, w2) < 3e-5


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 5e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("decode", [False, True])
def test_state_space_carries_a_far_token(dtype, tol, decode):
    """a loud token whose trace a slow decay keeps for 300 steps, in one prompt and decoded; without the token, or with a faster decay, the
    last rows differ"""
    def loud(W, h, m):
        W["A_log"] = torch.full_like(W["A_log"], -7.0)
        W["D"] = torch.zeros_like(W["D"])
        h[4] *= 12.0
    desc = R(heads=4, vdim=16, state=16, groups=2, conv=3, norm_groups=2)
    got, want = mixer_alone(desc, dtype, 310, 8, [40] + [1] * 270 if decode else [310], tweak=loud)
    assert rel_rows(got, want, 0.95) < tol and rel_rows(got[-20:], want[-20:], 0.95) < tol

    def quiet(W, h, m):
        loud(W, h, m)
        h[4] /= 12.0
    _, without = mixer_alone(desc, dtype, 310, 8, [310], tweak=quiet)

    def fast(W, h, m):
        loud(W, h, m)
        W["A_log"] += 6.0
    _, forgets = mixer_alone(desc, dtype, 310, 8, [310], tweak=fast)
    assert rel(without[-20:], want[-20:]) > 0.1 and rel(forgets[-20:], want[-20:]) > 0.1


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_decode_and_prompt_portions_in_one_launch(dtype):
    """portions of one, two and many tokens of different sequences in one state-space and one differential batch: the filter's windows and the
    states of neighbours do not mix"""
    from ktransformers_b200.models import configuration_rununex as cfgs
    from ktransformers_b200.models.custom_cache import PagedStateCache
    from ktransformers_b200.operators.attention import KDifferentialAttention
    from ktransformers_b200.operators.linear_attention import KStateSpace
    g = torch.Generator().manual_seed(3)
    rn = lambda *s, k=1.0: torch.randn(*s, generator=g) * k
    lin = lambda o, i, s=1.0: rn(o, i, k=s / i ** 0.5)
    width = 24
    for kind, desc in (("right", U.right(conv=4, heads=4, vdim=8, state=12, norm_groups=4)), ("attention", U.diff(conv=4, dim=8, vdim=8, chunk=50)["mixer"])):
        spec = (cfgs.StateSpaceSpec if kind == "right" else cfgs.DifferentialAttentionSpec).from_dict(desc)
        W = {k: v.to(dtype) for k, v in (U.right_weights if kind == "right" else U.diff_weights)(rn, lin, "", desc, width).items()}
        op = (KStateSpace if kind == "right" else KDifferentialAttention)(width, spec, 1e-5, dtype=dtype)
        op.load(DictLoader(W), "")
        h = {i: rn(n, width).to(dtype) for i, n in (("a", 90), ("b", 40), ("c", 71), ("d", 3))}
        widths = ([0], [spec.state_width()]) if kind == "right" else ([spec.cache_row_width()], [spec.state_width()])
        together, alone = (PagedStateCache(*widths, 512, 4, "cuda", dtype=dtype, page_size=8) for _ in range(2))
        steps = [[("a", 5), ("b", 1), ("c", 70)], [("a", 1), ("b", 2), ("d", 1)], [("a", 1), ("b", 1), ("c", 1), ("d", 1)], [("b", 36), ("a", 83), ("d", 1)]]
        at, got, want = {i: 0 for i in h}, {i: [] for i in h}, {i: [] for i in h}
        for step in steps:
            batch = together.build_batch([(i, [0] * n, []) for i, n in step])
            y = op(torch.cat([h[i][at[i]:at[i] + n] for i, n in step]).cuda().contiguous(), batch, together, 0)
            together.commit()
            k = 0
            for i, n in step:
                got[i].append(y[k:k + n])
                b1 = alone.build_batch([(i, [0] * n, [])])
                want[i].append(op(h[i][at[i]:at[i] + n].cuda().contiguous(), b1, alone, 0))
                alone.commit()
                k, at[i] = k + n, at[i] + n
        for i in h:
            assert rel_rows(torch.cat(got[i]), torch.cat(want[i]), 1.0 if dtype == torch.float32 else 0.9) < (2e-5 if dtype == torch.float32 else 3e-2)


# ------------------------------------------------------------------------------------------------ whole model (GPU)
@gpu
@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_prompt_decode_and_portions_agree_with_the_restatement(tmp_path, dtype, tol):
    cfg = U.config(MIXED)
    eng, om = serve(tmp_path, cfg, dtype, max_tokens=128, max_slots=2, page_size=4)
    t = toks(75)
    want = oracle_logits(om, t)
    err = rel if dtype == "float32" else rel_rows
    whole = run_steps(eng, cut("w", t, [75]))["w"]
    assert err(whole, want) < tol
    assert err(whole[:4], want[:4]) < tol                       # the first tokens of a sequence
    for sizes in ([1], [2], [3, 2, 7, 1, 5], [20, 2, 2, 1]):
        got = run_steps(eng, cut("p", t, sizes))["p"]
        assert err(got, want) < tol
        assert err(got, whole) < (5e-5 if dtype == "float32" else tol)   # the cut does not matter beyond rounding


@gpu
def test_whole_model_in_bf16_on_tensor_core_head_sizes(tmp_path):
    """head sizes that are multiples of 16: bf16 attention runs on the tensor-core tiles inside a whole model, 150 tokens over several key tiles
    and chunks, whole, in portions and with a decoded tail"""
    layers = [(U.parallel(U.left(heads=6, kv_heads=2, dim=32, vdim=48, chunk=40), U.right(heads=4, vdim=32, state=16, groups=1, conv=4, norm_groups=2)), U.moe(ff=32, experts=4, top=2, shared=48)),
              (U.diff(heads=4, kv_heads=1, dim=16, vdim=32, chunk=64, conv=3), U.moe(ff=32, experts=4, top=1, shared=32)), (U.diff(heads=4, kv_heads=2, dim=16, vdim=48, chunk=33), None)]
    cfg = U.config(layers, width=64, vocab=90)
    eng, om = serve(tmp_path, cfg, "bfloat16", seed=3, max_tokens=512, max_slots=2, page_size=16)
    t = toks(150, 90, seed=9)
    want = oracle_logits(om, t)
    for k, sizes in enumerate(([150], [70, 3, 2, 40, 1, 34], [130] + [1] * 20)):
        assert rel_rows(run_steps(eng, cut(("m", k), t, sizes))[("m", k)], want) < BF16_TOL


@gpu
def test_residual_stream_after_every_layer(tmp_path):
    cfg = U.config(MIXED)
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=64, max_slots=2, page_size=8)
    t = toks(11, seed=2)
    want, got = [], []
    om.forward(t, om.new_state(), want)
    eng.model(eng.cache.build_batch([("r", t, [])]), eng.cache, got)
    assert len(got) == len(want) == 4
    for a, b in zip(got, want):
        assert rel(a, b) < 1e-4


@gpu
def test_model_constants_matter(tmp_path):
    """the restatement with another embedding scale, residual factor, logit scale or mixer scale differs"""
    cfg = U.config(MIXED)
    eng, om = serve(tmp_path, cfg, "float32", seed=1, max_tokens=64, max_slots=2, page_size=8)
    t, w = toks(20, seed=4), U.weights(cfg, 1, torch.float32)
    want = oracle_logits(om, t)
    assert rel(run_steps(eng, cut("a", t, [13, 2, 1]))["a"], want) < F32_TOL
    other = json.loads(json.dumps(cfg))
    other["layers"][0]["mixer"]["left_scale"] = 1.0
    other2 = json.loads(json.dumps(cfg))
    other2["layers"][0]["mixer"]["right_scale"] = 1.0
    for c in (dict(cfg, embedding={"scale": 1.0}), dict(cfg, residual_mult=1.0), dict(cfg, logit_scale=1.0), other, other2):
        assert rel(oracle_logits(O.Model(c, w, torch.float64), t), want) > 1e-3


@gpu
def test_other_sizes_and_layer_orders(tmp_path):
    cases = [
        ([(U.diff(heads=1, kv_heads=1, dim=2, vdim=2, chunk=3, conv=1), U.moe(ff=3, experts=1, top=1, shared=2))], dict(width=8)),                                                       # one small layer, one expert
        ([(U.parallel(U.left(heads=1, kv_heads=1, dim=2, vdim=1, chunk=1), U.right(heads=1, vdim=1, state=1, groups=1, conv=1, norm_groups=1), 1.0, 1.0), None)], dict(width=4, residual_mult=1.0, logit_scale=1.0)),
        ([(U.parallel(U.left(heads=16, kv_heads=4, dim=12, vdim=10, chunk=12), U.right(heads=8, vdim=8, state=24, groups=4, conv=4, norm_groups=8)), U.moe(ff=20, experts=16, top=4)),
          (U.diff(heads=8, kv_heads=8, dim=4, vdim=9, chunk=30), None)] * 2, dict(width=72, vocab=31)),
        ([(U.diff(heads=5, kv_heads=5, dim=24, vdim=24, chunk=2, conv=5), U.moe(ff=5, experts=3, top=3, shared=1)), (U.diff(heads=2, kv_heads=1, dim=8, vdim=8, dims=4), U.moe())], dict(width=40)),
        ([(U.parallel(), None), (U.parallel(U.left(chunk=3), U.right(conv=6, state=33)), U.moe(ff=33, top=6)), (U.diff(chunk=1), U.moe(experts=4, top=1))], dict(width=16, eps=1e-3, embed_scale=1.0)),
        ([(U.parallel(U.left(heads=2, kv_heads=2, dim=4, vdim=3, chunk=500), U.right(heads=3, vdim=7, state=9, groups=3, conv=2, norm_groups=7)), U.moe(ff=33, experts=10, top=2))], dict(width=14, vocab=7))]
    for k, (layers, kw) in enumerate(cases):
        cfg = U.config(layers, **kw)
        eng, om = serve(tmp_path, cfg, "float32", seed=10 + k, max_tokens=64, max_slots=2, page_size=8)
        t = toks(30, cfg["vocab"], seed=k)
        assert rel(run_steps(eng, cut("a", t, [13, 2, 1]))["a"], oracle_logits(om, t)) < F32_TOL


@gpu
@pytest.mark.parametrize("seed", range(8))
def test_drawn_configurations(tmp_path, seed):
    """sizes, layer order and constants drawn per seed: one prompt whole, in uneven portions, and with a decoded tail"""
    r = random.Random(seed)
    width = r.choice([16, 40, 136, 320])
    layers = []
    for _ in range(r.randint(1, 4)):
        G = r.choice([1, 2, 4])
        a = dict(heads=G * r.choice([1, 2, 5]), kv_heads=G, dim=r.choice([4, 6, 24, 64]), vdim=r.choice([5, 8, 80]), scale=r.choice([None, 0.11, 0.6]), chunk=r.choice([1, 5, 31, 32, 33, 64, 100, 1000]))
        if r.random() < 0.5:
            J = r.choice([1, 2, 4])
            P, dv = J * r.choice([1, 3]), r.choice([4, 12, 40])
            m = U.parallel(U.left(**a), U.right(heads=P, vdim=dv, state=r.choice([4, 17, 64]), groups=J, conv=r.choice([1, 2, 3, 4, 5]), norm_groups=r.choice([1, 2, P])), r.choice([1.0, 0.4]), r.choice([1.0, 1.6]))
        else:
            m = U.diff(conv=r.choice([1, 2, 3, 4, 5]), diff=r.choice([0.2, 0.75]), dims=r.choice([0, 2, 4, a["dim"]]), base=r.choice([50.0, 10000.0]),
                       scaling=r.choice([None, (4.0, 1.0, 4.0, 40), (8.0, 2.0, 3.0, 500)]), **a)
        E = r.choice([1, 3, 8, 24])
        layers.append((m, None if r.random() < 0.2 else U.moe(ff=r.choice([8, 24, 100]), experts=E, top=r.randint(1, min(E, 6)), shared=r.choice([1, 8, 50]))))
    cfg = U.config(layers, vocab=r.choice([31, 77, 1000]), width=width, eps=r.choice([1e-6, 1e-5, 1e-3]), embed_scale=r.choice([1.0, 4.0, 12.5]), residual_mult=r.choice([0.3, 1.0]),
                   logit_scale=r.choice([0.2, 1.0]))
    eng, om = serve(tmp_path, cfg, "float32", seed=seed, max_tokens=256, max_slots=2, page_size=r.choice([4, 16, 64]))
    t = toks(r.choice([40, 90, 120]), cfg["vocab"], seed=seed)
    want = oracle_logits(om, t)
    for k, sizes in enumerate(([len(t)], [3, 17, 2, 1, 33, 2, 64], [len(t) - 20] + [1] * 20)):
        assert rel(run_steps(eng, cut(("d", k), t, sizes))[("d", k)], want) < F32_TOL


@gpu
def test_captured_decode_steps_in_a_large_cache(tmp_path):
    """decode steps replay a captured graph; the state rows flip between the replays, and a roomy cache changes nothing"""
    cfg = U.config(MIXED)
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=8192, max_slots=2, page_size=16)
    for r, n in enumerate((40, 130)):
        t = toks(n, seed=40 + r)
        got = run_steps(eng, cut(("g", r), t, [n - 12] + [1] * 12))[("g", r)]
        assert rel(got, oracle_logits(om, t)) < F32_TOL
    assert 1 in eng._captured and eng._captured[1].graph is not None


@gpu
def test_unequal_requests_in_one_batch_equal_each_alone(tmp_path):
    cfg = U.config(MIXED)
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=256, max_slots=4, page_size=4)
    ta, tb, tc = toks(23, seed=1), toks(9, seed=2), toks(14, seed=3)
    steps = [[("a", ta[:10], False), ("b", tb[:1], False)],
             [("a", ta[10:11], False), ("b", tb[1:9], True), ("c", tc[:2], False)],
             [("c", tc[2:14], True), ("a", ta[11:23], True)]]
    got = run_steps(eng, steps)
    for i, t in (("a", ta), ("b", tb), ("c", tc)):
        assert rel(got[i], oracle_logits(om, t)) < F32_TOL
        alone = run_steps(eng, cut(i + "'", t, [len(t)]))[i + "'"]
        assert rel(got[i], alone) < 5e-5


@gpu
def test_long_decode_over_reused_pages_and_slots(tmp_path):
    """pages of 4 and 2 slots: sequences come and go, pages and state rows are handed out again un-cleared, and a new sequence in a used
    slot must start from an empty state and an empty filter.  Every layer's mask is chunked, so the pages before the current chunk are given
    back while a sequence runs and its page table row wraps around."""
    layers = [(U.parallel(U.left(chunk=9)), U.moe()), (U.diff(chunk=21), U.moe()), (U.diff(heads=2, kv_heads=2, dim=8, vdim=8, chunk=4, conv=2), None)]
    cfg = U.config(layers)
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=48, max_slots=2, page_size=4)
    assert eng.cache.chunks == [4, 9, 21]
    for r in range(3):
        t = toks(150, seed=20 + r)                              # longer than the cache: only the current chunks' pages are held
        got = run_steps(eng, cut(("s", r), t, [6] + [1] * 144))[("s", r)]
        assert rel(got, oracle_logits(om, t)) < F32_TOL
        short = toks(3, seed=30 + r)
        assert rel(run_steps(eng, cut(("t", r), short, [3]))[("t", r)], oracle_logits(om, short)) < F32_TOL
    assert len(eng.cache._free_pages) == eng.cache.num_pages and len(eng.cache._free_slots) == 2


@gpu
def test_greedy_generation_through_the_scheduler_and_the_command_line(tmp_path, capsys):
    from ktransformers_b200 import local_chat
    cfg = U.config(MIXED)
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=256, max_slots=3, page_size=4, max_step_tokens=7)
    prompts = [toks(12, seed=5), toks(3, seed=6), toks(20, seed=7), toks(1, seed=8)]
    want = []
    for p in prompts:
        st, out = om.new_state(), []
        nxt = int(om.forward(p, st)[-1].argmax())
        for _ in range(6):
            out.append(nxt)
            nxt = int(om.forward([nxt], st)[-1].argmax())
        want.append(out)
    assert eng.generate(prompts, 6) == want                      # 4 requests, 3 slots, 7 tokens per step: portions and decode mix
    assert len(eng.cache._free_slots) == 3
    args = ["--model_path", str(tmp_path / "ckpt0"), "--dtype", "float32", "--max_new_tokens", "6", "--chunk_size", "5"]
    for p in prompts[:2]:
        args += ["--prompt_ids", ",".join(map(str, p))]
    assert local_chat.main(args) == 0
    lines = [json.loads(l) for l in capsys.readouterr().out.strip().splitlines() if l.startswith("{")]
    assert [l["output"] for l in lines] == want[:2]


@gpu
@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_trace_replay_runner(tmp_path, dtype, tol):
    """bin/trace_run as a process: steps on standard input, one logits file per step that asks for some, `done <n>` lines"""
    import os
    import subprocess
    import sys

    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = U.config(MIXED, vocab=41)
    w = U.weights(cfg, 5, torch.bfloat16 if dtype == "bfloat16" else torch.float32)
    path = U.save(tmp_path / "m", cfg, w)
    om = O.Model(cfg, w, torch.float64)
    a, b = toks(21, 41, seed=1), toks(9, 41, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:15], "want": [0, 14]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[15:17], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[17:18], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[18:21], "want": [2, 1]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [8]}], "end": ["b"]}]
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(5)]
    la, lb = oracle_logits(om, a), oracle_logits(om, b)
    want = {0: la[[0, 14]], 2: la[[17]], 3: la[[20, 19]], 4: lb[[8]]}
    assert not (out / "1.f32").exists()
    err = rel if dtype == "float32" else rel_rows
    for n, ref in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, 41))
        assert got.shape == ref.shape and err(got, ref) < tol
