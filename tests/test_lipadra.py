"""Lipadra through the framework (registry, loader, paged state cache, scheduler, engine, CUDA operators) against the plain
restatement in oracle/lipadra_oracle.py, on small random checkpoints made here.  CPU tests cover the host logic."""
import ctypes as C
import json
import math
import random

import pytest
import torch

import lipadra_util as U
from oracle import lipadra_oracle as O

gpu = pytest.mark.gpu
F32_TOL, BF16_TOL = 2e-4, 8e-2


def rel(a, b):
    a, b = a.detach().double().cpu(), b.detach().double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


def rel_rows(a, b, q=0.8):
    """the q-quantile of the per-row errors, for bf16 runs of whole models (a close call of the router may go the other way)"""
    a, b = a.detach().double().cpu(), b.detach().double().cpu()
    return float(((a - b).abs().amax(-1) / b.abs().max()).quantile(q))


class DictLoader:
    def __init__(self, w):
        self.w = w

    def load_tensor(self, key, device="cpu"):
        return self.w[key].to(device)


def part(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


MIXED = [(U.attention(), U.moe()), (U.retention(), U.moe(ff=7, experts=9, identity=0, top=1, groups=(1, 1), shared=5)), (U.scan(), None), (U.retention(heads=2, dim=4, vdim=8, dims=2), U.moe(identity=5)), 0,
         (U.scan(inner=9, state=3, dt_rank=2, conv=2), U.moe(experts=5, identity=7, top=3, groups=(4, 2), shared=0)), 1, 2, 5]


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
    from ktransformers_b200.models.configuration_lipadra import LipadraConfig
    cfg = U.config(MIXED, vocab=77, width=40, eps=2e-4, alpha=3.25)
    c = LipadraConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.norm_eps, c.alpha, c.num_hidden_layers) == (77, 40, 2e-4, 3.25, 9)
    a, r, m = c.layers[0].mixer, c.layers[3].mixer, c.layers[5].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.rot.base, a.rot.dims, a.rot.layout) == (4, 2, 6, 5, 7, 300.0, 4, "halves")
    assert (r.heads, r.dim, r.vdim, r.rot.dims, len(r.decay), r.decay[0]) == (2, 4, 8, 2, 2, 0.7)
    assert (m.inner, m.state_size, m.dt_rank, m.conv) == (9, 3, 2, 2)
    f = c.layers[5].mlp
    assert (f.ff, f.experts, f.identity, f.top, f.groups, f.keep_groups, f.out_scale, f.shared_ff) == (10, 5, 7, 3, 4, 2, 1.7, None) and c.layers[2].mlp is None
    assert [l.weights_of for l in c.layers] == [0, 1, 2, 3, 0, 5, 1, 2, 5]
    assert c.cache_row_widths() == [22, 0, 0, 0, 22, 0, 0, 0, 0]
    assert c.state_widths() == [0, 90, 14 * 8, 64, 0, 9 * 4, 90, 14 * 8, 9 * 4]
    assert c.chunks() == [7, 7]
    whole = json.loads(json.dumps(cfg))
    whole["layers"][0]["mixer"]["mask"] = whole["layers"][4]["mixer"]["mask"] = None
    assert LipadraConfig.from_dict(whole).chunks() is None
    for bad in (dict(type="conv"), dict(mlp={"kind": "dense", "ff": 3})):
        with pytest.raises(ValueError):
            LipadraConfig.from_dict(dict(cfg, layers=[dict(cfg["layers"][0], **bad)]))


def test_layers_that_use_other_layers_tensors():
    from ktransformers_b200.models.configuration_lipadra import LipadraConfig
    cfg = U.config([(U.retention(), None), 0, 1])                # a chain: both end at layer 0
    assert [l.weights_of for l in LipadraConfig.from_dict(cfg).layers] == [0, 0, 0]
    for change in (dict(weights_of=1), dict(weights_of=7), dict(mixer=U.retention(heads=2)["mixer"]), dict(type="mamba1", mixer=U.scan()["mixer"])):
        layers = [cfg["layers"][0], dict(cfg["layers"][1], **change)]
        with pytest.raises(ValueError):
            LipadraConfig.from_dict(dict(cfg, layers=layers))


def test_registry_picks_the_class_by_config():
    from ktransformers_b200.models import architecture_of, model_class
    assert model_class(architecture_of(U.config(MIXED))).__name__ == "LipadraForCausalLM"


def test_model_shares_tensors_not_caches():
    from ktransformers_b200.models.configuration_lipadra import LipadraConfig
    from ktransformers_b200.models.modeling_lipadra import LipadraForCausalLM
    m = LipadraForCausalLM(LipadraConfig.from_dict(U.config(MIXED)), dtype=torch.float32, device="cpu")
    layers = m.layers
    assert layers[4] is layers[0] and layers[8] is layers[5] and layers[7] is layers[2] and layers[6] is layers[1] and len(set(map(id, layers))) == 5
    cache = m.make_cache(64)
    assert len(cache.key_cache) == len(cache.state) == 9 and cache.state[6].data_ptr() != cache.state[1].data_ptr()
    assert len({n for n, _ in m.named_parameters() if n.startswith("owned.")}) == sum(1 for _ in (p for l in set(layers) for p in l.parameters()))


def test_pages_go_back_when_no_layer_keeps_rows():
    from ktransformers_b200.models.configuration_lipadra import LipadraConfig
    c = LipadraConfig.from_dict(U.config([(U.retention(), None), (U.scan(), None)]))
    assert c.chunks() == [1] and c.cache_row_widths() == [0, 0]


def test_oracle_portions_equal_whole_prompt():
    cfg = U.config(MIXED)
    om = O.Model(cfg, U.weights(cfg, 3, torch.float32))
    t = toks(23, seed=1)
    whole = om.forward(t, om.new_state())
    st = om.new_state()
    parts = torch.cat([om.forward(t[a:b], st) for a, b in ((0, 6), (6, 7), (7, 9), (9, 23))])
    assert rel(parts, whole) < 1e-9


def test_oracle_mechanisms_against_closed_forms():
    g = torch.Generator().manual_seed(0)
    rn = lambda *s: torch.randn(*s, generator=g).double()
    # the plus-one soft-max in matrix form
    q, k, v, pos = rn(11, 4, 3), rn(11, 2, 3), rn(11, 2, 2), torch.arange(11)
    s = torch.einsum("thd,nhd->htn", q, k.repeat_interleave(2, 1)) * 0.7
    e = torch.exp(s) * ((pos[None, :] <= pos[:, None]) & (pos[None, :] // 4 == pos[:, None] // 4))
    want = torch.einsum("htn,nhv->thv", e / (1.0 + e.sum(-1, keepdim=True)), v.repeat_interleave(2, 1))
    assert rel(O.plus_one_attention(q, k, v, pos, pos, 0.7, 4), want) < 1e-12
    # retention: o_t = sum_j decay^(t - j) (q_t . k_j) v_j
    q, k, v, decay = rn(9, 2, 3), rn(9, 2, 3), rn(9, 2, 4), [0.9, 0.5]
    o, _ = O.retention(q, k, v, decay, torch.zeros(2, 3, 4).double())
    for t in range(9):
        for h in range(2):
            assert rel(o[t, h], sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))) < 1e-10
    # the scan: y_t = sum_j sum_n exp(a_n sum of dt in (j, t]) dt_j x_j B_jn C_tn + D x_t
    x, dt, A, B, Cm, D = rn(9, 3), torch.rand(9, 3, generator=g).double(), -torch.rand(3, 4, generator=g).double(), rn(9, 4), rn(9, 4), rn(3)
    y, _ = O.selective_scan(x, dt, A, B, Cm, D, torch.zeros(3, 4).double())
    cum = torch.cumsum(dt, 0)
    for t in range(9):
        want = D * x[t] + sum((torch.exp(A * (cum[t] - cum[j])[:, None]) * B[j] * Cm[t]).sum(-1) * dt[j] * x[j] for j in range(t + 1))
        assert rel(y[t], want) < 1e-10


# ------------------------------------------------------------------------------------------------ mechanisms alone (GPU)
@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("width,n", [(20, 5), (35, 7), (6, 3), (256, 9), (1024, 300), (7168, 3), (9000, 2), (12288, 301), (20000, 2)])
def test_norm_behind_the_sum(dtype, tol, width, n):
    from ktransformers_b200.operators.norm import KSumRMSNorm
    g = torch.Generator().manual_seed(width)
    rn = lambda *s: torch.randn(*s, generator=g)
    x, a, b, bs = rn(n, width) + 0.5, rn(n, width), rn(n, width).to(dtype), torch.rand(n, generator=g)
    w, dot = (1 + 0.3 * rn(width)).to(dtype), (rn(width) / width ** 0.5).to(dtype)
    ids, iw = torch.randint(0, 9, (n, 3), generator=g), torch.rand(n, 3, generator=g)
    op = KSumRMSNorm(width, 1e-3, dtype=dtype)
    op.load(DictLoader({"n": w}), "n")
    c = lambda t: t.cuda()
    wid = (iw * (ids >= 6)).sum(-1, keepdim=True).double()
    s = (2.5 + wid) * x.double() + a.double() + bs.double()[:, None] * b.double()
    want = O.rms(s, 1e-3) * w.double()
    y, h, gate = op(c(x), 2.5, c(a), c(b), c(bs), (c(ids), c(iw), 6), dot=c(dot))
    assert y.dtype == torch.float32 and h.dtype == dtype and rel(y, want) < 1e-5 and rel(h, want) < tol
    assert rel(gate, torch.sigmoid(want @ dot.double())) < 1e-5
    # picked rows of everything; each term alone
    rows = torch.tensor([n - 1, 0, 1, 0])
    y, h, gate = op(c(x), 2.5, c(a), c(b), c(bs), (c(ids), c(iw), 6), rows=c(rows), keep_x=False)
    assert rel(h, want[rows]) < tol and gate is None and (y is None or dtype == torch.float32)
    assert rel(op(c(x), 0.7, a=c(b))[0], O.rms(0.7 * x.double() + b.double(), 1e-3) * w.double()) < 1e-5
    assert rel(op(c(b), 1.0, b=c(a))[0], O.rms(b.double() + a.double(), 1e-3) * w.double()) < 1e-5
    assert rel(op(c(x))[0], O.rms(x.double(), 1e-3) * w.double()) < 1e-5
    assert rel(op(c(x), 2.5, identity=(c(ids), c(iw), 9))[0], O.rms(2.5 * x.double(), 1e-3) * w.double()) < 1e-5      # nothing chosen among the identities
    assert rel(O.rms(2.5 * x.double() + a.double() + bs.double()[:, None] * b.double(), 1e-3) * w.double(), want) > 1e-3


@gpu
@pytest.mark.parametrize("outputs,top,groups,keep", [(6, 2, 3, 1), (12, 3, 4, 2), (5, 5, 1, 1), (64, 8, 8, 3), (9, 1, 9, 2), (512, 32, 32, 4), (10, 4, 5, 5)])
@pytest.mark.parametrize("width,n", [(24, 7), (24, 130), (30, 5)])
@pytest.mark.parametrize("shift", [0.0, -1.0])
def test_grouped_softmax_router(outputs, top, groups, keep, width, n, shift):
    """decode-sized batches (one launch), prompt-sized ones (GEMM + selection), a width the GEMV kernel does not take; choice scores of both
    signs and all below zero (an excluded output counts as minus infinity, not as 0)"""
    from ktransformers_b200.operators.gate import KGroupedSoftmaxGate
    g = torch.Generator().manual_seed(n + outputs)
    W, x, corr = torch.randn(outputs, width, generator=g) * 0.4, torch.randn(n, width, generator=g), torch.randn(outputs, generator=g) * 0.3 + shift
    op = KGroupedSoftmaxGate(width, outputs, top, groups, keep, 2.25)
    op.load(DictLoader({"r": W, "c": corr}), "r", "c")
    ids, wts = op(x.cuda())
    want_ids, want_w = O.grouped_softmax_router(x.double(), W.double(), corr.double(), top, groups, keep, 2.25)
    assert ids.cpu().tolist() == want_ids.tolist() and rel(wts, want_w) < 1e-5
    if groups > keep and top > keep and n > 100:      # the groups matter
        free, _ = O.grouped_softmax_router(x.double(), W.double(), corr.double(), top, 1, 1, 2.25)
        assert free.tolist() != want_ids.tolist()
    plain, _ = O.grouped_softmax_router(x.double(), W.double(), torch.zeros(outputs).double(), top, groups, keep, 2.25)
    assert top == outputs or n < 100 or plain.tolist() != want_ids.tolist()


@gpu
@pytest.mark.parametrize("outputs,top,groups,keep", [(13, 3, 1, 1), (24, 5, 4, 2), (320, 8, 8, 3)])
@pytest.mark.parametrize("n", [1, 6, 200])
@pytest.mark.parametrize("width", [64, 72, 1024, 50])
def test_router_on_bf16_rows(outputs, top, groups, keep, n, width):
    """bf16 rows and bf16 router weights: one GEMM with exact products and fp32 sums beyond a few tokens; weights that are no bf16 numbers, or a
    width the GEMM does not take, keep to fp32 products"""
    from ktransformers_b200.operators.gate import KGroupedSoftmaxGate
    g = torch.Generator().manual_seed(n + outputs)
    x, corr = torch.randn(n, width, generator=g).bfloat16(), torch.randn(outputs, generator=g) * 0.3
    for rounded in (True, False):
        W = torch.randn(outputs, width, generator=g) * 3.0 / width ** 0.5
        W = W.bfloat16() if rounded else W
        op = KGroupedSoftmaxGate(width, outputs, top, groups, keep, 1.5)
        op.load(DictLoader({"r": W, "c": corr}), "r", "c")
        assert (op.weight_bf16 is not None) == (rounded and width % 8 == 0)
        ids, wts = op(x.cuda())
        want_ids, want_w = O.grouped_softmax_router(x.double(), W.double(), corr.double(), top, groups, keep, 1.5)
        assert ids.cpu().tolist() == want_ids.tolist() and rel(wts, want_w) < 1e-5


def test_router_refuses_impossible_sizes():
    from ktransformers_b200.operators.gate import KGroupedSoftmaxGate
    for outputs, top, groups, keep in ((7, 1, 2, 1), (8, 5, 2, 1), (8, 2, 2, 3), (8, 2, 2, 0), (600, 2, 2, 1), (64, 33, 1, 1)):
        with pytest.raises(ValueError):
            KGroupedSoftmaxGate(8, outputs, top, groups, keep, 1.0, device="cpu")


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("n,path", [(1, "pair"), (5, "pair"), (3, "expert"), (9, "expert"), (70, "grouped")])
def test_experts_pass_over_choices_without_tensors(dtype, tol, n, path):
    """ids at or beyond the experts add nothing on any path, also where every choice of a token or of the whole batch is one of them"""
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
        ids = torch.stack([torch.randperm(2 * E, generator=g)[:top] for _ in range(n)])
        ids[-1] = torch.arange(E, E + top)
        wts = 0.2 + 0.6 * torch.rand(n, top, generator=g)
        torch.full((1 << 22,), float("nan"), device="cuda")                # what the allocator hands out next holds NaNs
        got = op(x.cuda(), ids.cuda(), wts.cuda())
        Wd = {k: v.double() for k, v in W.items()}
        one = lambda t, j: O.gated_expert(x[t].double(), Wd[f"e{int(ids[t, j])}.gate"], Wd[f"e{int(ids[t, j])}.up"], Wd[f"e{int(ids[t, j])}.down"])
        want = torch.stack([sum((wts[t, j].double() * one(t, j) for j in range(top) if int(ids[t, j]) < E), torch.zeros(width).double()) for t in range(n)])
        assert float((got.double().cpu() - want).abs().max()) < tol * max(1.0, float(want.abs().max()))
        none = op(x.cuda(), (ids % E + E).cuda(), wts.cuda())
        assert float(none.abs().max()) == 0.0


@gpu
@pytest.mark.parametrize("n", [9, 60])
@pytest.mark.parametrize("kw", [{}, dict(identity=0, groups=(7, 3)), dict(shared=0), dict(experts=4, identity=4, top=4, groups=(2, 1))])
def test_feed_forward_with_its_norms(n, kw):
    """router, experts, identity experts, shared expert and its gate, as the two norms around them put the sum together"""
    from ktransformers_b200.operators.experts import KIdentityMoE
    from ktransformers_b200.operators.norm import KSumRMSNorm
    cfg = U.config([(U.retention(), U.moe(**dict(dict(ff=11, shared=19), **kw)))], width=28)
    W, f = part(U.weights(cfg, 4, torch.float32), "l0.mlp."), cfg["layers"][0]["mlp"]
    r = f["router"]
    op = KIdentityMoE(28, 11, r["experts"], r["identity"], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"], f["shared"]["ff"] if f["shared"] else None, dtype=torch.float32)
    op.load(DictLoader(W), "")
    n1, n2 = KSumRMSNorm(28, 1e-5, dtype=torch.float32), KSumRMSNorm(28, 1e-5, dtype=torch.float32)
    x0 = torch.randn(n, 28, generator=torch.Generator().manual_seed(0))
    x, h, gate = n1(x0.cuda(), dot=op.shared_gate)
    routed, ids, w, shared = op(h)
    y, _, _ = n2(x, 1.5, a=routed, b=shared, b_scale=gate, identity=(ids, w, op.experts.experts) if op.identity else None)
    xd = O.rms(x0.double(), 1e-5)
    Wd = {k: v.double() for k, v in W.items()}
    want = O.rms(1.5 * xd + O.moe_mlp(xd, Wd, f), 1e-5)
    assert rel(y, want) < 3e-5
    if r["identity"]:
        assert int((ids >= r["experts"]).sum()) > 0
        lost = O.moe_mlp(xd, Wd, f) - sum((w.cpu().double() * (ids.cpu() >= r["experts"]))[:, j:j + 1] * xd for j in range(r["top"]))
        assert rel(O.rms(1.5 * xd + lost, 1e-5), want) > 1e-2
    if f["shared"]:
        ungated = dict(Wd, **{"shared.sg": torch.zeros(1, 28).double()})
        assert rel(O.rms(1.5 * xd + O.moe_mlp(xd, ungated, f), 1e-5), want) > 1e-2


def mixer_alone(desc, dtype, n, page_size, portions, seed=4, width=24, tweak=None, tensor_path=True):
    """one mixer over one sequence cut into `portions` (the last size repeats), against the restatement over the whole sequence"""
    from ktransformers_b200.models.configuration_lipadra import MIXER_SPECS
    from ktransformers_b200.models.custom_cache import PagedStateCache
    from ktransformers_b200.models.modeling_lipadra import MIXERS
    kind, m = desc["type"], desc["mixer"]
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s, k=1.0: torch.randn(*s, generator=g) * k
    lin = lambda o, i, s=1.0: rn(o, i, k=s / i ** 0.5)
    W = U.WEIGHTS[kind](rn, lin, "", m, width)
    h = rn(n, width)
    if tweak:
        tweak(W, h, m)
    W, h = {k: v.to(dtype) for k, v in W.items()}, h.to(dtype)
    spec = MIXER_SPECS[kind].from_dict(m)
    op = MIXERS[kind](width, spec, 1e-5, dtype=dtype)
    op.use_tensor_cores = tensor_path
    op.load(DictLoader(W), "")
    st = O.Model({"layers": [desc]}, {}).new_state()["layers"][0]
    Wd, pos = {k: v.double() for k, v in W.items()}, torch.arange(n)
    if kind == "attention":
        want, _ = O.attention_mixer(h.double(), pos, st, Wd, m, 1e-5)
    elif kind == "retention":
        want, _ = O.retention_mixer(h.double(), pos, st, Wd, m, 1e-5)
    else:
        want, _ = O.selective_scan_mixer(h.double(), st, Wd, m)
    cache = PagedStateCache([spec.cache_row_width()], [spec.state_width()], n + page_size, 2, "cuda", dtype=dtype, page_size=page_size)
    got, at, k = [], 0, 0
    while at < n:
        p = min(portions[min(k, len(portions) - 1)], n - at)
        batch = cache.build_batch([("s", [0] * p, [])])
        got.append(op(h[at:at + p].cuda().contiguous(), batch, cache, 0))
        cache.commit()
        at, k = at + p, k + 1
    return torch.cat(got), want


A, R, S = U.attention, U.retention, U.scan


def changed(desc, **kw):
    def tweak(W, h, m):
        for k, f in kw.items():
            k = k.replace("_b", ".b").replace("_norm", ".norm")
            W[k] = f(W[k])
    return mixer_alone(desc, torch.float32, 40, 8, [40], tweak=tweak)


ATTN_SHAPES = [A(), A(heads=6, kv_heads=6, dim=6, vdim=3, chunk=4, dims=6), A(heads=9, kv_heads=1, dim=16, vdim=40, chunk=33, dims=8), A(heads=20, kv_heads=2, dim=7, vdim=70, chunk=1000, scale=0.4, dims=2),
               A(heads=1, kv_heads=1, dim=33, vdim=1, scale=0.9, chunk=64, dims=32), A(heads=4, kv_heads=4, dim=130, vdim=130, chunk=1, dims=130), A(heads=3, kv_heads=3, dim=1, vdim=2, chunk=5, dims=0)]


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("desc", ATTN_SHAPES)
def test_attention_alone(dtype, tol, desc):
    width = 24 if desc["mixer"]["dim"] < 100 else 48
    err = rel if dtype == torch.float32 else rel_rows
    got, want = mixer_alone(desc, dtype, 70, 8, [70], width=width)
    assert err(got, want) < tol
    assert err(got[:3], want[:3]) < tol                          # the first tokens: one, two, three visible keys
    got2, _ = mixer_alone(desc, dtype, 70, 8, [33, 1, 1, 2, 30, 3], width=width)
    assert err(got2, want) < tol and err(got2, got) < (2e-5 if dtype == torch.float32 else tol)


@gpu
def test_each_ingredient_of_the_attention_matters():
    desc = A(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20)
    got, want = mixer_alone(desc, torch.float32, 40, 8, [40])
    assert rel(got, want) < 3e-5
    for kw in (dict(q_b=torch.zeros_like), dict(k_b=torch.zeros_like), dict(v_b=torch.zeros_like), dict(q_norm=torch.ones_like), dict(k_norm=torch.ones_like), dict(k_norm=lambda x: x.flip(0))):
        g2, w2 = changed(desc, **kw)
        assert rel(g2, w2) < 3e-5 and rel(w2, want) > 1e-2
    g2, w2 = changed(desc, k=lambda x: 5.0 * x, k_b=lambda x: 5.0 * x)      # normed keys: their length does not count
    assert rel(g2, w2) < 3e-5 and rel(w2, want) < 1e-4
    for other in (A(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20, dims=2), A(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20, base=30.0), A(heads=4, kv_heads=2, dim=6, vdim=5, chunk=20, scale=0.3),
                  A(heads=4, kv_heads=2, dim=6, vdim=5, chunk=19)):
        g2, w2 = mixer_alone(other, torch.float32, 40, 8, [40])
        assert rel(g2, w2) < 3e-5 and rel(w2, want) > 1e-2
    # the one in the denominator: scores far below zero leave nothing, far above leave a plain soft-max; nothing overflows
    low, w2 = changed(A(heads=4, kv_heads=2, dim=1, vdim=5, chunk=20, dims=0, scale=-40.0), q_norm=torch.ones_like, k_norm=torch.ones_like, q=torch.zeros_like, k=torch.zeros_like,
                      q_b=torch.ones_like, k_b=torch.ones_like)
    assert torch.isfinite(low).all() and float(low.abs().max()) < 1e-12
    high, w2 = changed(A(heads=4, kv_heads=2, dim=1, vdim=5, chunk=20, dims=0, scale=95.0), q_norm=torch.ones_like, k_norm=torch.ones_like, q=torch.zeros_like, k=torch.zeros_like,
                       q_b=torch.ones_like, k_b=torch.ones_like)
    assert torch.isfinite(high).all() and rel(high, w2) < 3e-5


def standout(j):
    """Makes token j's key the one every query looks for: the first input column is one for every token and the queries read only it (all
    queries of a key/value head are one vector), the keys do not read it, token j's row is solved so that its keys are those vectors, and
    every other row is made orthogonal to what the keys would need.  Norm weights of one and no biases on q and k (and, in the descriptions
    used with it, no rotation)."""
    def tweak(W, h, m):
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        g = torch.Generator().manual_seed(99)
        c = torch.randn(G, d, generator=g)
        c = c / c.square().mean(-1, keepdim=True).sqrt()
        W["q"] = torch.zeros_like(W["q"])
        W["q"][:, 0] = c.repeat_interleave(H // G, 0).reshape(-1)
        W["k"][:, 0] = 0
        for n in ("q", "k"):
            W[n + ".b"], W[n + ".norm"] = torch.zeros_like(W[n + ".b"]), torch.ones_like(W[n + ".norm"])
        a = torch.stack([W["k"][i * d:(i + 1) * d].double().T @ c[i].double() for i in range(G)], 1)
        basis = torch.linalg.qr(a).Q
        for i in range(h.shape[0]):
            h[i, 0] = 0.0
            if i == j:
                h[i] = torch.linalg.lstsq(W["k"].double(), c.reshape(-1, 1).double()).solution.reshape(-1).to(h.dtype)
            else:
                h[i] = (h[i].double() - basis @ (basis.T @ h[i].double())).to(h.dtype)
            h[i, 0] = 1.0
    return tweak


SHARP = dict(heads=4, kv_heads=2, dim=6, dims=0)


@gpu
@pytest.mark.parametrize("chunk", [1, 2, 7, 32, 33, 40])
@pytest.mark.parametrize("decode", [False, True])
def test_chunk_edge_with_a_key_that_stands_out(chunk, decode):
    """every query looks for token j's key, the second token of a chunk: the rows from j to the end of that chunk find it, the last row of the
    chunk before and the first of the chunk after do not.  Page size 4 puts the edges on and off page borders; a chunk one longer or
    shorter must differ."""
    j = 2 * chunk + min(1, chunk - 1)
    n = 4 * chunk + 3
    got, want = mixer_alone(A(chunk=chunk, scale=4.0, **SHARP), torch.float32, n, 4, [j + 1] + [1] * n if decode else [n], tweak=standout(j), width=40)
    assert rel(got, want) < 1e-4
    edges = (2 * chunk - 1, 2 * chunk, j, 3 * chunk - 1, 3 * chunk, 3 * chunk + 1)
    for r in edges:
        assert rel(got[r], want[r]) < 1e-4
    for other in (chunk + 1, max(1, chunk - 1)):
        if other != chunk:
            _, shifted = mixer_alone(A(chunk=other, scale=4.0, **SHARP), torch.float32, n, 4, [n], tweak=standout(j), width=40)
            assert max(rel(shifted[r], want[r]) for r in edges) > 1e-2      # the test bites


@gpu
def test_far_key_among_hundreds_and_the_split_path():
    """token 3's key is the one every query looks for; 600 tokens later (one chunk, pages of 16) each decoded token still finds it.  A
    single decoded token on a long range cuts the range into several parts."""
    from ktransformers_b200.operators.attention import softmax_attention_splits
    assert softmax_attention_splits(4, 2, 600, 1) > 1
    got, want = mixer_alone(A(chunk=4096, scale=4.0, **SHARP), torch.float32, 600, 16, [590] + [1] * 10, tweak=standout(3), width=40)
    assert rel(got, want) < 1e-4 and rel(got[-10:], want[-10:]) < 1e-4
    _, blind = mixer_alone(A(chunk=300, scale=4.0, **SHARP), torch.float32, 600, 16, [600], tweak=standout(3), width=40)
    assert rel(blind[-10:], want[-10:]) > 1e-2                   # the test bites
    got_b, _ = mixer_alone(A(chunk=4096, scale=4.0, **SHARP), torch.bfloat16, 600, 16, [590] + [1] * 10, tweak=standout(3), width=40)
    assert rel_rows(got_b, want, 0.9) < 6e-2 and rel(got_b[-10:], want[-10:]) < 6e-2


@gpu
@pytest.mark.parametrize("desc", [A(heads=4, kv_heads=2, dim=16, vdim=16, chunk=40), A(heads=8, kv_heads=1, dim=32, vdim=48, chunk=33, dims=32), A(heads=6, kv_heads=2, dim=64, vdim=32, chunk=1000, dims=16),
                                  A(heads=20, kv_heads=1, dim=128, vdim=128, chunk=64, dims=64), A(heads=3, kv_heads=3, dim=48, vdim=96, chunk=1)])
def test_tensor_core_attention_path(desc):
    """bf16 with head sizes that are multiples of 16: the tensor-core tiles against the restatement and against the CUDA-core kernel"""
    for portions in ([150], [70, 3, 2, 40, 1, 34], [130] + [1] * 20):
        got, want = mixer_alone(desc, torch.bfloat16, 150, 16, portions, width=160)
        plain, _ = mixer_alone(desc, torch.bfloat16, 150, 16, portions, width=160, tensor_path=False)
        assert rel_rows(got, want, 0.95) < 4e-2 and rel_rows(got, plain, 0.95) < 4e-2


@gpu
@pytest.mark.parametrize("chunk", [1, 31, 32, 33, 65])
@pytest.mark.parametrize("decode", [False, True])
def test_tensor_core_chunk_edges_inside_and_between_key_tiles(chunk, decode):
    """(the keys that are not looked for score zero up to bf16 rounding of their rows, times the scale: rows that average over such keys carry a
    few percent of noise)"""
    kw = dict(heads=4, kv_heads=2, dim=16, vdim=16, scale=2.0, dims=0)
    j = 2 * chunk + min(1, chunk - 1)
    n = 4 * chunk + 3
    got, want = mixer_alone(A(chunk=chunk, **kw), torch.bfloat16, n, 16, [j + 1] + [1] * n if decode else [n], tweak=standout(j), width=96)
    edges = (2 * chunk - 1, 2 * chunk, j, 3 * chunk - 1, 3 * chunk, 3 * chunk + 1)
    for r in edges:
        assert rel(got[r], want[r]) < 0.1
    for other in (chunk + 1, max(1, chunk - 1)):
        if other != chunk:
            _, shifted = mixer_alone(A(chunk=other, **kw), torch.bfloat16, n, 16, [n], tweak=standout(j), width=96)
            assert max(rel(shifted[r], want[r]) for r in edges) > 0.2


RET_SHAPES = [R(), R(heads=1, dim=1, vdim=1, dims=0), R(heads=2, dim=7, vdim=33, dims=4), R(heads=3, dim=20, vdim=70), R(heads=2, dim=128, vdim=64, dims=64), R(heads=5, dim=16, vdim=16, dims=6),
              R(heads=2, dim=130, vdim=300), R(heads=1, dim=256, vdim=40), R(heads=4, dim=12, vdim=8, decay=[1.0, 0.001, 0.5, 0.9999])]


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("desc", RET_SHAPES)
def test_retention_alone(dtype, tol, desc):
    """whole, in portions down to one and two tokens (on, before and after the scan's staging edges and the 64-token chunks), and decoded"""
    err = rel if dtype == torch.float32 else rel_rows
    if desc["mixer"]["dim"] == 1:                                # a head of one column is its sign times one
        tol = max(tol, 1e-3)
    whole, want = mixer_alone(desc, dtype, 150, 8, [150])
    assert err(whole, want) < tol and err(whole[:4], want[:4]) < tol
    for portions in ([33, 1, 1, 2, 31, 16, 3, 2], [64, 65, 1], [1], [2], [17, 15, 16]):
        got, _ = mixer_alone(desc, dtype, 150, 8, portions)
        assert err(got, want) < tol and err(got, whole) < tol


def retention_call(form, H, d, dv, dims, layout, lens, rds, decay, pos0, seed=0):
    """one call into the library on bf16 rows (dtype of the projections), returning (normed and gated output or plain o, states)"""
    from ktransformers_b200 import native
    lib, st = native.seq_lib(), torch.cuda.current_stream().cuda_stream
    g = torch.Generator().manual_seed(seed)
    T, w = sum(lens), 2 * H * d + 2 * H * dv
    proj = torch.randn(T, w, generator=g).bfloat16()
    before = torch.randn(H, d, dv, generator=g)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    pos = torch.cat([torch.arange(p, p + n) for p, n in zip(pos0, lens)]).int()
    inv = 100.0 ** (-2.0 * torch.arange(max(1, dims // 2)).double() / max(1, dims))
    seqs = torch.tensor([starts, lens, rds, [7 + i for i in range(len(lens))]], dtype=torch.int32).cuda()
    state = torch.zeros(20, H * d * dv + 4)
    state[2, :H * d * dv] = before.reshape(-1)
    dev = [t.cuda() for t in (proj, pos, inv, state, torch.tensor(decay).float(), torch.tensor([x - float(torch.tensor(x).float()) for x in decay]), torch.tensor([math.log2(x) for x in decay]))]
    turn = torch.empty(T, max(1, dims // 2), 2, device="cuda")
    if dims:
        native.check_seq(lib.ktb200_turn_table(dev[1].data_ptr(), dev[2].data_ptr(), dims // 2, turn.data_ptr(), T, st))
    a = native.RetentionParams(proj=dev[0].data_ptr(), proj_stride=w, q_off=0, k_off=H * d, v_off=2 * H * d, g_off=2 * H * d + H * dv, heads=H, dim=d, vdim=dv, rot_dims=dims, rot_layout=layout,
                               turn=turn.data_ptr(), k_scale=0.3, decay=dev[4].data_ptr(), decay_low=dev[5].data_ptr(), log2_decay=dev[6].data_ptr(), eps=1e-4, seqs=seqs.data_ptr(),
                               seqs_stride=len(lens), n_seqs=len(lens), state=dev[3].data_ptr(), state_stride=dev[3].stride(0))
    if form == "scan":
        y = torch.full((T, H * dv), float("nan"), device="cuda")
        native.check_seq(lib.ktb200_retention_scan(C.byref(a), y.data_ptr(), 30, st))
    else:
        y = torch.full((T, H * dv), float("nan"), device="cuda", dtype=torch.bfloat16)
        if form == "step":
            native.check_seq(lib.ktb200_retention_step(C.byref(a), y.data_ptr(), 30, st))
        else:
            ws = torch.full((lib.ktb200_retention_chunk_workspace(H, d, dv, T, len(lens)),), 255, dtype=torch.uint8, device="cuda")      # (NaNs)
            native.check_seq(lib.ktb200_retention_chunk(C.byref(a), y.data_ptr(), T, ws.data_ptr(), ws.numel(), 30, st))
    p = proj.double()
    head = lambda lo, n: p[:, lo:lo + H * n].reshape(T, H, n)
    def rot(x):
        if layout == 1:
            return torch.cat([O.rotated_halves(x[i:i + 1], pos[i:i + 1], 100.0, dims) for i in range(T)]) if dims else x
        perm = list(range(0, dims, 2)) + list(range(1, dims, 2)) + list(range(dims, x.shape[-1]))      # neighbouring columns as halves
        out = x.clone()
        out[..., perm] = O.rotated_halves(x[..., perm], pos, 100.0, dims)
        return out
    q, k, v, gate = rot(head(0, d)), rot(head(H * d, d)) * 0.3, head(2 * H * d, dv), p[:, 2 * H * d + H * dv:]
    want, states = [], []
    for lo, n, rd in zip(starts, lens, rds):
        o, S = O.retention(q[lo:lo + n], k[lo:lo + n], v[lo:lo + n], decay, before.double() if rd >= 0 else torch.zeros(H, d, dv).double())
        want.append(o)
        states.append(S)
    want = torch.cat(want)
    out = want.reshape(T, H * dv) if form == "scan" else O.rms(want, 1e-4).reshape(T, H * dv) * O.silu(gate)
    return y.cpu(), dev[3].cpu()[:, :H * d * dv], out, states


RET_CHUNK = [(4, 16, 16, 16, 1), (2, 128, 128, 128, 1), (3, 48, 112, 40, 1), (2, 64, 64, 24, 1), (2, 80, 32, 6, 1), (1, 32, 128, 0, 1), (2, 96, 48, 32, 0), (2, 128, 16, 8, 1)]


@gpu
@pytest.mark.parametrize("H,d,dv,dims,layout", RET_CHUNK)
@pytest.mark.parametrize("slow", [False, True])
def test_retention_forms_on_bf16_rows(H, d, dv, dims, layout, slow):
    """outputs and states of the chunked form and of the scan against the restatement: portions that end on, before and after the 64-token chunk
    edge, one of them starting from a state, late positions; fast decays (a state that is gone within a chunk) and slow ones"""
    lens, rds = [64, 65, 190, 1, 15, 128, 2], [-1, 2, -1, -1, -1, -1, -1]
    decay = [0.9999 - 0.002 * h for h in range(H)] if slow else [0.3 + 0.6 * h / max(1, H) for h in range(H)]
    pos0 = [0, 1000, 0, 0, 0, 0, 0]
    for form, tol, st_tol in (("chunk", 2e-2, 5e-4), ("scan", 2e-5, 2e-5)):
        y, state, want, states = retention_call(form, H, d, dv, dims, layout, lens, rds, decay, pos0)
        assert rel_rows(y, want, 0.99) < tol
        for i, S in enumerate(states):
            assert rel(state[7 + i], S.reshape(-1)) < st_tol


@gpu
@pytest.mark.parametrize("H,d,dv,dims,layout", RET_CHUNK + [(2, 7, 5, 4, 1), (3, 130, 300, 64, 1), (1, 3, 1, 2, 0), (80, 16, 256, 16, 1), (1, 8, 1100, 8, 1)])
@pytest.mark.parametrize("n", [1, 9])
def test_retention_step_with_blocks_of_a_head_as_a_cluster(H, d, dv, dims, layout, n):
    """decode steps: one column block per head and several (the norm's sum crosses them), states read and fresh"""
    decay = [0.5 + 0.45 * h / H for h in range(H)]
    y, state, want, states = retention_call("step", H, d, dv, dims, layout, [1] * n, [2 if i % 2 == 0 else -1 for i in range(n)], decay, [7 * i for i in range(n)])
    assert rel(y, want) < 2e-2
    for i, S in enumerate(states):
        assert rel(state[7 + i], S.reshape(-1)) < 2e-5


@gpu
def test_each_ingredient_of_the_retention_matters():
    desc = R(heads=4, dim=6, vdim=5)
    got, want = mixer_alone(desc, torch.float32, 40, 8, [40])
    assert rel(got, want) < 3e-5
    for kw in (dict(g=torch.zeros_like), dict(g=lambda x: -x), dict(q=lambda x: x.flip(0)), dict(v=lambda x: x.flip(0))):
        g2, w2 = changed(desc, **kw)
        assert rel(g2, w2) < 3e-5 and rel(w2, want) > 1e-2
    g2, w2 = changed(desc, v=lambda x: 50.0 * x)                  # unit-rms outputs: the values' length does not count (but for eps)
    assert rel(g2, w2) < 3e-5 and rel(w2, want) < 1e-2
    for other in (R(heads=4, dim=6, vdim=5, dims=4), R(heads=4, dim=6, vdim=5, base=30.0), R(heads=4, dim=6, vdim=5, decay=[0.7, 0.9, 0.95, 0.99]),
                  R(heads=4, dim=6, vdim=5, decay=list(reversed(desc["mixer"]["decay"])))):
        g2, w2 = mixer_alone(other, torch.float32, 40, 8, [40])
        assert rel(g2, w2) < 3e-5 and rel(w2, want) > 1e-2
    # the scale of k shows against eps: outputs near zero
    small = lambda x: 3e-3 * x
    g2, w2 = changed(desc, v=small)
    assert rel(g2, w2) < 3e-5
    _, w3 = changed(desc, v=small, k=lambda x: x * 6 ** 0.5)
    assert rel(w3, w2) > 1e-2


SCAN_SHAPES = [S(), S(inner=1, state=1, dt_rank=1, conv=1), S(inner=33, state=4, dt_rank=2, conv=2), S(inner=130, state=8, dt_rank=5, conv=3), S(inner=64, state=16, dt_rank=8, conv=4),
               S(inner=40, state=33, dt_rank=3, conv=5), S(inner=24, state=64, dt_rank=4, conv=4), S(inner=10, state=100, dt_rank=4, conv=3), S(inner=12, state=256, dt_rank=7, conv=2), S(inner=9, state=6, conv=6)]


@gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("desc", SCAN_SHAPES)
def test_selective_scan_alone(dtype, tol, desc):
    """whole, in portions down to one and two tokens (shorter than the filter; on, before and after the scan's staging edges), and decoded"""
    err = rel if dtype == torch.float32 else rel_rows
    whole, want = mixer_alone(desc, dtype, 150, 8, [150])
    assert err(whole, want) < tol and err(whole[:4], want[:4]) < tol
    for portions in ([33, 1, 1, 2, 31, 16, 3, 2], [64, 65, 1], [1], [2], [17, 15, 16]):
        got, _ = mixer_alone(desc, dtype, 150, 8, portions)
        assert err(got, want) < tol and err(got, whole) < (2e-5 if dtype == torch.float32 else tol)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("I,N", [(37, 16), (64, 16), (64, 5), (200, 1), (16, 128), (5, 200), (8, 200), (300, 32), (36, 8), (132, 4), (20, 64)])
@pytest.mark.parametrize("portions", [True, False])
@pytest.mark.parametrize("rate", [-7.0, 0.0, 3.0])
def test_selective_scan_kernel_on_rows(dtype, I, N, rate, portions):
    """the recurrence, skip and gate against the restatement, outputs and states: portions on, before and after the staging edge, one starting from a
    state; decays from almost one to almost zero, steps from almost none to past the soft-plus's straight part"""
    from ktransformers_b200 import native
    lib, lens, g = native.seq_lib(), [16, 17, 70, 1, 3, 32] if portions else [1] * 6, torch.Generator().manual_seed(I * N)
    T, code = sum(lens), 30 if dtype == torch.bfloat16 else 0
    rn = lambda *s: torch.randn(*s, generator=g)
    pad, lo_b = (4, 4) if I % 4 == 0 and N % 4 == 0 else (3, 1)      # rows in groups of four, or not
    x, dtl, bc, z = rn(T, I).to(dtype), (2.0 * rn(T, I)).to(dtype), rn(T, 2 * N + pad).to(dtype), rn(T, I + pad).to(dtype)
    dtl[::7], dtl[3::11] = -9.0, 25.0
    bias, al, D, before = rn(I), torch.full((I, N), rate) + 0.3 * rn(I, N), rn(I), rn(I, N)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    seqs = torch.tensor([starts, lens, [-1, 2, -1, -1, -1, -1], [7 + i for i in range(len(lens))]], dtype=torch.int32).cuda()
    state = torch.zeros(20, I * N + pad)
    state[2, :I * N] = before.reshape(-1)
    dev = [t.cuda() for t in (x, dtl, bc, z, bias, -torch.exp(al), D, state)]
    y = torch.full((T, I), float("nan"), dtype=dtype, device="cuda")
    a = native.SelectiveScanParams(x=dev[0].data_ptr(), dt_logit=dev[1].data_ptr(), b=dev[2][:, lo_b:].data_ptr(), c=dev[2][:, N + lo_b:].data_ptr(), z=dev[3].data_ptr(), dt_stride=I,
                                   bc_stride=2 * N + pad, z_stride=I + pad, dt_bias=dev[4].data_ptr(), a=dev[5].data_ptr(), d_skip=dev[6].data_ptr(), inner=I, state_size=N, seqs=seqs.data_ptr(),
                                   seqs_stride=len(lens), n_seqs=len(lens), state=dev[7].data_ptr(), state_stride=dev[7].stride(0))
    native.check_seq(lib.ktb200_selective_scan(C.byref(a), y.data_ptr(), T, code, torch.cuda.current_stream().cuda_stream))
    xd, bcd = x.double(), bc.double()
    dt = O.softplus(dtl.double() + bias.double())
    for i, (lo, n) in enumerate(zip(starts, lens)):
        r = slice(lo, lo + n)
        S0 = before.double() if i == 1 else torch.zeros(I, N).double()
        want, st = O.selective_scan(xd[r], dt[r], -torch.exp(al.double()), bcd[r, lo_b:N + lo_b], bcd[r, N + lo_b:2 * N + lo_b], D.double(), S0)
        want = want * O.silu(z[r, :I].double())
        assert rel(y[r], want) < (1e-2 if dtype == torch.bfloat16 else 2e-5)
        assert rel(dev[7][7 + i, :I * N], st.reshape(-1)) < 2e-5


@gpu
def test_each_ingredient_of_the_selective_scan_matters():
    desc = S(inner=14, state=5, dt_rank=3, conv=3)
    got, want = mixer_alone(desc, torch.float32, 40, 8, [40])
    assert rel(got, want) < 3e-5
    split = lambda f: (lambda x: torch.cat([x[:14], f(x[14:])]))
    for k, f in (("conv.b", torch.zeros_like), ("conv", lambda x: x.flip(1)), ("dt.b", lambda x: x + 1), ("dt", torch.zeros_like), ("A_log", lambda x: x - 1), ("A_log", lambda x: x.flip(1)),
                 ("A_log", lambda x: x.flip(0)), ("D", torch.zeros_like), ("in", split(lambda z: -z)), ("x", lambda x: torch.cat([x[:3], x[8:], x[3:8]])), ("x", lambda x: torch.cat([0 * x[:3], x[3:]]))):
        def tweak(W, h, m):
            W[k] = f(W[k])
        g2, w2 = mixer_alone(desc, torch.float32, 40, 8, [40], tweak=tweak)
        assert rel(g2, w2) < 3e-5 and rel(w2, want) > 1e-2, k
    def large(W, h, m):
        W["dt.b"] += 40.0
    g2, w2 = mixer_alone(desc, torch.float32, 40, 8, [40], tweak=large)      # large steps: the soft-plus is the identity there, decays vanish
    assert torch.isfinite(g2).all() and rel(g2, w2) < 3e-5


@gpu
@pytest.mark.parametrize("kind", ["scan", "retention", "retention tiles"])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 5e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("decode", [False, True])
def test_state_carries_a_far_token(kind, dtype, tol, decode):
    """a loud token whose trace a slow decay keeps for 300 steps, in one prompt and decoded; without the token, or with a faster decay, the
    last rows differ"""
    slow = {"scan": S(inner=32, state=8, dt_rank=4), "retention": R(heads=3, dim=12, vdim=8, decay=[0.9995, 0.999, 0.9999], dims=0),
            "retention tiles": R(heads=3, dim=16, vdim=32, decay=[0.9995, 0.999, 0.9999], dims=0)}[kind]

    def make(loud, fast):
        def tweak(W, h, m):
            if kind == "scan":
                W["A_log"] = torch.full_like(W["A_log"], -1.0 if fast else -7.0)
                W["D"] = torch.zeros_like(W["D"])
            if loud:
                h[4] *= 12.0
        desc = json.loads(json.dumps(slow))
        if fast and kind != "scan":
            desc["mixer"]["decay"] = [0.9, 0.8, 0.95]
        return desc, tweak
    desc, tweak = make(True, False)
    got, want = mixer_alone(desc, dtype, 310, 8, [40] + [1] * 270 if decode else [310], tweak=tweak)
    assert rel_rows(got, want, 0.95) < tol and rel_rows(got[-20:], want[-20:], 0.95) < tol
    for other in (make(False, False), make(True, True)):
        _, without = mixer_alone(other[0], dtype, 310, 8, [310], tweak=other[1])
        assert rel(without[-20:], want[-20:]) > 0.1


@gpu
def test_thousands_of_tokens_in_32_bit_keep_their_slow_states():
    """slow channels and decays that are not 32-bit numbers: the rounding of a decay must not add up along the tokens"""
    def slow(W, h, m):
        if "A_log" in W:
            W["A_log"] = torch.full_like(W["A_log"], -6.0) + 0.1 * W["A_log"]
            W["dt"] *= 0.05
    for desc in (S(inner=8, state=4, dt_rank=2, conv=2), R(heads=2, dim=4, vdim=4, decay=[0.9996123, 0.99991234], dims=2)):
        got, want = mixer_alone(desc, torch.float32, 3000, 64, [3000], tweak=slow, width=16)
        assert rel(got[-200:], want[-200:]) < 1e-5


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_decode_and_prompt_portions_in_one_launch(dtype):
    """portions of one, two and many tokens of different sequences in one batch: windows and states of neighbours do not mix"""
    from ktransformers_b200.models.configuration_lipadra import MIXER_SPECS
    from ktransformers_b200.models.custom_cache import PagedStateCache
    from ktransformers_b200.models.modeling_lipadra import MIXERS
    g = torch.Generator().manual_seed(3)
    rn = lambda *s, k=1.0: torch.randn(*s, generator=g) * k
    lin = lambda o, i, s=1.0: rn(o, i, k=s / i ** 0.5)
    width = 24
    for desc in (S(inner=20, state=12, conv=4), R(heads=2, dim=16, vdim=16, dims=8), R(), A(chunk=50), A(heads=4, kv_heads=2, dim=16, vdim=16, chunk=30)):
        kind, m = desc["type"], desc["mixer"]
        spec = MIXER_SPECS[kind].from_dict(m)
        W = {k: v.to(dtype) for k, v in U.WEIGHTS[kind](rn, lin, "", m, width).items()}
        op = MIXERS[kind](width, spec, 1e-5, dtype=dtype)
        op.load(DictLoader(W), "")
        h = {i: rn(n, width).to(dtype) for i, n in (("a", 90), ("b", 40), ("c", 71), ("d", 3))}
        widths = ([spec.cache_row_width()], [spec.state_width()])
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


@gpu
def test_one_table_of_turns_per_rotation_and_step():
    from ktransformers_b200.models.configuration_lipadra import RetentionSpec
    from ktransformers_b200.models.custom_cache import PagedStateCache
    cache = PagedStateCache([0], [0], 64, 2, "cuda", page_size=8)
    batch = cache.build_batch([("a", [0] * 5, []), ("b", [0] * 3, [])])
    tables = []
    for base, dims in ((500.0, 6), (500.0, 6), (500.0, 4), (70.0, 6)):
        rot = RetentionSpec.from_dict(R(dim=6, dims=dims, base=base)["mixer"]).rot
        t = batch.turn_table(rot, rot.inv_freq("cuda"))
        angles = torch.tensor([0, 1, 2, 3, 4, 0, 1, 2]).double()[:, None] * base ** (-2.0 * torch.arange(dims // 2).double() / dims)
        assert rel(t[..., 0], torch.cos(angles)) < 1e-6 and rel(t[..., 1], torch.sin(angles)) < 1e-6
        tables.append(t.data_ptr())
    assert tables[0] == tables[1] and len(set(tables)) == 3


# ------------------------------------------------------------------------------------------------ whole model (GPU)
@gpu
@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_prompt_decode_and_portions_agree_with_the_restatement(tmp_path, dtype, tol):
    cfg = U.config(MIXED, alpha=3.0 if dtype == "float32" else 8.0)
    eng, om = serve(tmp_path, cfg, dtype, max_tokens=128, max_slots=2, page_size=4)
    t = toks(75)
    want = oracle_logits(om, t)
    err = rel if dtype == "float32" else (lambda a, b: rel_rows(a, b, 0.7))
    whole = run_steps(eng, cut("w", t, [75]))["w"]
    assert err(whole, want) < tol
    assert err(whole[:4], want[:4]) < tol                       # the first tokens of a sequence
    for sizes in ([1], [2], [3, 2, 7, 1, 5], [20, 2, 2, 1]):
        got = run_steps(eng, cut("p", t, sizes))["p"]
        assert err(got, want) < tol
        assert err(got, whole) < (5e-5 if dtype == "float32" else tol)   # the cut does not matter beyond rounding


@gpu
def test_whole_model_in_bf16_on_tensor_core_head_sizes(tmp_path):
    """head sizes that are multiples of 16: bf16 attention and retention run on the tensor cores inside a whole model, 150 tokens over several tiles
    and chunks, whole, in portions and with a decoded tail"""
    f = dict(ff=32, experts=5, identity=1, top=2, groups=(2, 1), shared=48)
    layers = [(U.attention(heads=6, kv_heads=2, dim=32, vdim=48, chunk=40, dims=16), U.moe(**f)), (U.retention(heads=3, dim=32, vdim=48, dims=32), U.moe(**f)), 0, (U.scan(inner=96, state=16, dt_rank=8), None), 1]
    cfg = U.config(layers, width=64, vocab=90, alpha=6.0)
    eng, om = serve(tmp_path, cfg, "bfloat16", seed=3, max_tokens=512, max_slots=2, page_size=16)
    t = toks(150, 90, seed=9)
    want = oracle_logits(om, t)
    for k, sizes in enumerate(([150], [70, 3, 2, 40, 1, 34], [130] + [1] * 20)):
        assert rel_rows(run_steps(eng, cut(("m", k), t, sizes))[("m", k)], want, 0.7) < BF16_TOL


@gpu
def test_residual_stream_after_every_layer(tmp_path):
    cfg = U.config(MIXED)
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=64, max_slots=2, page_size=8)
    t = toks(11, seed=2)
    want, got = [], []
    logits = om.forward(t, om.new_state(), want)
    mine = eng.model(eng.cache.build_batch([("r", t, [0, 10])]), eng.cache, got)
    assert len(got) == len(want) == 9
    for a, b in zip(got, want):
        assert rel(a, b) < 1e-4
    assert rel(mine, logits[[0, 10]]) < F32_TOL


@gpu
def test_model_constants_matter(tmp_path):
    """the restatement with another alpha, eps, router scale, group count or owner of a layer's tensors differs"""
    cfg = U.config(MIXED, eps=1e-2)
    eng, om = serve(tmp_path, cfg, "float32", seed=1, max_tokens=64, max_slots=2, page_size=8)
    t, w = toks(20, seed=4), U.weights(cfg, 1, torch.float32)
    want = oracle_logits(om, t)
    assert rel(run_steps(eng, cut("a", t, [13, 2, 1]))["a"], want) < F32_TOL
    others = [dict(cfg, postln_alpha=1.0), dict(cfg, norm={"eps": 1e-6})]
    for key, val in (("scale", 1.0), ("groups", {"count": 1, "keep": 1}), ("top", 1)):
        c = json.loads(json.dumps(cfg))
        for i in (0, 4):
            c["layers"][i]["mlp"]["router"][key] = val
        others.append(c)
    c = json.loads(json.dumps(cfg))
    c["layers"] = c["layers"][:6]                                # the shared layers run: without them the result is another
    others.append(c)
    for c in others:
        assert rel(oracle_logits(O.Model(c, w, torch.float64), t), want) > 1e-3


@gpu
def test_other_sizes_and_layer_orders(tmp_path):
    one = dict(experts=1, identity=0, top=1, groups=(1, 1))
    cases = [
        ([(U.attention(heads=1, kv_heads=1, dim=2, vdim=2, chunk=3, dims=2), U.moe(ff=3, shared=2, **one))], dict(width=8)),                                                       # one small layer, one expert
        ([(U.retention(heads=1, dim=1, vdim=1, decay=[0.5], dims=0), None)], dict(width=4, alpha=1.0)),
        ([(U.scan(inner=1, state=1, dt_rank=1, conv=1), U.moe(ff=2, experts=1, identity=1, top=1, groups=(2, 1), scale=1.0, shared=0))], dict(width=6, alpha=0.5)),
        ([(U.attention(heads=16, kv_heads=4, dim=12, vdim=10, chunk=12, dims=8), U.moe(ff=20, experts=12, identity=4, top=4, groups=(4, 2))), (U.retention(heads=8, dim=4, vdim=9), None)] * 2 + [1, 0], dict(width=72, vocab=31)),
        ([(U.scan(inner=50, state=24, dt_rank=5, conv=5), U.moe(ff=5, experts=3, identity=0, top=3, groups=(1, 1), shared=1)), 0, 0, (U.attention(chunk=1), None)], dict(width=40)),
        ([(U.retention(), None), (U.retention(heads=5, dim=34, vdim=2), U.moe(ff=33, experts=2, identity=10, top=6, groups=(2, 2))), (U.attention(chunk=500, dims=0), U.moe(experts=4, identity=0, top=1, groups=(2, 1)))], dict(width=16, eps=1e-3)),
        ([(U.scan(), None), (U.scan(inner=200, state=130, dt_rank=17), None)], dict(width=14, vocab=7))]
    for k, (layers, kw) in enumerate(cases):
        cfg = U.config(layers, **kw)
        eng, om = serve(tmp_path, cfg, "float32", seed=10 + k, max_tokens=64, max_slots=2, page_size=8)
        t = toks(30, cfg["vocab"], seed=k)
        assert rel(run_steps(eng, cut("a", t, [13, 2, 1]))["a"], oracle_logits(om, t)) < F32_TOL, k


@gpu
@pytest.mark.parametrize("seed", range(10))
def test_drawn_configurations(tmp_path, seed):
    """sizes, layer order and constants drawn per seed: one prompt whole, in uneven portions, and with a decoded tail"""
    r = random.Random(seed)
    width = r.choice([16, 40, 136, 320])
    layers = []
    for n in range(r.randint(1, 5)):
        if n and r.random() < 0.3:
            layers.append(r.randrange(n))
            continue
        kind = r.choice("ars")
        if kind == "a":
            G, d = r.choice([1, 2, 4]), r.choice([4, 6, 24, 64])
            m = U.attention(heads=G * r.choice([1, 2, 5]), kv_heads=G, dim=d, vdim=r.choice([5, 8, 80]), scale=r.choice([None, 0.11, 0.6]), chunk=r.choice([1, 5, 31, 32, 33, 64, 100, 1000]),
                            dims=r.choice([0, 2, 4, d]), base=r.choice([50.0, 10000.0, 3e6]))
        elif kind == "r":
            H, d = r.choice([1, 2, 5]), r.choice([3, 8, 16, 80])
            m = U.retention(heads=H, dim=d, vdim=r.choice([1, 8, 32, 90]), decay=[r.choice([0.3, 0.9, 0.99, 0.9993]) for _ in range(H)], dims=r.choice([0, 2, d // 2 * 2]), base=r.choice([50.0, 1e5]))
        else:
            m = U.scan(inner=r.choice([7, 32, 96]), state=r.choice([1, 6, 16, 40]), dt_rank=r.choice([1, 4, 9]), conv=r.choice([1, 2, 3, 4, 5]))
        groups = r.choice([(1, 1), (2, 1), (2, 2), (4, 3)])
        per = r.choice([1, 2, 5])
        outputs = groups[0] * per
        identity = r.randint(0, outputs - 1)
        f = U.moe(ff=r.choice([8, 24, 100]), experts=outputs - identity, identity=identity, top=r.randint(1, min(groups[1] * per, 6)), groups=groups, scale=r.choice([1.0, 3.0]), shared=r.choice([0, 1, 8, 50]))
        layers.append((m, None if r.random() < 0.2 else f))
    cfg = U.config(layers, vocab=r.choice([31, 77, 1000]), width=width, eps=r.choice([1e-6, 1e-5, 1e-3]), alpha=r.choice([1.0, 3.1, 7.0]))
    eng, om = serve(tmp_path, cfg, "float32", seed=seed, max_tokens=256, max_slots=2, page_size=r.choice([4, 16, 64]))
    t = toks(r.choice([40, 90, 120]), cfg["vocab"], seed=seed)
    want = oracle_logits(om, t)
    for k, sizes in enumerate(([len(t)], [3, 17, 2, 1, 33, 2, 64], [len(t) - 20] + [1] * 20)):
        assert rel(run_steps(eng, cut(("d", k), t, sizes))[("d", k)], want) < F32_TOL


@gpu
def test_only_wanted_rows_and_none(tmp_path):
    """the last layer runs its feed-forward for the rows asked for only; a portion that asks for none still leaves its caches and states"""
    cfg = U.config(MIXED + [(U.attention(chunk=16), U.moe())])
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=64, max_slots=2, page_size=8)
    t = toks(30, seed=6)
    want = oracle_logits(om, t)
    assert eng.step([("a", t[:9], [])]).shape == (0, 50)
    got = eng.step([("a", t[9:20], [10, 3])])
    assert rel(got, want[[19, 12]]) < F32_TOL
    assert eng.step([("a", t[20:21], [])]).shape == (0, 50)
    assert rel(eng.step([("a", t[21:], [8, 0])], ["a"]), want[[29, 21]]) < F32_TOL


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
@pytest.mark.parametrize("recurrent_only", [False, True])
def test_long_decode_over_reused_pages_and_slots(tmp_path, recurrent_only):
    """pages of 4 and 2 slots: sequences come and go, pages and state rows are handed out again un-cleared, and a new sequence in a used
    slot must start from an empty state and an empty filter.  Every attention layer's mask is chunked, so the pages before the current chunk are
    given back while a sequence runs and its page table row wraps around; without attention layers no page is held for long."""
    layers = [(U.retention(), U.moe()), (U.scan(conv=3), None), 0]
    if not recurrent_only:
        layers = [(U.attention(chunk=9), U.moe()), (U.attention(heads=2, kv_heads=2, dim=8, vdim=8, chunk=21), None), 0] + [(U.retention(), U.moe()), (U.scan(conv=3), None), 3]
    cfg = U.config(layers)
    eng, om = serve(tmp_path, cfg, "float32", max_tokens=48, max_slots=2, page_size=4)
    assert eng.cache.chunks == ([1] if recurrent_only else [9, 21])
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
    cfg = U.config(MIXED, vocab=41, alpha=5.0 if dtype == "float32" else 15.0)
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
    rows = []
    for n, ref in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, 41))
        assert got.shape == ref.shape
        rows.append((got, ref))
    got, ref = (torch.cat(x) for x in zip(*rows))
    assert (rel(got, ref) if dtype == "float32" else rel_rows(got, ref, 0.7)) < tol
