"""Sanarax on the GPU: every new kernel option alone against the plain kernel statements (themselves held to the plain
implementation by the CPU tests), attention with planted keys at every edge of the window and of the kept first tokens,
then whole models through the step function, the replay program and the engine."""
import numpy as np
import pytest
import torch

import helpers
import sanarax_models as sm
from plain import plain_sanarax as P
from plain.plain_kernels import PlainKernels

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def sanarax_dirs(tmp_path_factory):
    out = {}
    for i, (name, (raw, page)) in enumerate(sm.configs().items()):
        out[name] = (sm.write_model(raw, tmp_path_factory.mktemp(f"sanarax_{name}"), seed=61 + i), page, raw)
    return out


def _partial(t, splits, g, dtype=torch.bfloat16):
    """`t` (float32) as a PartialSum: slices that add up to it."""
    from inferflux_b200.csrc.ops import PartialSum
    parts = [torch.randn(t.shape, generator=g) for _ in range(splits - 1)]
    return PartialSum(torch.stack([t - sum(parts)] + parts if parts else [t]).to(DEV).contiguous(), dtype)


def _cache(dtype, spec, page, device, tokens=400):
    from inferflux_b200.cache.manager import CacheManager
    pages = -(-tokens // page)
    return CacheManager([(spec, None)], page_size=page, num_pages=pages, max_seqs=4, max_seq_len=page * pages, dtype=dtype, device=device)


def _step_ctx(kernels, dtype, cache, spans, device):
    from inferflux_b200.engine.batch import StepContext, StepEntry
    entries, starts, slots = [], [], []
    for rid, n in spans:
        if rid not in cache:
            cache.add_request(rid)
        start = cache.length(rid)
        cache.reserve(rid, start + n)
        entries.append(StepEntry(rid, [0] * n, []))
        starts.append(start)
        slots.append(cache.slot(rid))
    ctx = StepContext.build(kernels, dtype, device, entries, starts, slots, cache.drain_table_updates())
    for g, (idx, page) in zip(cache.groups, ctx.table_updates):
        kernels.scatter_i32(g.table, idx, page)
    for (rid, n), s in zip(spans, starts):
        cache.commit(rid, s + n)
    return ctx


def _view(cache):
    from inferflux_b200.config.plan import ScheduleEntry
    return cache.view(ScheduleEntry(layer=0, cache=0))


def _rotary(base, dims, interleaved, dev):
    from inferflux_b200.parts.base import RotaryTable
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64).float()
    return RotaryTable(f.to(dev), dims, interleaved)


# ------------------------------------------------------------------ rows: values that are the keys, a gate per head

@pytest.mark.parametrize("dtype,tol", [(torch.float32, 5e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("nq,nkv,d,rot,inter,page", [(4, 2, 16, 8, False, 8), (6, 1, 8, 4, False, 4), (3, 3, 10, 2, False, 16), (5, 1, 14, 10, False, 4),
                                                     (12, 4, 64, 32, False, 16), (16, 2, 128, 128, False, 16), (8, 2, 112, 44, False, 16),
                                                     (20, 4, 80, 40, False, 8), (4, 4, 24, 6, True, 8)])
def test_values_from_keys_partial_rotation_and_head_gates(cuda_kernels, dtype, tol, nq, nkv, d, rot, inter, page):
    """Queries, both halves of the cache and the gates against the plain statement: few tokens (a cluster of blocks per token)
    and many, plain rows in both dtypes and K slices, with and without biases; parts of a head rotated whose halves are even
    and odd."""
    from inferflux_b200.parts.base import KVCacheSpec
    g = torch.Generator().manual_seed(nq * 100 + d)
    rnd = lambda *s: torch.randn(*s, generator=g)
    used = (nq + nkv) * d
    width = -(-(used + nq) // 8) * 8
    bias = 0.5 * rnd(used)
    spec = KVCacheSpec(nkv, -(-d // 8) * 8, None)
    caches = {"plain": _cache(F64, spec, page, "cpu"), "cuda": _cache(dtype, spec, page, DEV)}
    for step, (spans, kind) in enumerate((([("a", 37), ("b", 5)], "same"), ([("a", 1), ("b", 1)], "slices"), ([("b", 70)], "float"),
                                          ([("a", 1), ("b", 2), ("c", 1)], "slices"))):
        T = sum(n for _r, n in spans)
        rows = 2.0 * rnd(T, width)
        rows = rows.to(dtype) if kind == "same" else rows
        res = {}
        for name, kern, dev, dt in (("plain", PlainKernels(wide=True), "cpu", F64), ("cuda", cuda_kernels, DEV, dtype)):
            ctx = _step_ctx(kern, dt, caches[name], spans, dev)
            src = rows.double() if name == "plain" else (_partial(rows.float(), 5, g) if kind == "slices" else rows.to(DEV))
            q, back, gate = kern.row_norm_rope_append(src, 0, None if step == 2 else bias.to(dev), _rotary(90.0, rot, inter, dev), None, None,
                                                      nq, nkv, d, d, ctx, _view(caches[name]), v_from_k=True, gate_col=used)
            assert back is None and q.dtype == dt and gate.dtype == torch.float32 and tuple(gate.shape) == (T, nq)
            held = [_view(caches[name]).kv[list(caches[name].pages_of(r).values())].double().cpu() for r, _n in spans]
            res[name] = [q.double().cpu(), gate.double().cpu()] + held
        for a, b in zip(res["cuda"], res["plain"]):
            assert a.shape == b.shape and float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max())), (step, kind)
        assert float((res["cuda"][1] - res["plain"][1]).abs().max()) < 2e-6          # gates in float32 in both runs


# ------------------------------------------------------------------ latent rows and attention with a gate

@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,page", [(3, 12, 4, 10, 24, 8), (6, 32, 32, 40, 64, 16), (1, 16, 16, 8, 16, 4), (5, 7, 6, 5, 11, 16),
                                                          (16, 64, 64, 64, 256, 16), (20, 24, 16, 32, 112, 16), (4, 16, 0, 24, 48, 8)])
def test_latent_attention_with_a_gate(cuda_kernels, dtype, tol, heads, dim, rot, vdim, rank, page):
    """Rotated query parts, cached rows, gates and attention: a prompt, portions beside single tokens, single tokens over a
    long past (key splits and their merge); the tiled kernels and the per-token ones."""
    from inferflux_b200.parts.base import KVCacheSpec
    g = torch.Generator().manual_seed(heads * 100 + rank)
    rnd = lambda *s: torch.randn(*s, generator=g)
    spec = KVCacheSpec(1, rank + rot, None, planes=1)
    col0 = 5 * 8
    width = -(-(col0 + rank + rot + heads) // 8) * 8
    w, uk, uv = 1 + 0.3 * rnd(rank), rnd(heads * dim, rank) / rank ** 0.5, rnd(heads * vdim, rank) / rank ** 0.5
    if dtype == torch.bfloat16:
        uk, uv = uk.bfloat16().float(), uv.bfloat16().float()
    caches = {"plain": _cache(F64, spec, page, "cpu", 700), "cuda": _cache(dtype, spec, page, DEV, 700)}
    scale = 1.3 / (dim + rot) ** 0.5
    for spans in ([("a", 300)], [("a", 130), ("b", 9)], [("a", 1), ("b", 33)], [("a", 1), ("b", 1)]):
        T = sum(n for _r, n in spans)
        rows, q = (rnd(T, width) * 1.5).to(dtype), (rnd(T, heads * (dim + rot)) * 1.5).to(dtype)
        res = {}
        for name, kern, dev, dt in (("plain", PlainKernels(wide=True), "cpu", F64), ("cuda", cuda_kernels, DEV, dtype)):
            ctx = _step_ctx(kern, dt, caches[name], spans, dev)
            to = lambda t: t.double() if name == "plain" else t.to(dt).to(dev)
            rt = _rotary(70.0, rot, True, dev) if rot else None
            qq, gate = kern.latent_rope_append(to(rows), col0, rank, rot, w.to(dev), 1e-5, to(q).clone(), heads, dim, rt, ctx, _view(caches[name]),
                                               vdim=vdim, gate_col=col0 + rank + rot)
            out = kern.latent_attention(qq, to(uk), to(uv), None, heads, dim, vdim, rank, None, scale, ctx, _view(caches[name]), rot=rot, head_gate=gate)
            res[name] = [gate.double().cpu(), out.double().cpu()]
        assert float((res["cuda"][0] - res["plain"][0]).abs().max()) < 2e-6
        assert float((res["cuda"][1] - res["plain"][1]).abs().max()) <= tol * max(1.0, float(res["plain"][1].abs().max())), spans
    cuda_kernels.check_errors()


# ------------------------------------------------------------------ activated columns, the norm over all heads, squared ReLU

@pytest.mark.parametrize("T,width,acted", [(1, 9, 4), (7, 300, 211), (40, 1030, 1030), (200, 640, 480), (3, 12288, 9000), (5, 16, 0)])
def test_silu_on_columns_in_place_and_from_slices(cuda_kernels, T, width, acted):
    g = torch.Generator().manual_seed(width)
    rows = 6.0 * torch.randn(T, width, generator=g)
    want = PlainKernels(wide=True).silu_columns(rows, acted, None).double()
    plain = rows.clone().to(DEV)
    got = cuda_kernels.silu_columns(plain, acted, None)
    assert got.data_ptr() == plain.data_ptr() and float((got.double().cpu() - want).abs().max()) < 5e-6
    got = cuda_kernels.silu_columns(_partial(rows, 6, g, torch.float32), acted, None)
    assert got.dtype == torch.float32 and float((got.double().cpu() - want).abs().max()) < 2e-5
    far = torch.tensor([[-200.0, -90.0, 90.0, 200.0]], device=DEV)
    assert cuda_kernels.silu_columns(far, 4, None).tolist()[0][2:] == [90.0, 200.0] and float(far[0, :2].abs().max()) < 1e-30


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("C,groups", [(60, 1), (3, 1), (320, 1), (3072, 1), (96, 12), (64, 4)])
def test_gated_norm_with_a_sigmoid_gate(cuda_kernels, dtype, tol, C, groups):
    g = torch.Generator().manual_seed(C)
    y, wide, w = 2.0 * torch.randn(9, C, generator=g), 3.0 * torch.randn(9, C + 11, generator=g), 1 + 0.3 * torch.randn(C, generator=g)
    for first in (False, True):
        want = PlainKernels(wide=True).gated_groupnorm(y.double(), wide[:, 3:3 + C].double(), w, 1e-5, groups, first, F64, kind="sigmoid")
        got = cuda_kernels.gated_groupnorm(y.to(DEV), wide.to(DEV)[:, 3:3 + C], w.to(DEV), 1e-5, groups, first, dtype, kind="sigmoid")
        assert got.dtype == dtype and float((got.double().cpu() - want).abs().max()) <= tol * float(want.abs().max())


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 1.5e-2)])
@pytest.mark.parametrize("T,K,F", [(1, 72, 88), (5, 96, 200), (16, 64, 9600), (33, 320, 192), (150, 128, 10000), (160, 64, 40), (161, 320, 448),
                                   (300, 256, 128), (700, 72, 333), (200, 4200, 64), (3, 50, 33), (190, 50, 75)])
def test_squared_relu_product(cuda_kernels, dtype, tol, T, K, F):
    """Every way it is made: the weight-streaming kernel, K slices and the kernel that adds them, the many-rows kernel (whole
    tiles and edges), the library product with the activation kernel (long inner sizes, odd sizes), float32."""
    g = torch.Generator().manual_seed(T + K)
    a, w = torch.randn(T, K, generator=g).to(dtype), (1.5 / K ** 0.5 * torch.randn(F, K, generator=g)).to(dtype)
    want = PlainKernels(wide=True).linear_relu2(a.double(), w.double())
    got = cuda_kernels.linear_relu2(a.to(DEV), w.to(DEV))
    assert got.dtype == dtype and tuple(got.shape) == (T, F)
    assert float((got.double().cpu() - want).abs().max()) <= tol * max(1.0, float(want.abs().max()))
    assert bool((got >= 0).all()) and float((got == 0).float().mean()) > 0.3
    cuda_kernels.check_errors()


# ------------------------------------------------------------------ attention: window, kept first tokens, sink, gate

@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("nq,nkv,d,page,window,keep,rot", [
    (4, 2, 16, 8, 40, 5, 8), (4, 1, 64, 16, 100, 20, 32), (2, 2, 128, 16, 60, 130, 64), (4, 2, 64, 4, 33, 7, 32), (8, 8, 48, 16, 70, 16, 24),
    (4, 2, 64, 16, 150, 1, 64), (2, 1, 128, 32, 200, 150, 128), (32, 1, 32, 16, 24, 9, 32), (8, 2, 80, 16, 90, 65, 40), (2, 1, 256, 16, 50, 33, 64),
    (6, 3, 20, 16, 31, 17, 10), (4, 2, 64, 16, 17, 0, 32), (8, 4, 112, 16, 129, 48, 28), (2, 2, 64, 64, 140, 100, 32)])
def test_attention_with_kept_first_tokens_and_planted_keys(cuda_kernels, dtype, tol, nq, nkv, d, page, window, keep, rot):
    """A prompt of 400 tokens (the kernels of prompt portions, beyond their tiles of 128 and 256), a portion of 30 and then 40
    decoded ones; values are the keys before rotation, every head has a sink and a gate.  For queries in all parts one key
    is planted, a large product with that query alone: the sequence's first, the last kept one, the first that is not kept,
    the first of the query's window, the one before it, at a page's border, and the query's own.  The output must be the
    planted key when it is seen, and far from it when it is not; and it must agree with the plain statement."""
    from inferflux_b200.parts.base import KVCacheSpec
    cuts = [400, 30] + [1] * 40
    n_all = sum(cuts)
    g = torch.Generator().manual_seed(nq * 100 + d)
    q = 0.3 * torch.randn(n_all, nq, d, generator=g, dtype=F64)
    k = 0.3 * torch.randn(n_all, nkv, d, generator=g, dtype=F64)
    logits = 2.0 * torch.randn(n_all, nq, generator=g)
    sinks = torch.randn(nq, generator=g)
    sinks[0] = 15.0                                          # a head whose sink takes a visible share beside a planted key
    plain = PlainKernels(wide=True)
    unturn = lambda x, p: plain._turn(x[None], _rotary(60.0, rot, False, "cpu"), torch.tensor([-p]))[0]
    plants, used = {}, set()
    for base in (150, 262, 372, 404, 421, 433, 452):
        for j in range(7):
            p = base + 2 * j
            first = p - window + 1
            kp = [0, keep - 1, keep, first, first - 1, (p // page - 1) * page, p][j]
            if kp < 0 or kp in used or p in used or kp > p:
                continue
            used.add(kp)
            direction = torch.randn(d, generator=g, dtype=F64)
            direction *= 14.0 / direction.norm()
            q[p] = 0.05 * torch.randn(nq, d, generator=g, dtype=F64) + unturn(direction.expand(nq, d), p)
            k[kp] = 0.05 * torch.randn(nkv, d, generator=g, dtype=F64) + unturn(direction.expand(nkv, d), kp)
            plants[p] = (kp, kp >= first or kp < keep)
    assert len(plants) >= 12 and {s for _k, s in plants.values()} == {True, False} and any(p >= 430 for p in plants)
    scale = 16.0 / 14.0 ** 2 * (2.0 if d < 32 else 1.0)
    outs, gates = {}, None
    for name, kern, dev, dt in (("plain", plain, "cpu", F64), ("cuda", cuda_kernels, DEV, dtype)):
        cache = _cache(dt, KVCacheSpec(nkv, -(-d // 8) * 8, window, keep_first=keep), page, dev, tokens=n_all + page)
        got, pos = [], 0
        for n in cuts:
            ctx = _step_ctx(kern, dt, cache, [("r", n)], dev)
            sl = slice(pos, pos + n)
            rows = torch.cat([q[sl].reshape(n, -1), k[sl].reshape(n, -1), logits[sl].double(), torch.zeros(n, nq % 2, dtype=F64)], dim=1).to(dt).to(dev)
            qq, _back, gate = kern.row_norm_rope_append(rows, 0, None, _rotary(60.0, rot, False, dev), None, None, nq, nkv, d, d, ctx, _view(cache),
                                                        v_from_k=True, gate_col=(nq + nkv) * d)
            got.append(kern.attention(qq, nq, nkv, d, window, scale, ctx, _view(cache), dv=d, sink=sinks.to(dev), keep_first=keep,
                                      head_gate=gate).double().cpu())
            pos += n
        outs[name] = torch.cat(got).view(n_all, nq, d)
    cuda_kernels.check_errors()
    err = float((outs["cuda"] - outs["plain"]).abs().max())
    assert err <= tol * max(1.0, float(outs["plain"].abs().max())), err
    per = nq // nkv
    for p, (kp, seen) in plants.items():
        for h in range(1, nq):
            open_ = float(torch.sigmoid(logits[p, h]))
            away = float((outs["cuda"][p, h] / open_ - k[kp, h // per]).norm()) / 14.0
            assert (away < 0.25) == seen, (p, kp, seen, h, away)


def test_float32_attention_is_the_same_however_the_tokens_are_cut(cuda_kernels):
    from inferflux_b200.parts.base import KVCacheSpec
    nq, nkv, d, page, window, keep, n = 4, 2, 24, 8, 37, 11, 150
    g = torch.Generator().manual_seed(8)
    rows = torch.randn(n, (nq + nkv) * d + nq, generator=g).to(DEV)
    sinks = torch.randn(nq, generator=g).to(DEV)

    def run(cuts):
        cache, out, pos = _cache(torch.float32, KVCacheSpec(nkv, d, window, keep_first=keep), page, DEV), [], 0
        for m in cuts:
            ctx = _step_ctx(cuda_kernels, torch.float32, cache, [("r", m)], DEV)
            qq, _b, gate = cuda_kernels.row_norm_rope_append(rows[pos:pos + m].contiguous(), 0, None, _rotary(50.0, 12, False, DEV), None, None, nq, nkv,
                                                             d, d, ctx, _view(cache), v_from_k=True, gate_col=(nq + nkv) * d)
            out.append(cuda_kernels.attention(qq, nq, nkv, d, window, 0.4, ctx, _view(cache), dv=d, sink=sinks, keep_first=keep, head_gate=gate))
            pos += m
        return torch.cat(out)
    whole = run([n])
    for cuts in ([1] * n, [2, 35, 1, 64, 2, 46], [100] + [1] * 50):
        assert torch.equal(run(cuts), whole), cuts


# ------------------------------------------------------------------ whole models

LENS = [40, 33, 50, 61, 97, 70, 25, 64, 1, 2]


@pytest.fixture(scope="module")
def oracle(sanarax_dirs):
    memo = {}

    def get(name):
        if name not in memo:
            d, _page, raw = sanarax_dirs[name]
            reqs = sm.requests_for(raw, LENS, 100)
            memo[name] = {"reqs": reqs, "float32": sm.plain_logits(d, reqs),
                          "bfloat16": sm.plain_logits(d, reqs, weights_as=torch.bfloat16),
                          "yard": sm.plain_logits(d, reqs, weights_as=torch.bfloat16, dtype=torch.bfloat16)}
        return memo[name]
    return get


def _runner(d, dtype, page, kernels, pages=None, **kw):
    from inferflux_b200.engine import ModelRunner
    from inferflux_b200.models import load_model
    _c, model = load_model(d, dtype=dtype, device=DEV)
    return ModelRunner(model, kernels, page_size=page, num_pages=pages or 256 // page, max_seqs=4, max_seq_len=512, **kw)


def _bf16_close(name, got, want, yard):
    """bfloat16 logits against the exact ones, with the plain implementation in bfloat16 arithmetic on the same rounded
    weights as the yardstick.  The test models are sharp (a norm behind a sublayer magnifies a small output's rounding), so
    the largest of many rows is a matter of luck in both: up to three times the yardstick's, but not more in the middle."""
    err, bound = np.abs(got - want).max(axis=1), np.abs(yard - want).max(axis=1)
    assert float(err.max()) <= 3.0 * float(bound.max()), f"{name}: row {int(err.argmax())} is off by {float(err.max()):.4f}; rounding alone gives {float(bound.max()):.4f}"
    assert float(np.median(err)) <= 1.25 * float(np.median(bound)), f"{name}: median error {float(np.median(err)):.4f} against {float(np.median(bound)):.4f}"


def _check(name, dtype, got, o):
    if dtype == "float32":
        top = max(float(np.abs(v).max()) for v in o["float32"].values())
        bad = helpers.first_bad(got, o["float32"], 3e-4 + 1e-5 * top)
        assert bad is None, f"{name}: first wrong row (request, position, diff): {bad}"
    else:                                                  # all rows together: a request of one token has only one row
        rids = list(o["reqs"])
        _bf16_close(name, *(np.concatenate([x[r] for r in rids]) for x in (got, o["bfloat16"], o["yard"])))


@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cutting", ["whole", "tail", "portions", "mixed"])
def test_step_function_cuttings(name, dtype, cutting, sanarax_dirs, oracle, cuda_kernels):
    d, page, raw = sanarax_dirs[name]
    o = oracle(name)
    steps = {"whole": helpers.trace_whole, "tail": helpers.trace_tail, "portions": helpers.trace_portions,
             "mixed": lambda r: helpers.trace_mixed(r, 256)}[cutting](o["reqs"])
    runner = _runner(d, dtype, page, cuda_kernels, cuda_graphs=(cutting == "tail"))
    got = helpers.collect(steps, helpers.run_steps_in_process(runner, steps), raw["vocab"])
    cuda_kernels.check_errors()
    _check(f"{name} {cutting}", dtype, got, o)
    assert not runner.cache.live_requests() and runner.cache.free_pages() == [256 // page] * len(runner.cache.groups)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_float32_is_the_same_under_every_cutting(name, sanarax_dirs, oracle, cuda_kernels):
    d, page, raw = sanarax_dirs[name]
    reqs = oracle(name)["reqs"]
    results = []
    for make in (helpers.trace_whole, helpers.trace_tail, helpers.trace_portions, lambda r: helpers.trace_mixed(r, 256)):
        steps = make(reqs)
        runner = _runner(d, "float32", page, cuda_kernels)
        results.append(helpers.collect(steps, helpers.run_steps_in_process(runner, steps), raw["vocab"]))
    for other in results[1:]:
        for rid in reqs:
            assert np.array_equal(results[0][rid], other[rid]), rid


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_down_to_two_tokens_from_the_first_token_on(dtype, sanarax_dirs, cuda_kernels):
    from inferflux_b200.engine import StepEntry
    d, page, raw = sanarax_dirs["A"]
    toks = sm.requests_for(raw, [60], 3)["r0"]
    rounded = torch.bfloat16 if dtype == "bfloat16" else None
    want = sm.plain_logits(d, {"r0": toks}, weights_as=rounded)["r0"]
    yard = sm.plain_logits(d, {"r0": toks}, weights_as=torch.bfloat16, dtype=torch.bfloat16)["r0"]
    runner = _runner(d, dtype, page, cuda_kernels)
    got, pos, sizes, i = [], 0, [2, 1, 3, 2, 2, 5, 1, 1, 2, 17], 0
    while pos < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - pos)
        i += 1
        got += list(runner.step([StepEntry("r0", toks[pos:pos + n], list(range(n)))]).cpu().numpy())
        pos += n
    runner.end_request("r0")
    cuda_kernels.check_errors()
    if dtype == "float32":
        assert float(np.abs(np.stack(got) - want).max()) < 3e-4
    else:
        _bf16_close("short portions", np.stack(got), want, yard)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_medium_model_with_long_prompts(dtype, tmp_path, cuda_kernels):
    """Prompts of 700 and 300 tokens: whole, then in portions of 200 and 128 beside each other's decoded tokens.  These steps
    reach the kernels of many rows (library and tcgen05 products, the tiled attention kernels with kept first tokens and
    gates, the scan's long spans) inside a whole model."""
    from inferflux_b200.engine import ModelRunner, StepEntry
    from inferflux_b200.models import load_model
    raw, page = sm.medium_config()
    d = sm.write_model(raw, tmp_path / "medium", seed=77)
    reqs = sm.requests_for(raw, [700, 300], 12)
    rows = {"r0": [0, 1, 36, 37, 127, 128, 150, 199, 200, 201, 255, 256, 257, 383, 384, 511, 512, 640, 698, 699],
            "r1": [0, 63, 64, 127, 128, 170, 200, 298, 299]}
    rounded = torch.bfloat16 if dtype == "bfloat16" else None
    want = {k: v[rows[k]] for k, v in sm.plain_logits(d, reqs, weights_as=rounded).items()}
    yard = {k: v[rows[k]] for k, v in sm.plain_logits(d, reqs, weights_as=torch.bfloat16, dtype=torch.bfloat16).items()} \
        if dtype == "bfloat16" else None

    def compare(name, got):
        for rid in reqs:
            if dtype == "float32":
                # sharp attention: an angle of 700 rounded to float32 alone moves the logits by up to 1e-2
                err = np.abs(got[rid] - want[rid])
                assert float(err.max()) < 1.5e-2 and float(err.mean()) < 5e-4, (name, rid, float(err.max()), float(err.mean()))
            else:
                _bf16_close(f"{name} {rid}", got[rid], want[rid], yard[rid])
    _c, model = load_model(d, dtype=dtype, device=DEV)
    runner = ModelRunner(model, cuda_kernels, page_size=page, num_pages=80, max_seqs=4, max_seq_len=1024)
    got = {}
    for rid, toks in reqs.items():
        got[rid] = runner.step([StepEntry(rid, toks, rows[rid])]).cpu().numpy()
        runner.end_request(rid)
    cuda_kernels.check_errors()
    compare("whole", got)
    got = {rid: {} for rid in reqs}
    at = {"r0": 0, "r1": 0}
    size = {"r0": 200, "r1": 128}
    while any(at[r] < len(reqs[r]) for r in reqs):
        entries, asked = [], []
        for rid, toks in reqs.items():
            if at[rid] >= len(toks):
                continue
            n = 1 if len(toks) - at[rid] <= 20 else min(size[rid], len(toks) - 20 - at[rid])
            w = [p - at[rid] for p in rows[rid] if at[rid] <= p < at[rid] + n]
            entries.append(StepEntry(rid, toks[at[rid]:at[rid] + n], w))
            asked += [(rid, p) for p in rows[rid] if at[rid] <= p < at[rid] + n]
            at[rid] += n
        out = runner.step(entries).cpu().numpy()
        for (rid, p), row in zip(asked, out):
            got[rid][p] = row
        for rid in reqs:
            if at[rid] == len(reqs[rid]) and rid in runner.cache:
                runner.end_request(rid)
        runner.cache.check()
    cuda_kernels.check_errors()
    compare("portions", {rid: np.stack([got[rid][p] for p in rows[rid]]) for rid in reqs})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_reused_pages_slots_and_graphs(dtype, sanarax_dirs, cuda_kernels):
    """12 prompt tokens, then 300 decoded one by one beside requests that join and leave: page borders and windows are
    crossed by decoded tokens, the pages and the slot of a request that left serve the next one, decode steps replay a
    CUDA graph."""
    from inferflux_b200.engine import StepEntry
    d, page, raw = sanarax_dirs["A"]
    reqs = sm.requests_for(raw, [312, 90, 60], 9)
    want = sm.plain_logits(d, reqs, weights_as=torch.bfloat16 if dtype == "bfloat16" else None)
    yard = sm.plain_logits(d, reqs, weights_as=torch.bfloat16, dtype=torch.bfloat16) if dtype == "bfloat16" else None
    runner = _runner(d, dtype, page, cuda_kernels, pages=52, cuda_graphs=True)     # 40 pages for r0, 12 for one of the others
    a = reqs["r0"]
    got = {rid: [] for rid in reqs}
    got["r0"] += list(runner.step([StepEntry("r0", a[:12], list(range(12)))]).cpu().numpy())
    at = {"r1": 0, "r2": 0}
    for i in range(12, len(a)):
        entries, order = [StepEntry("r0", [a[i]], [0])], ["r0"]
        other = "r1" if at["r1"] < len(reqs["r1"]) else ("r2" if at["r2"] < len(reqs["r2"]) else None)
        if i >= 100 and other is not None:
            n = 7 if at[other] < 49 else 1
            n = min(n, len(reqs[other]) - at[other])
            entries.append(StepEntry(other, reqs[other][at[other]:at[other] + n], list(range(n))))
            order += [other] * n
            at[other] += n
        out = runner.step(entries).cpu().numpy()
        for rid, row in zip(order, out):
            got[rid].append(row)
        if other is not None and at[other] == len(reqs[other]) and other in runner.cache:
            runner.end_request(other)
        runner.cache.check()
    cuda_kernels.check_errors()
    assert runner.graph_replays > 50
    got = {k: np.stack(v) for k, v in got.items()}
    if dtype == "float32":
        for rid in reqs:
            assert float(np.abs(got[rid] - want[rid]).max()) < 5e-4, rid
    else:
        _bf16_close("long decoding", *(np.concatenate([x[r] for r in reqs]) for x in (got, want, yard)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(dtype, sanarax_dirs, oracle, tmp_path):
    d, page, raw = sanarax_dirs["B"]
    o = oracle("B")
    steps = helpers.trace_mixed(o["reqs"], 256)
    got = helpers.collect(steps, helpers.run_trace_cli(d, dtype, steps, tmp_path / "out", 256, raw["vocab"], page_size=page),
                          raw["vocab"])
    _check("B through the program", dtype, got, o)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_engine_and_scheduler(dtype, sanarax_dirs):
    from inferflux_b200 import Engine, SamplingParams
    d, page, raw = sanarax_dirs["A"]
    _raw, W = sm.load(d)
    if dtype == "bfloat16":
        W = {k: (v.to(torch.bfloat16) if v.is_floating_point() else v) for k, v in W.items()}
    prompts = list(sm.requests_for(raw, [7, 19, 33, 4, 1, 70], 40).values())
    for pages in (64, 14):                                 # 14 pages of 8: the requests do not all fit at once
        eng = Engine(d, dtype=dtype, device=DEV, kv_page_size=page, kv_num_pages=pages, kv_max_batch=4, kv_max_seq=128,
                     chunked_prefill_tokens=16, max_batch_tokens=48)
        res = eng.generate(prompts, SamplingParams(temperature=0.0), max_tokens=24)
        for prompt, r in zip(prompts, res):
            seq = list(prompt) + list(r.token_ids)
            exact = P.forward(raw, W, seq)
            rough = P.forward(raw, W, seq, dtype=torch.bfloat16).double() if dtype == "bfloat16" else None
            for i, tok in enumerate(r.token_ids):
                row = len(prompt) - 1 + i
                gap = float(exact[row].max() - exact[row, tok])
                slack = 1e-3 if rough is None else 4.0 * float((rough - exact).abs().max())
                assert gap <= slack, f"token {i}: {gap:.4f} below the best logit, rounding allows {slack:.4f}"
        assert not eng.runner.cache.live_requests()
