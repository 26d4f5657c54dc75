"""Vononex on the GPU: every new kernel alone against the plain kernel statements (themselves held to the plain
implementation by the CPU tests), attention with turned values and planted keys, then whole models through the step
function, the replay program and the engine."""
import math

import numpy as np
import pytest
import torch

import helpers
import vononex_models as vm
from plain import plain_vononex as P
from plain.plain_kernels import PlainKernels

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def vononex_dirs(tmp_path_factory):
    out = {}
    for i, (name, (raw, page)) in enumerate(vm.configs().items()):
        out[name] = (vm.write_model(raw, tmp_path_factory.mktemp(f"vononex_{name}"), seed=51 + i), page, raw)
    return out


class _Ctx:
    """The few fields of a step context that the kernels of this file read, on a device."""

    def __init__(self, spans, slots, device):
        cu, pos, req = [0], [], []
        for r, (start, n) in enumerate(spans):
            cu.append(cu[-1] + n)
            pos += list(range(start, start + n))
            req += [r] * n
        mk = lambda v: torch.tensor(v, dtype=torch.int32, device=device)
        self.cu_seqlens, self.positions, self.token_req, self.req_slot = mk(cu), mk(pos), mk(req), mk(slots)
        self.num_requests, self.num_tokens = len(spans), cu[-1]
        self.spans, self.slots_host = list(spans), list(slots)
        self.max_span = max(n for _s, n in spans)
        self.max_kv_len = max(s + n for s, n in spans)
        self.extra, self.extra_len = {}, {}


def _steps(lens_per_step, slot_of):
    """[(spans, slots)] for requests that bring lens_per_step[step][request] tokens (0: the request sits the step out)."""
    starts = [0] * len(slot_of)
    for lens in lens_per_step:
        spans, slots = [], []
        for q, n in enumerate(lens):
            if n:
                spans.append((starts[q], n))
                slots.append(slot_of[q])
                starts[q] += n
        yield spans, slots


# ------------------------------------------------------------------ the norm of a sum

def _partial(t, splits, g):
    """`t` (float32) as a PartialSum: slices that add up to it."""
    from inferflux_b200.csrc.ops import PartialSum
    parts = [torch.randn(t.shape, generator=g) for _ in range(splits - 1)]
    return PartialSum(torch.stack([t - sum(parts)] + parts if parts else [t]).to(DEV).contiguous(), torch.bfloat16)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("H", [48, 50, 64, 321, 1024, 4096, 5000])
def test_norm_of_sum_with_slices_biases_and_weights(cuda_kernels, dtype, tol, H):
    plain = PlainKernels(wide=True)
    g = torch.Generator().manual_seed(H)
    rnd = lambda *s: torch.randn(*s, generator=g)
    for T, splits in ((1, 3), (7, 10), (40, 1)):
        x, y1, y2, b1, w = 2.0 * rnd(T, H), rnd(T, H), 3.0 * rnd(T, H), rnd(H), 1 + 0.3 * rnd(H)
        yb = rnd(T, H).to(torch.bfloat16)
        for alpha, terms in ((2.5, [(0.7, y1, b1), (-1.3, y2, None)]), (1.0, [(1.0, yb, b1)]), (0.4, [(1.1, yb, None), (0.3, y2, b1)])):
            for weight in (w, None):
                xp, xg = x.double().clone(), x.clone().to(DEV)
                want = plain.norm_of_sum(xp, alpha, [(c, y.double(), b) for c, y, b in terms], weight, 1e-4, out_dtype=F64)
                on_gpu = [(c, _partial(y, splits, g) if y.dtype == torch.float32 else y.to(DEV), None if b is None else b.to(DEV)) for c, y, b in terms]
                got = cuda_kernels.norm_of_sum(xg, alpha, on_gpu, None if weight is None else weight.to(DEV), 1e-4, out_dtype=dtype)
                top = float(want.abs().max())
                assert got.dtype == dtype and float((got.double().cpu() - want).abs().max()) <= tol * top
                assert float((xg.double().cpu() - want).abs().max()) <= 3e-6 * top
                assert cuda_kernels.norm_of_sum(xg, alpha, on_gpu, None, 0.0) is None


# ------------------------------------------------------------------ rows: norm, rotation, cache; rotation alone

def _cache(dtype, nkv, row, page, window, device, tokens=400):
    pages = -(-tokens // page)
    from inferflux_b200.cache.manager import CacheManager
    from inferflux_b200.parts.base import KVCacheSpec
    return CacheManager([(KVCacheSpec(nkv, row, window), None)], page_size=page, num_pages=pages, max_seqs=4, max_seq_len=page * pages,
                        dtype=dtype, device=device)


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


def _freqs(base, dims):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64).float()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 5e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("nq,nkv,d,dv,rot,inter,page", [(4, 2, 16, 8, 16, False, 8), (6, 1, 8, 32, 4, False, 4), (3, 3, 10, 6, 10, False, 16),
                                                         (12, 4, 64, 64, 32, False, 16), (16, 2, 128, 128, 128, False, 16), (5, 1, 14, 14, 2, True, 4),
                                                         (8, 8, 32, 48, 0, True, 8)])
def test_row_norm_rotation_factors_and_turned_values(cuda_kernels, dtype, tol, nq, nkv, d, dv, rot, inter, page):
    """Queries, both halves of the cache and the angles' table against the plain statement: few tokens (a cluster of blocks
    per token) and many, plain rows in both dtypes and K slices, rows that start inside wider ones, with and without
    norms, biases, factors and turned values; every key head large beside another, so that a norm per head would show."""
    from inferflux_b200.config.plan import ScheduleEntry
    from inferflux_b200.parts.base import RotaryTable
    g = torch.Generator().manual_seed(nq * 100 + d)
    rnd = lambda *s: torch.randn(*s, generator=g)
    width = (nq + nkv) * d + nkv * dv
    spread = torch.cat([torch.exp(rnd(nq, 1)).expand(nq, d).reshape(-1), torch.exp(rnd(nkv, 1)).expand(nkv, d).reshape(-1), torch.ones(nkv * dv)])
    bias, temp, wq, wk = 0.5 * rnd(width), 0.5 + torch.rand(nq, generator=g), 1 + 0.3 * rnd(nq * d), 1 + 0.3 * rnd(nkv * d)
    row = -(-max(d, dv) // 8) * 8
    caches = {"plain": _cache(F64, nkv, row, page, None, "cpu"), "cuda": _cache(dtype, nkv, row, page, None, DEV)}
    for step, (spans, kind) in enumerate((([("a", 37), ("b", 5)], "same"), ([("a", 1), ("b", 1)], "slices"), ([("b", 70)], "float"),
                                          ([("a", 1), ("b", 2), ("c", 1)], "slices"))):
        full = step != 2
        T = sum(n for _r, n in spans)
        col0, extra = (6, 10) if kind == "slices" else (0, 0)
        wide = rnd(T, width + extra)
        wide[:, col0:col0 + width] *= spread
        if kind == "same":
            wide = wide.to(dtype)
        res = {}
        for name, kern, dev, dt in (("plain", PlainKernels(wide=True), "cpu", F64), ("cuda", cuda_kernels, DEV, dtype)):
            to = lambda t: None if t is None or not full else t.to(dev)
            ctx = _step_ctx(kern, dt, caches[name], spans, dev)
            view = caches[name].view(ScheduleEntry(layer=0, cache=0))
            rows = wide.double() if name == "plain" else (_partial(wide.float(), 5, g) if kind == "slices" else wide.to(DEV))
            rt = RotaryTable(_freqs(90.0, rot).to(dev), rot, inter) if rot else None
            turn = RotaryTable(_freqs(40.0, dv).to(dev), dv, inter) if full else None
            q, back = kern.row_norm_rope_append(rows, col0, to(bias), rt, turn, to(temp), nq, nkv, d, dv, ctx, view, q_norm=to(wq),
                                                k_norm=to(wk), norm_eps=1e-5)
            assert (back is None) != full and q.dtype == dt
            held = [view.kv[list(caches[name].pages_of(r).values())].double().cpu() for r, _n in spans]
            res[name] = [q.double().cpu()] + held + ([] if back is None else [back[0].double().cpu()])
        for a, b in zip(res["cuda"], res["plain"]):
            assert a.shape == b.shape and float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max())), (step, kind)


@pytest.mark.parametrize("heads,dk,rest,rot,inter", [(3, 12, 30, 12, False), (2, 64, 96, 32, False), (1, 6, 7, 2, True), (5, 24, 60, 0, False),
                                                     (2, 256, 512, 256, False), (4, 10, 300, 8, True)])
def test_rotated_rows_in_place_from_slices_and_from_wider_rows(cuda_kernels, heads, dk, rest, rot, inter):
    from inferflux_b200.parts.base import RotaryTable
    g = torch.Generator().manual_seed(heads * 100 + dk)
    width = 2 * heads * dk + rest
    plain = PlainKernels(wide=True)
    for spans in ([(0, 33), (900, 1)], [(7, 1), (150, 1), (3, 2)]):
        T = sum(n for _s, n in spans)
        slots = list(range(len(spans)))
        wide = torch.randn(T, width + 9, generator=g)
        rt = lambda dev: RotaryTable(_freqs(700.0, rot).to(dev), rot, inter) if rot else None
        for col0 in (0, 9):
            want = plain.rotate_rows(wide.double(), col0, width, heads, dk, rt("cpu"), 0.3, _Ctx(spans, slots, "cpu"))
            own = wide[:, col0:col0 + width].contiguous().to(DEV)
            for rows, at in ((own, 0), (wide.to(DEV), col0), (_partial(wide, 4, g), col0)):
                got = cuda_kernels.rotate_rows(rows, at, width, heads, dk, rt(DEV), 0.3, _Ctx(spans, slots, DEV))
                assert got.dtype == torch.float32 and (got.data_ptr() == own.data_ptr()) == (rows is own)
                assert float((got.double().cpu() - want).abs().max()) <= 1e-5 * max(1.0, float(want.abs().max()))


# ------------------------------------------------------------------ the two recurrences

@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("W", [1, 24, 32, 104, 456, 2048])
def test_gated_scan_over_steps_and_requests(cuda_kernels, dtype, tol, W):
    """Three requests over five steps: spans shorter and longer than a tile of the walk, a request that sits a step out,
    states in slots that lie inside longer rows, plain rows and K slices; gates from shut to open."""
    plain = PlainKernels(wide=True)
    g = torch.Generator().manual_seed(W)
    bias = torch.randn(2 * W, generator=g)
    sg, sp = torch.zeros(4, W + 5, device=DEV), torch.zeros(4, W + 5, dtype=F64)
    for step, (spans, slots) in enumerate(_steps([(200, 1, 63), (1, 16, 0), (2, 64, 1), (1, 1, 129), (1, 1, 1)], [3, 0, 2])):
        T = sum(n for _s, n in spans)
        rows = 4.0 * torch.randn(T, 3 * W, generator=g)
        want = plain.gated_scan(rows.double(), bias, sp[:, 5:], W, _Ctx(spans, slots, "cpu"), F64)
        src = rows.to(DEV) if step % 2 == 0 else _partial(rows, 6, g)
        got = cuda_kernels.gated_scan(src, bias.to(DEV), sg[:, 5:], W, _Ctx(spans, slots, DEV), dtype)
        assert got.dtype == dtype and float((got.double().cpu() - want).abs().max()) <= tol * max(1.0, float(want.abs().max())), step
        assert float((sg.double().cpu() - sp).abs().max()) <= 5e-6 * max(1.0, float(sp.abs().max())), step
    assert float(sg[1].abs().max()) == 0.0 and float(sg[:, :5].abs().max()) == 0.0


def test_gated_scan_is_the_same_however_it_is_cut_and_keeps_what_is_far_back(cuda_kernels):
    W, T = 40, 331
    g = torch.Generator().manual_seed(5)
    rows = torch.randn(T, 3 * W, generator=g)
    rows[:, :W] -= 18.0                                                      # gates all but shut: z about 1e-8 ...
    rows[3, :W] = 9.0                                                        # ... but for token 3, whose candidate stays
    rows[3, W:2 * W] = 5.0 + torch.arange(W)
    bias = torch.zeros(2 * W)

    def run(cuts, others=0):
        state, out, pos = torch.zeros(3, W, device=DEV), [], 0
        for n in cuts:
            part, spans, slots = rows[pos:pos + n], [(pos, n)], [1]
            if others:
                part, spans, slots = torch.cat([rows[:others] * 0.5, part]), [(0, others)] + spans, [2, 1]
            out.append(cuda_kernels.gated_scan(part.contiguous().to(DEV), bias.to(DEV), state, W, _Ctx(spans, slots, DEV), torch.float32)[others:])
            pos += n
        return torch.cat(out), state[1].clone()
    whole, s0 = run([T])
    for cuts, others in (([1] * T, 0), ([64, 64, 64, 64, 64, 11], 0), ([2, 63, 1, 65, 2, 198], 0), ([100, 231], 70)):
        got, s1 = run(cuts, others)
        assert torch.equal(got, whole) and torch.equal(s0, s1), cuts
    assert float((s0.cpu() - (5.5 + torch.arange(W))).abs().max()) < 2e-2    # what token 3 wrote, 328 tokens later


@pytest.mark.parametrize("H,dk,dv", [(3, 12, 20), (1, 6, 3), (2, 64, 40), (5, 10, 7), (4, 128, 64), (2, 256, 96), (1, 200, 1), (8, 24, 40)])
def test_constant_decay_scan_over_steps_and_requests(cuda_kernels, H, dk, dv):
    plain = PlainKernels(wide=True)
    front = 8
    sg, sp = torch.zeros(4, front + H * dk * dv, device=DEV), torch.zeros(4, front + H * dk * dv, dtype=F64)
    g = torch.Generator().manual_seed(H * 1000 + dk)
    rate = torch.cat([torch.rand(H, generator=g)[1:] * 0.5 + 0.5, torch.ones(1)])
    for step, (spans, slots) in enumerate(_steps([(37, 1, 5), (1, 16, 0), (2, 17, 1), (1, 1, 1), (100, 1, 70)], [3, 0, 2])):
        T = sum(n for _s, n in spans)
        wide = torch.randn(T, 2 * H * (dk + dv), generator=g)                # q | k | v | gate side by side
        cut = lambda t: (t[:, :H * dk], t[:, H * dk:2 * H * dk], t[:, 2 * H * dk:2 * H * dk + H * dv])
        kw = dict(heads=H, groups=H, dk=dk, dv=dv, decay="constant")
        want = plain.decay_scan(*cut(wide.double()), None, sp[:, front:], _Ctx(spans, slots, "cpu"), rate=rate, **kw)
        got = cuda_kernels.decay_scan(*cut(wide.to(DEV)), None, sg[:, front:], _Ctx(spans, slots, DEV), rate=rate.to(DEV), **kw)
        assert float((got.double().cpu() - want.double()).abs().max()) <= 3e-5 * max(1.0, float(want.abs().max())), step
        assert float((sg.double().cpu() - sp).abs().max()) <= 3e-5 * max(1.0, float(sp.abs().max())), step
    assert float(sg[1].abs().max()) == 0.0 and float(sg[:, :front].abs().max()) == 0.0


def test_constant_decay_scan_is_the_same_however_it_is_cut_and_reads_far_back(cuda_kernels):
    """What token 3 wrote is read back by token 600 (q along k_3) in a head that does not decay, and is gone in one that does."""
    H, dk, dv, T = 2, 32, 24, 601
    g = torch.Generator().manual_seed(4)
    q, k, v = torch.randn(T, H * dk, generator=g), 0.02 * torch.randn(T, H * dk, generator=g), torch.randn(T, H * dv, generator=g)
    k[3] = 3.0 * torch.randn(H * dk, generator=g)
    k3 = k[3].view(H, dk)
    q[600] = (k3 / (k3 * k3).sum(-1, keepdim=True)).reshape(-1) * 50.0
    rate = torch.tensor([1.0, 0.9]).to(DEV)

    def run(cuts):
        state, out, pos = torch.zeros(2, H * dk * dv, device=DEV), [], 0
        for n in cuts:
            sl = slice(pos, pos + n)
            out.append(cuda_kernels.decay_scan(q[sl].to(DEV), k[sl].to(DEV), v[sl].to(DEV), None, state, _Ctx([(pos, n)], [1], DEV), heads=H,
                                               groups=H, dk=dk, dv=dv, decay="constant", rate=rate))
            pos += n
        return torch.cat(out), state.clone()
    whole, s0 = run([T])
    for cuts in ([590] + [1] * 11, [16, 17, 63, 64, 65, 2, 374]):
        got, s1 = run(cuts)
        assert torch.equal(got, whole) and torch.equal(s0, s1), cuts
    cos = torch.nn.functional.cosine_similarity(whole[600].view(H, dv).cpu(), v[3].view(H, dv), dim=-1)
    assert float(cos[0]) > 0.97 and abs(float(cos[1])) < 0.9


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("C,groups", [(64, 4), (30, 5), (320, 1), (2048, 2), (96, 12)])
def test_gated_norm_without_a_weight(cuda_kernels, dtype, tol, C, groups):
    g = torch.Generator().manual_seed(C)
    y, wide = 2.0 * torch.randn(9, C, generator=g), 2.0 * torch.randn(9, C + 11, generator=g)
    for first in (True, False):
        want = PlainKernels(wide=True).gated_groupnorm(y.double(), wide[:, 3:3 + C].double(), None, 1e-5, groups, first, F64)
        got = cuda_kernels.gated_groupnorm(y.to(DEV), wide.to(DEV)[:, 3:3 + C], None, 1e-5, groups, first, dtype)
        assert got.dtype == dtype and float((got.double().cpu() - want).abs().max()) <= tol * float(want.abs().max())


# ------------------------------------------------------------------ the gelu-gated product

@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 1.5e-2)])
@pytest.mark.parametrize("T,K,F", [(1, 72, 88), (5, 96, 200), (16, 64, 2500), (33, 320, 192), (150, 128, 10000), (160, 64, 40), (161, 320, 448),
                                   (300, 256, 128), (700, 72, 333), (200, 4200, 64), (3, 50, 33), (190, 50, 75)])
def test_gelu_gated_product_with_biases(cuda_kernels, dtype, tol, T, K, F):
    """Every way it is made: the weight-streaming kernel with one tile and with two half tiles, the many-rows kernel (whole
    tiles and edges), the library product with the activation kernel (long inner sizes, odd sizes), float32."""
    g = torch.Generator().manual_seed(T + K)
    a, w = torch.randn(T, K, generator=g).to(dtype), (1.5 / math.sqrt(K) * torch.randn(2 * F, K, generator=g)).to(dtype)
    for bias in (torch.randn(2 * F, generator=g), None):
        want = PlainKernels(wide=True).linear_geglu(a.double(), w.double(), bias)
        got = cuda_kernels.linear_geglu(a.to(DEV), w.to(DEV), None if bias is None else bias.to(DEV))
        assert got.dtype == dtype and float((got.double().cpu() - want).abs().max()) <= tol * max(1.0, float(want.abs().max()))
    cuda_kernels.check_errors()


def test_gelu_gate_far_out(cuda_kernels):
    """Large gates of either sign: the activation is the identity or zero there, never NaN."""
    for dtype in (torch.float32, torch.bfloat16):
        for T in (3, 300):
            a = torch.zeros(T, 64, dtype=dtype)
            a[:, 0] = torch.linspace(-60.0, 60.0, T).to(dtype)
            w = torch.zeros(2 * 64, 64, dtype=dtype)
            w[:64, 0] = torch.linspace(-8.0, 8.0, 64).to(dtype)
            want = PlainKernels(wide=True).linear_geglu(a.double(), w.double(), torch.cat([torch.zeros(64), torch.ones(64)]))
            got = cuda_kernels.linear_geglu(a.to(DEV), w.to(DEV), torch.cat([torch.zeros(64), torch.ones(64)]).to(DEV)).double().cpu()
            assert bool(torch.isfinite(got).all()) and float((got - want).abs().max()) <= (1e-2 if dtype == torch.bfloat16 else 1e-5) * 480


# ------------------------------------------------------------------ attention with turned values and planted keys

@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("nq,nkv,d,dv,page,window,rot,inter", [
    (4, 2, 16, 16, 8, None, 16, False), (4, 1, 64, 64, 16, None, 64, False), (2, 2, 128, 128, 16, None, 64, False), (4, 2, 64, 64, 4, None, 32, False),
    (8, 8, 48, 48, 16, 40, 24, False), (2, 1, 64, 32, 16, None, 16, False), (2, 2, 24, 48, 8, None, 24, False), (3, 3, 20, 12, 16, 33, 6, True),
    (4, 2, 64, 64, 16, 100, 64, True), (2, 1, 128, 128, 32, None, 128, True), (32, 1, 32, 32, 16, None, 32, False), (8, 2, 80, 80, 16, None, 80, True),
    (2, 1, 256, 256, 16, None, 64, False)])
def test_attention_turned_values_and_planted_keys(cuda_kernels, dtype, tol, nq, nkv, d, dv, page, window, rot, inter):
    """A prompt of 400 tokens (the kernels of prompt portions, beyond their tiles of 128 and 256) and then 40 decoded ones,
    values turned by their own position and the output turned back.  For queries in both parts one key is planted, a large
    product with that query alone: as far back as the query sees, at the first key of its window, just outside it, at a
    page's border, and the query's own.  The output must be the planted key's value turned by minus the distance when
    the key is seen, and must not be when it is not; and it must agree with the plain statement."""
    from inferflux_b200.config.plan import ScheduleEntry
    from inferflux_b200.parts.base import RotaryTable
    n_prompt, n_all = 400, 440
    g = torch.Generator().manual_seed(nq * 100 + d)
    q = 0.3 * torch.randn(n_all, nq, d, generator=g, dtype=F64)
    k = 0.3 * torch.randn(n_all, nkv, d, generator=g, dtype=F64)
    v = torch.randn(n_all, nkv, dv, generator=g, dtype=F64)
    w = window or 10 ** 6
    plain = PlainKernels(wide=True)
    rt = lambda dev: RotaryTable(_freqs(60.0, rot).to(dev), rot, inter)
    turn = lambda dev: RotaryTable(_freqs(35.0, dv).to(dev), dv, inter)
    unturn = lambda x, p: plain._turn(x[None], rt("cpu"), torch.tensor([-p]))[0]         # so that it arrives unturned
    plants, used = {}, set()
    for base in (130, 258, 384, 410, 427):
        for j in range(4):
            p = base + 3 * j
            first = max(0, p - w + 1)
            kp, seen = [(first + 1 + len(used) if not window else first, True), (p - w, False), (max(first, (p // page - 1) * page), True), (p, True)][j]
            if kp < 0 or kp in used or p in used:
                continue
            used.add(kp)
            direction = torch.randn(d, generator=g, dtype=F64)
            direction *= 14.0 / direction.norm()
            q[p] = 0.05 * torch.randn(nq, d, generator=g, dtype=F64) + unturn(direction.expand(nq, d), p)
            k[kp] = 0.05 * torch.randn(nkv, d, generator=g, dtype=F64) + unturn(direction.expand(nkv, d), kp)
            plants[p] = (kp, seen)
    assert len(plants) >= 12
    scale = 16.0 / 14.0 ** 2 * (2.0 if d < 32 else 1.0)
    outs = {}
    for name, kern, dev, dt in (("plain", plain, "cpu", F64), ("cuda", cuda_kernels, DEV, dtype)):
        cache = _cache(dt, nkv, -(-max(d, dv) // 8) * 8, page, window, dev, tokens=n_all + page)
        got, pos = [], 0
        for n in [n_prompt] + [1] * (n_all - n_prompt):
            ctx = _step_ctx(kern, dt, cache, [("r", n)], dev)
            view = cache.view(ScheduleEntry(layer=0, cache=0))
            sl = slice(pos, pos + n)
            rows = torch.cat([q[sl].reshape(n, -1), k[sl].reshape(n, -1), v[sl].reshape(n, -1)], dim=1).to(dt).to(dev)
            qq, back = kern.row_norm_rope_append(rows, 0, None, rt(dev), turn(dev), None, nq, nkv, d, dv, ctx, view)
            got.append(kern.attention(qq, nq, nkv, d, window, scale, ctx, view, dv=dv, turn_back=back).double().cpu())
            pos += n
        outs[name] = torch.cat(got).view(n_all, nq, dv)
    cuda_kernels.check_errors()
    err = float((outs["cuda"] - outs["plain"]).abs().max())
    assert err <= tol * max(1.0, float(outs["plain"].abs().max())), err
    per = nq // nkv
    for p, (kp, seen) in plants.items():
        away = plain._turn(v[kp][None], turn("cpu"), torch.tensor([kp - p]))[0]
        for h in range(nq):
            close = float((outs["cuda"][p, h] - away[h // per]).abs().max())
            assert (close < 0.15) == seen, (p, kp, seen, h, close)


# ------------------------------------------------------------------ whole models

LENS = [40, 33, 50, 61, 97, 70, 25, 64, 1, 2]


@pytest.fixture(scope="module")
def oracle(vononex_dirs):
    memo = {}

    def get(name):
        if name not in memo:
            d, _page, raw = vononex_dirs[name]
            reqs = vm.requests_for(raw, LENS, 100)
            memo[name] = {"reqs": reqs, "float32": vm.plain_logits(d, reqs),
                          "bfloat16": vm.plain_logits(d, reqs, weights_as=torch.bfloat16),
                          "yard": vm.plain_logits(d, reqs, weights_as=torch.bfloat16, dtype=torch.bfloat16)}
        return memo[name]
    return get


def _runner(d, dtype, page, kernels, pages=None, **kw):
    from inferflux_b200.engine import ModelRunner
    from inferflux_b200.models import load_model
    _c, model = load_model(d, dtype=dtype, device=DEV)
    return ModelRunner(model, kernels, page_size=page, num_pages=pages or 256 // page, max_seqs=4, max_seq_len=512, **kw)


def _bf16_close(name, got, want, yard):
    """bfloat16 logits against the exact ones, with the plain implementation in bfloat16 arithmetic on the same rounded
    weights as the yardstick.  The test models are sharp, so two correct bfloat16 computations differ by about as much as
    either differs from the exact result: up to twice the yardstick's worst row, and no worse on average."""
    err, bound = np.abs(got - want).max(axis=1), np.abs(yard - want).max(axis=1)
    assert float(err.max()) <= 2.0 * float(bound.max()), f"{name}: row {int(err.argmax())} is off by {float(err.max()):.4f}; rounding alone gives {float(bound.max()):.4f}"
    assert float(err.mean()) <= 1.2 * float(bound.mean()), f"{name}: mean error {float(err.mean()):.4f} against {float(bound.mean()):.4f}"


def _check(name, dtype, got, o):
    if dtype == "float32":
        top = max(float(np.abs(v).max()) for v in o["float32"].values())
        bad = helpers.first_bad(got, o["float32"], 2e-4 + 1e-5 * top)
        assert bad is None, f"{name}: first wrong row (request, position, diff): {bad}"
    else:
        for rid in o["reqs"]:
            _bf16_close(f"{name} {rid}", got[rid], o["bfloat16"][rid], o["yard"][rid])


@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cutting", ["whole", "tail", "portions", "mixed"])
def test_step_function_cuttings(name, dtype, cutting, vononex_dirs, oracle, cuda_kernels):
    d, page, raw = vononex_dirs[name]
    o = oracle(name)
    steps = {"whole": helpers.trace_whole, "tail": helpers.trace_tail, "portions": helpers.trace_portions,
             "mixed": lambda r: helpers.trace_mixed(r, 256)}[cutting](o["reqs"])
    runner = _runner(d, dtype, page, cuda_kernels, cuda_graphs=(cutting == "tail"))
    got = helpers.collect(steps, helpers.run_steps_in_process(runner, steps), raw["vocab"])
    cuda_kernels.check_errors()
    _check(f"{name} {cutting}", dtype, got, o)
    assert not runner.cache.live_requests()


@pytest.mark.parametrize("name", ["A", "C"])
def test_float32_is_the_same_under_every_cutting(name, vononex_dirs, oracle, cuda_kernels):
    d, page, raw = vononex_dirs[name]
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
def test_portions_down_to_two_tokens_from_the_first_token_on(dtype, vononex_dirs, cuda_kernels):
    from inferflux_b200.engine import StepEntry
    d, page, raw = vononex_dirs["A"]
    toks = vm.requests_for(raw, [60], 3)["r0"]
    rounded = torch.bfloat16 if dtype == "bfloat16" else None
    want = vm.plain_logits(d, {"r0": toks}, weights_as=rounded)["r0"]
    yard = vm.plain_logits(d, {"r0": toks}, weights_as=torch.bfloat16, dtype=torch.bfloat16)["r0"]
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
    """Prompts of 700 and 300 tokens through a model of four layers: whole, then in portions of 200 and 128 beside each
    other's decoded tokens.  These steps reach the kernels of many rows (library and tcgen05 products, the tiled attention
    kernels with turned values, both scans' long spans) inside a whole model."""
    from inferflux_b200.engine import ModelRunner, StepEntry
    from inferflux_b200.models import load_model
    raw, page = vm.medium_config()
    d = vm.write_model(raw, tmp_path / "medium", seed=77)
    reqs = vm.requests_for(raw, [700, 300], 12)
    rows = {"r0": [0, 1, 127, 128, 129, 255, 256, 257, 383, 384, 511, 512, 640, 698, 699], "r1": [0, 63, 64, 127, 128, 200, 298, 299]}
    rounded = torch.bfloat16 if dtype == "bfloat16" else None
    want = {k: v[rows[k]] for k, v in vm.plain_logits(d, reqs, weights_as=rounded).items()}
    yard = {k: v[rows[k]] for k, v in vm.plain_logits(d, reqs, weights_as=torch.bfloat16, dtype=torch.bfloat16).items()} \
        if dtype == "bfloat16" else None

    def compare(name, got):
        for rid in reqs:
            if dtype == "float32":
                # logits up to 20, sharp attention: an angle of 700 rounded to float32 alone moves them by up to 1e-2
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
def test_long_decoding_with_reused_pages_slots_and_graphs(dtype, vononex_dirs, cuda_kernels):
    """12 prompt tokens, then 300 decoded one by one beside requests that join and leave: page borders and windows are
    crossed by decoded tokens, the pages and the slot of a request that left serve the next one, decode steps replay a
    CUDA graph."""
    from inferflux_b200.engine import StepEntry
    d, page, raw = vononex_dirs["A"]
    reqs = vm.requests_for(raw, [312, 90, 60], 9)
    want = vm.plain_logits(d, reqs, weights_as=torch.bfloat16 if dtype == "bfloat16" else None)
    yard = vm.plain_logits(d, reqs, weights_as=torch.bfloat16, dtype=torch.bfloat16) if dtype == "bfloat16" else None
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
    for rid in reqs:
        if dtype == "float32":
            assert float(np.abs(got[rid] - want[rid]).max()) < 3e-4, rid
        else:
            _bf16_close(rid, got[rid], want[rid], yard[rid])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(dtype, vononex_dirs, oracle, tmp_path):
    d, page, raw = vononex_dirs["B"]
    o = oracle("B")
    steps = helpers.trace_mixed(o["reqs"], 256)
    got = helpers.collect(steps, helpers.run_trace_cli(d, dtype, steps, tmp_path / "out", 256, raw["vocab"], page_size=page),
                          raw["vocab"])
    _check("B through the program", dtype, got, o)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_engine_and_scheduler(dtype, vononex_dirs):
    from inferflux_b200 import Engine, SamplingParams
    d, page, raw = vononex_dirs["A"]
    _raw, W = vm.load(d)
    if dtype == "bfloat16":
        W = {k: (v.to(torch.bfloat16) if v.is_floating_point() else v) for k, v in W.items()}
    prompts = list(vm.requests_for(raw, [7, 19, 33, 4, 1, 70], 40).values())
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
