"""Sanarax without a GPU: the plain implementation's mechanisms against values worked out by hand, the
configuration and plan, and the engine's host logic (plan, cache and state manager, batching, scheduler)
run on the plain kernel table against the plain implementation."""
import copy
import math

import numpy as np
import pytest
import torch

import helpers
import sanarax_models as sm
from plain import plain_sanarax as P
from plain.plain_kernels import PlainKernels

F64 = torch.float64


@pytest.fixture(scope="module")
def sanarax_dirs(tmp_path_factory):
    out = {}
    for i, (name, (raw, page)) in enumerate(sm.configs().items()):
        out[name] = (sm.write_model(raw, tmp_path_factory.mktemp(f"sanarax_{name}"), seed=61 + i), page, raw)
    return out


# ------------------------------------------------------------------ mechanisms, by hand

def test_norm_weight_is_the_distance_from_one():
    x = torch.tensor([[3.0, -4.0]], dtype=F64)
    rms = math.sqrt(25 / 2 + 0.5)
    assert torch.allclose(P.norm(x, torch.tensor([0.0, 1.0], dtype=F64), 0.5), torch.tensor([[3 / rms, -8 / rms]], dtype=F64))


def test_both_pairings_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 9.0]], [[1.0, 2.0, 3.0, 4.0, 9.0]]], dtype=F64)      # two tokens, one head of five
    c, s, c2, s2 = math.cos(1), math.sin(1), math.cos(0.1), math.sin(0.1)            # frequencies 1 and 100^(-1/2)
    halves, near = P.rotate_halves(x, [0, 1], 4, 100.0), P.rotate_neighbours(x, [0, 1], 4, 100.0)
    assert torch.equal(halves[0], x[0]) and torch.equal(near[0], x[0])
    assert torch.allclose(halves[1, 0], torch.tensor([c - 3 * s, 2 * c2 - 4 * s2, 3 * c + s, 4 * c2 + 2 * s2, 9.0], dtype=F64))
    assert torch.allclose(near[1, 0], torch.tensor([c - 2 * s, 2 * c + s, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 9.0], dtype=F64))


def test_window_and_first_tokens_by_hand():
    seen = P.visible(7, 2, 1)
    assert [r.nonzero().flatten().tolist() for r in seen] == [[0], [0, 1], [0, 1, 2], [0, 2, 3], [0, 3, 4], [0, 4, 5], [0, 5, 6]]
    assert torch.equal(P.visible(7, 2, 0)[5].nonzero().flatten(), torch.tensor([4, 5]))
    assert P.visible(7, 1, 4)[6].nonzero().flatten().tolist() == [0, 1, 2, 3, 6]
    assert P.visible(3).tolist() == [[True, False, False], [True, True, False], [True, True, True]]


def test_sink_and_gate_by_hand():
    s = torch.tensor([[0.0, 5.0], [1.0, 2.0]], dtype=F64)
    w = P.softmax_rows(s, P.visible(2), torch.tensor(3.0, dtype=F64))
    e = [math.exp(1), math.exp(2), math.exp(3)]
    assert torch.allclose(w, torch.tensor([[1 / (1 + e[2]), 0.0], [e[0] / sum(e), e[1] / sum(e)]], dtype=F64))
    assert torch.allclose(P.softmax_rows(s, P.visible(2))[1], torch.tensor([e[0], e[1]], dtype=F64) / (e[0] + e[1]))
    o = torch.tensor([[[2.0, 4.0], [6.0, 8.0]]], dtype=F64)
    got = P.gate_heads(o, torch.tensor([[0.0, math.log(3.0)]], dtype=F64))
    assert torch.allclose(got, torch.tensor([[[1.0, 2.0], [4.5, 6.0]]], dtype=F64))


def test_values_are_the_keys_before_rotation_with_their_bias():
    W = {"a.q": torch.zeros(2, 2, dtype=F64), "a.q.b": torch.zeros(2, dtype=F64), "a.k": torch.eye(2, dtype=F64),
         "a.k.b": torch.tensor([0.5, -1.0], dtype=F64), "a.sink": torch.tensor([-1e9], dtype=F64), "a.g": torch.zeros(1, 2, dtype=F64),
         "a.o": torch.eye(2, dtype=F64)}
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0, "rot": {"base": 10.0, "dims": 2}, "mask": {"size": 2, "keep_first": 0}}
    h = torch.tensor([[1.0, 0.0], [3.0, 2.0], [5.0, 7.0]], dtype=F64)
    got = P.attention(h, W, "a.", m, [0, 1, 2])                                       # no query: the mean of the window, gated by 1/2
    assert torch.allclose(got[2], 0.5 * torch.tensor([4.5, 3.5], dtype=F64)) and torch.allclose(got[0], torch.tensor([0.75, -0.5], dtype=F64))


def test_latent_attention_by_hand():
    """One head, one latent number: keys and values follow from it; the rotated part alone tells the first token's key."""
    W = {"m.dq": torch.tensor([[1.0, 0.0]], dtype=F64), "m.dq.norm": torch.tensor([2.0], dtype=F64),
         "m.uq": torch.tensor([[0.0], [1.0], [0.0]], dtype=F64), "m.dkv": torch.tensor([[0.0, 1.0], [1.0, 0.0], [0.0, 0.0]], dtype=F64),
         "m.dkv.norm": torch.tensor([3.0], dtype=F64), "m.uk": torch.tensor([[0.7]], dtype=F64), "m.uv": torch.tensor([[1.0], [10.0]], dtype=F64),
         "m.g": torch.tensor([[0.0, 0.0]], dtype=F64), "m.o": torch.eye(2, dtype=F64)}
    m = {"heads": 1, "dim": 1, "rot_dim": 2, "vdim": 2, "kv_rank": 1, "q_rank": 1, "scale": 0.5, "rot": {"base": 10.0, "dims": 2}}
    h = torch.tensor([[1.0, 2.0], [1.0, -4.0]], dtype=F64)
    got = P.latent_attention(h, W, "m.", m, 1e-12, [0, 1])
    # c = 3, -3; q = (0 | 2, 0) and k = (0.7 c | 1, 0), both turned by their position: the scores are cos(1) and 1
    w0 = 1.0 / (1.0 + math.exp(1.0 - math.cos(1.0)))
    v = 3.0 * w0 - 3.0 * (1 - w0)
    assert torch.allclose(got, torch.tensor([[1.5, 15.0], [0.5 * v, 5.0 * v]], dtype=F64), atol=1e-9)


def test_lightning_by_hand():
    q = torch.tensor([[[2.0]], [[3.0]]], dtype=F64)
    k = torch.tensor([[[1.0]], [[-2.0]]], dtype=F64)
    v = torch.tensor([[[10.0]], [[1.0]]], dtype=F64)
    assert P.decay_scan(q, k, v, torch.tensor([0.25], dtype=F64))[:, 0, 0].tolist() == [20.0, 1.5]      # S: 10, 2.5 - 2
    two = P.decay_scan(q.repeat(1, 2, 1), k.repeat(1, 2, 1), v.repeat(1, 2, 1), torch.tensor([0.25, 1.0], dtype=F64))
    assert two[1, :, 0].tolist() == [1.5, 24.0]                                       # a decay per head
    W = {"r.q": torch.ones(2, 1, dtype=F64), "r.k": torch.ones(2, 1, dtype=F64), "r.v": torch.tensor([[3.0], [-4.0]], dtype=F64),
         "r.g": torch.tensor([[1.0], [2.0]], dtype=F64), "r.norm": torch.tensor([1.0, 2.0], dtype=F64), "r.o": torch.eye(2, dtype=F64)}
    m = {"heads": 2, "dim": 1, "vdim": 1, "decay": [0.5, 0.5]}
    a = lambda z: z / (1 + math.exp(-z))
    o = [a(1) * a(1) * a(3), a(1) * a(1) * a(-4)]                                     # both heads share one root mean square
    rms = math.sqrt((o[0] ** 2 + o[1] ** 2) / 2 + 0.5)
    want = [o[0] / rms / (1 + math.exp(-1)), 2 * o[1] / rms / (1 + math.exp(-2))]
    assert torch.allclose(P.lightning(torch.tensor([[1.0]], dtype=F64), W, "r.", m, 0.5)[0], torch.tensor(want, dtype=F64))


def test_feed_forward_by_hand():
    W = {"f.up": torch.tensor([[1.0], [-1.0]], dtype=F64), "f.down": torch.tensor([[3.0, 5.0]], dtype=F64)}
    assert P.feed_forward(torch.tensor([[2.0], [-3.0], [0.0]], dtype=F64), W, "f.")[:, 0].tolist() == [12.0, 45.0, 0.0]


# ------------------------------------------------------------------ every option changes the result

def test_every_option_matters(sanarax_dirs):
    for name in ("A", "B", "C"):
        d, _page, raw = sanarax_dirs[name]
        _raw, W = sm.load(d)
        toks = sm.requests_for(raw, [36], 9)["r0"]
        base = P.forward(raw, W, toks)

        def differs(other_raw=None, other_W=None):
            return float((P.forward(other_raw or raw, other_W or W, toks) - base).abs().max())

        def edit(kind, path, f):
            """config.json with the mixer entry at `path` changed by f in every layer of that kind."""
            r = copy.deepcopy(raw)
            for lay in r["layers"]:
                if lay["type"] == kind:
                    m = lay["mixer"]
                    for key in path[:-1]:
                        m = m[key]
                    m[path[-1]] = f(m[path[-1]])
            return r
        for n in W:
            assert differs(other_W={**W, n: W[n].roll(1, 0) + 0.01}) > 1e-7, (name, n)
        assert differs({**raw, "embedding": {"scale": 1.1 * raw["embedding"]["scale"]}}) > 1e-4
        assert differs({**raw, "logit_scale": 1.1 * raw["logit_scale"]}) > 1e-4 and differs({**raw, "norm": {"eps": 30 * raw["norm"]["eps"]}}) > 1e-9
        for kind, path, f in (("attention", ("scale",), lambda v: v * 1.1), ("attention", ("mask", "size"), lambda v: v + 1 if v < 36 else v - 60),
                              ("attention", ("mask", "keep_first"), lambda v: v + 1), ("latent_attention", ("scale",), lambda v: v * 1.1),
                              ("latent_attention", ("rot", "base"), lambda v: v * 1.5), ("lightning", ("decay",), lambda v: [x * 0.97 for x in v])):
            assert differs(edit(kind, path, f)) > 1e-6, (name, kind, path)
        # one more run of a layer that is there already counts
        if raw["layers"][-1].get("weights_of") is not None:
            assert differs({**raw, "layers": raw["layers"][:-1]}) > 1e-3


# ------------------------------------------------------------------ configuration and plan

def test_config_round_trip_and_plan(sanarax_dirs):
    from inferflux_b200.config import ConfigError, SanaraxConfig, config_from_dict, load_config
    from inferflux_b200.models.model import Model
    d, _page, raw = sanarax_dirs["A"]
    cfg = load_config(d)
    assert isinstance(cfg, SanaraxConfig) and cfg.to_dict() == raw
    plan = cfg.to_plan()
    assert [l.mixer.kind for l in plan.layers] == ["attention", "latent_attention", "lightning", "attention"]
    assert [l.prefix for l in plan.layers] == ["l0.", "l1.", "l2.", "l4."] and {l.block.kind for l in plan.layers} == {"sandwich"}
    assert [(e.layer, e.cache, e.writes_cache) for e in plan.schedule] == [(0, 0, True), (1, 1, True), (2, 2, True), (0, 3, True),
                                                                           (3, 4, True), (2, 5, True), (1, 6, True)]
    model = Model(plan)
    exp = model.expected_tensors()
    assert set(exp) == set(sm.load(d)[1])
    assert exp["l0.mix.k"].shape == (32, 72) and exp["l0.mix.g"].shape == (4, 72) and exp["l1.mix.dkv"].shape == (28, 72)
    assert exp["l2.mix.norm"].shape == (60,) and not {"l0.mix.v", "l2.norm2", "l3.norm1", "l5.mix.q"} & set(exp)
    specs = model.cache_specs()
    kv = specs[0][0]
    assert (kv.num_kv_heads, kv.head_dim, kv.window, kv.keep_first) == (2, 16, 24, 5) and specs[3][0] == kv and specs[0][1] is None
    assert (specs[1][0].num_kv_heads, specs[1][0].head_dim, specs[1][0].planes, specs[1][0].window) == (1, 28, 1, None)
    assert specs[2][0] is None and specs[2][1].shape == (3 * 12 * 20,) and specs[5][1] == specs[2][1]
    att, lat, lig = raw["layers"][:3]

    def one(lay, **kw):
        return {**raw, "layers": [{**lay, "mixer": {**lay["mixer"], **kw}}]}
    for bad in ({**raw, "layers": []}, {**raw, "layers": [{**att, "type": "other"}]}, {k: v for k, v in raw.items() if k != "width"},
                one(att, kv_heads=3), one(att, vdim=8), one(att, dim=15, vdim=15), one(att, rot={"base": 10.0, "dims": 18}),
                one(att, rot=None), one(att, mask={"size": 0}), one(att, mask={"size": 4, "keep_first": -1}), one(att, scale=0.0),
                one(lat, q_rank=None), one(lat, kv_rank=1022), one(lat, rot={"base": 10.0, "dims": 6}), one(lig, decay=[0.5]), one(lig, dim=600),
                {**raw, "layers": [{**att, "mlp": {"kind": "moe", "ff": 3}}]}, {**raw, "layers": [att, {**att, "weights_of": 1}]},
                {**raw, "layers": [att, {**lig, "weights_of": 0}]}, {**raw, "layers": [att, {**att, "mlp": None, "weights_of": 0}]},
                {**raw, "layers": [att, {**att, "weights_of": 0}, {**att, "weights_of": 1}]}, {**raw, "logit_scale": "big"}):
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_wrong_weights_are_refused(sanarax_dirs, tmp_path):
    from inferflux_b200.models import load_model
    from inferflux_b200.weights import WeightError, write_safetensors
    d, _page, _raw = sanarax_dirs["A"]
    _raw, W = sm.load(d)
    (tmp_path / "config.json").write_text((d / "config.json").read_text())
    W2 = {k: v for k, v in W.items() if k not in ("l0.mix.sink", "l1.mix.dq.norm")}
    W2["l0.mix.g"] = W["l0.mix.g"][:-1].contiguous()
    W2["l3.norm1"] = W["l0.norm1"].clone()
    write_safetensors(tmp_path / "model.safetensors", W2)
    with pytest.raises(WeightError) as e:
        load_model(tmp_path, dtype="float32", device="cpu")
    assert e.value.missing == ["l0.mix.sink", "l1.mix.dq.norm"] and e.value.unexpected == ["l3.norm1"]
    assert [w[0] for w in e.value.wrong_shape] == ["l0.mix.g"]


# ------------------------------------------------------------------ pages of the first tokens

@pytest.mark.parametrize("keep,window", [(0, 6), (1, 6), (4, 6), (5, 6), (9, 2), (3, 1)])
def test_cache_holds_the_first_tokens_and_the_window_and_no_more(keep, window):
    from inferflux_b200.cache.manager import CacheManager
    from inferflux_b200.parts.base import KVCacheSpec
    m = CacheManager([(KVCacheSpec(1, 8, window, keep_first=keep), None)], page_size=4, num_pages=12, max_seqs=2, max_seq_len=200)
    m.add_request("r")
    length, firsts = 0, None
    for n in (3, 1, 9, 1, 1, 1, 1, 17, 1, 1, 30) + (1,) * 20:
        m.reserve("r", length + n)
        held = m.pages_of("r")
        need = {j // 4 for i in range(length, length + n) for j in range(i + 1) if i - j < window or j < keep}
        assert need <= set(held)                          # everything this step's queries see has a page
        length += n
        m.commit("r", length)
        held = m.pages_of("r")
        later = {j // 4 for j in range(length) if length - j < window or j < keep} | ({length // 4} if length % 4 else set())
        assert set(held) == later                         # what the next token sees or writes to, and nothing else
        kept = {b: held[b] for b in range(-(-keep // 4)) if b in held}
        if length > keep:
            assert firsts is None or kept == firsts       # the same pages all along
            firsts = kept
        m.check()
    m.free("r")
    assert m.free_pages() == [12]
    m.check()


# ------------------------------------------------------------------ the engine's host logic on plain kernels

LENS = [40, 33, 50, 61, 97, 70, 25, 64, 1, 2]


def _plain_runner(d, page, pages=None, max_seqs=4, max_seq_len=512):
    from inferflux_b200.engine import ModelRunner
    from inferflux_b200.models import load_model
    _c, model = load_model(d, dtype="float32", device="cpu")
    return ModelRunner(model, PlainKernels(wide=True), page_size=page, num_pages=pages or 256 // page, max_seqs=max_seqs,
                       max_seq_len=max_seq_len)


@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("cutting", ["whole", "portions", "mixed"])
def test_engine_host_logic_on_plain_kernels(name, cutting, sanarax_dirs):
    d, page, raw = sanarax_dirs[name]
    reqs = sm.requests_for(raw, LENS, 100)
    want = sm.plain_logits(d, reqs)
    steps = {"whole": helpers.trace_whole, "portions": helpers.trace_portions,
             "mixed": lambda r: helpers.trace_mixed(r, 256)}[cutting](reqs)
    runner = _plain_runner(d, page)
    got = helpers.collect(steps, helpers.run_steps_in_process(runner, steps), raw["vocab"])
    bad = helpers.first_bad(got, want, 3e-4)
    assert bad is None, f"first wrong row (request, position, diff): {bad}"
    assert not runner.cache.live_requests() and runner.cache.free_pages() == [256 // page] * len(runner.cache.groups)


def test_portions_down_to_two_tokens_and_the_first_tokens(sanarax_dirs):
    """Portions of 2, 1, 3, 2, 2, 5 ... tokens from the first token on: the recurrences read the state that the portion
    before left (and zeros before the sequence's start), attention its pages and the first tokens' pages."""
    from inferflux_b200.engine import StepEntry
    for name in ("A", "C"):
        d, page, raw = sanarax_dirs[name]
        toks = sm.requests_for(raw, [60], 3)["r0"]
        want = sm.plain_logits(d, {"r0": toks})["r0"]
        runner = _plain_runner(d, page)
        got, pos, sizes, i = [], 0, [2, 1, 3, 2, 2, 5, 1, 1, 2, 17], 0
        while pos < len(toks):
            n = min(sizes[i % len(sizes)], len(toks) - pos)
            i += 1
            got += list(runner.step([StepEntry("r0", toks[pos:pos + n], list(range(n)))]).double().numpy())
            pos += n
        runner.end_request("r0")
        assert float(np.abs(np.stack(got) - want).max()) < 3e-4, name


def test_a_slot_and_pages_that_are_used_again_start_clean(sanarax_dirs):
    from inferflux_b200.engine import StepEntry
    d, page, raw = sanarax_dirs["A"]
    reqs = sm.requests_for(raw, [9, 1, 3, 2, 30, 5], 7)
    want = sm.plain_logits(d, reqs)
    runner = _plain_runner(d, page, pages=4, max_seqs=1, max_seq_len=32)
    for rid, toks in reqs.items():                         # one slot, four pages: everybody inherits them
        got = runner.step([StepEntry(rid, toks, list(range(len(toks))))]).double().numpy()
        assert float(np.abs(got - want[rid]).max()) < 3e-4, rid
        runner.end_request(rid)
        runner.cache.check()
    assert all(g.alloc.allocations > 4 for g in runner.cache.groups)


def test_greedy_generation_through_engine_and_scheduler(sanarax_dirs):
    from inferflux_b200 import Engine, SamplingParams
    d, page, raw = sanarax_dirs["A"]
    _raw, W = sm.load(d)
    prompts = list(sm.requests_for(raw, [7, 19, 33, 4, 1], 40).values())

    def greedy(prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(P.forward(raw, W, seq)[-1].argmax()))
        return seq[len(prompt):]
    want = [greedy(p, 12) for p in prompts]
    for pages in (64, 8):                                  # 8 pages of 8: the requests do not all fit at once
        eng = Engine(d, dtype="float32", device="cpu", kernels=PlainKernels(wide=True), kv_page_size=page,
                     kv_num_pages=pages, kv_max_batch=4, kv_max_seq=128, chunked_prefill_tokens=16, max_batch_tokens=48)
        res = eng.generate(prompts, SamplingParams(temperature=0.0), max_tokens=12)
        assert [r.token_ids for r in res] == want
        assert not eng.runner.cache.live_requests()


def test_command_line_info_and_random_model(sanarax_dirs, tmp_path, capsys):
    import json
    from inferflux_b200.cli.main import main
    _d, _page, raw = sanarax_dirs["B"]
    (tmp_path / "config.json").write_text(json.dumps(raw))
    assert main(["random-model", "--config", str(tmp_path / "config.json"), "--seed", "3", "--out", str(tmp_path / "m")]) == 0
    capsys.readouterr()
    assert main(["info", "--model", str(tmp_path / "m")]) == 0
    assert "Sanarax" in capsys.readouterr().out
