"""Vononex without a GPU: the plain implementation's mechanisms against values worked out by hand, the
configuration and plan, and the engine's host logic (plan, cache and state manager, batching, scheduler)
run on the plain kernel table against the plain implementation."""
import copy
import math

import numpy as np
import pytest
import torch

import helpers
import vononex_models as vm
from plain import plain_vononex as P
from plain.plain_kernels import PlainKernels

F64 = torch.float64


@pytest.fixture(scope="module")
def vononex_dirs(tmp_path_factory):
    out = {}
    for i, (name, (raw, page)) in enumerate(vm.configs().items()):
        out[name] = (vm.write_model(raw, tmp_path_factory.mktemp(f"vononex_{name}"), seed=51 + i), page, raw)
    return out


# ------------------------------------------------------------------ mechanisms, by hand

def test_norm_of_the_sum_by_hand():
    x, y = torch.tensor([[1.0, -2.0]], dtype=F64), torch.tensor([[1.0, 1.0]], dtype=F64)
    got = P.sum_norm(x, y, 3.0, torch.tensor([1.0, 10.0], dtype=F64), 0.5)          # the sum is (4, -5)
    rms = math.sqrt((16 + 25) / 2 + 0.5)
    assert torch.allclose(got, torch.tensor([[4 / rms, -50 / rms]], dtype=F64))


def test_rotation_of_halves_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 9.0]], [[1.0, 2.0, 3.0, 4.0, 9.0]]], dtype=F64)      # two tokens, one head of five
    got = P.rotate_halves(x, [0, 1], 4, 100.0)
    assert torch.equal(got[0], x[0])
    c, s, c2, s2 = math.cos(1), math.sin(1), math.cos(0.1), math.sin(0.1)            # frequencies 1 and 100^(-1/2)
    assert torch.allclose(got[1, 0], torch.tensor([c - 3 * s, 2 * c2 - 4 * s2, 3 * c + s, 4 * c2 + 2 * s2, 9.0], dtype=F64))
    assert torch.allclose(P.rotate_halves(got, [0, 1], 4, 100.0, direction=-1.0), x)


def test_attention_scale_temp_and_grouping_by_hand():
    q = torch.tensor([[[1.0], [2.0]], [[1.0], [2.0]]], dtype=F64)                     # two tokens, two heads, one key head
    k = torch.tensor([[[0.0]], [[1.0]]], dtype=F64)
    v = torch.tensor([[[10.0]], [[20.0]]], dtype=F64)
    got = P.attend(q, k, v, 0.5, torch.tensor([2.0, 3.0], dtype=F64))
    assert got[0, :, 0].tolist() == [10.0, 10.0]                                      # the first token sees itself alone
    for h, score in ((0, 1.0), (1, 3.0)):
        w = math.exp(score) / (1 + math.exp(score))
        assert abs(float(got[1, h, 0]) - (10 * (1 - w) + 20 * w)) < 1e-12


def test_queries_and_keys_are_normed_over_all_heads_together():
    W = {"a.q": torch.eye(4, dtype=F64), "a.k": torch.eye(4, dtype=F64), "a.v": torch.eye(4, dtype=F64), "a.o": torch.eye(4, dtype=F64),
         **{f"a.{s}.b": torch.zeros(4, dtype=F64) for s in "qkvo"}, "a.q.norm": torch.ones(4, dtype=F64),
         "a.k.norm": torch.ones(4, dtype=F64), "a.temp": torch.ones(2, dtype=F64)}
    m = {"heads": 2, "kv_heads": 2, "dim": 2, "vdim": 2, "scale": 1.0, "rot": {"base": 10.0, "dims": 2}}
    h = torch.tensor([[3.0, 0.0, 0.0, 0.0], [3.0, 0.0, 0.0, 1e-3]], dtype=F64)
    got = P.attention(h, W, "a.", m, 0.0, [0, 1])
    # the second head's key is tiny beside the first head's, and stays so: its two scores are almost equal
    q = P.unit_rms(h, 0.0).view(2, 2, 2)
    assert float(q[1, 1].norm()) < 1e-3 and float(q[1, 0].norm()) > 1.9
    assert torch.allclose(got[1, 3], torch.tensor(1e-3 / 2, dtype=F64), rtol=1e-3)


def test_turned_values_depend_on_distances_only():
    """Values turned by their own position and turned back by the query's: moving a whole sequence changes nothing, and a
    value's share arrives turned by minus the distance."""
    g = torch.Generator().manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    H, d, dv = 2, 4, 6
    W = {"a.q": rnd(H * d, 5), "a.k": rnd(H * d, 5), "a.v": rnd(H * dv, 5), "a.o": rnd(7, H * dv), "a.q.b": rnd(H * d), "a.k.b": rnd(H * d),
         "a.v.b": rnd(H * dv), "a.o.b": rnd(7), "a.q.norm": 1 + rnd(H * d), "a.k.norm": 1 + rnd(H * d), "a.temp": rnd(H)}
    m = {"heads": H, "kv_heads": H, "dim": d, "vdim": dv, "scale": 0.4, "rot": {"base": 30.0, "dims": 2}}
    h = rnd(6, 5)
    assert torch.allclose(P.attention(h, W, "a.", m, 1e-6, range(6)), P.attention(h, W, "a.", m, 1e-6, range(100, 106)))
    # keys zero: uniform weights; the output is the mean of the values, each turned by minus its distance
    W.update({"a.k": 0 * W["a.k"], "a.k.b": 0 * W["a.k.b"]})
    v = (h @ W["a.v"].T + W["a.v.b"]).view(6, H, dv)
    want = sum(P.rotate_halves(v[j:j + 1], [j - 5], dv, 30.0) for j in range(6)) / 6
    assert torch.allclose(P.attention(h, W, "a.", m, 1e-6, range(6))[5], want.reshape(-1) @ W["a.o"].T + W["a.o.b"])


def test_retention_by_hand():
    q = torch.tensor([[[2.0]], [[3.0]]], dtype=F64)
    k = torch.tensor([[[1.0]], [[-2.0]]], dtype=F64)
    v = torch.tensor([[[10.0]], [[1.0]]], dtype=F64)
    assert P.retention_scan(q, k, v, torch.tensor([0.25], dtype=F64))[:, 0, 0].tolist() == [20.0, 1.5]      # S: 10, 2.5 - 2
    two = P.retention_scan(q.repeat(1, 2, 1), k.repeat(1, 2, 1), v.repeat(1, 2, 1), torch.tensor([0.25, 1.0], dtype=F64))
    assert two[1, :, 0].tolist() == [1.5, 24.0]                                       # a decay per head
    W = {"r.q": torch.full((4, 1), 1.0, dtype=F64), "r.k": torch.full((4, 1), 1.0, dtype=F64), "r.v": torch.tensor([[3.0], [4.0]], dtype=F64),
         "r.g": torch.tensor([[1.0], [2.0]], dtype=F64), "r.o": torch.eye(2, dtype=F64)}
    m = {"heads": 1, "dim": 4, "vdim": 2, "rot": {"base": 10.0, "dims": 2}, "decay": [0.5]}
    got = P.retention(torch.tensor([[1.0]], dtype=F64), W, "r.", m, 0.5, [0])
    o = torch.tensor([3.0, 4.0], dtype=F64) * 4 * 0.5                                 # q . k = 4, keys times 4^(-1/2)
    o = o / math.sqrt((36 + 64) / 2 + 0.5)
    assert torch.allclose(got[0], o * P.silu(torch.tensor([1.0, 2.0], dtype=F64)))


def test_gated_recurrence_by_hand():
    assert P.gated_scan(torch.tensor([[0.5], [0.25], [1.0]], dtype=F64), torch.tensor([[4.0], [-2.0], [7.0]], dtype=F64))[:, 0].tolist() == [
        2.0, 0.75 * 2 - 0.5, 7.0]
    W = {"m.z": torch.zeros(1, 1, dtype=F64), "m.z.b": torch.zeros(1, dtype=F64), "m.x": torch.ones(1, 1, dtype=F64),
         "m.x.b": torch.zeros(1, dtype=F64), "m.g": torch.zeros(1, 1, dtype=F64), "m.o": torch.ones(1, 1, dtype=F64)}
    W["m.g"] = torch.full((1, 1), 1.0, dtype=F64)
    for u, cand in ((2.0, 2.5), (0.0, 0.5), (-1.0, 1 / (1 + math.exp(1.0)))):          # continuous at zero
        got = P.mingru(torch.tensor([[u]], dtype=F64), W, "m.")
        assert abs(float(got) - 0.5 * cand * u / (1 + math.exp(-u))) < 1e-12


def test_feed_forward_by_hand():
    z = torch.tensor([-1.5, 0.0, 0.7], dtype=F64)
    want = [0.5 * v * (1 + math.tanh(math.sqrt(2 / math.pi) * (v + 0.044715 * v ** 3))) for v in z.tolist()]
    assert torch.allclose(P.gelu_tanh(z), torch.tensor(want, dtype=F64))
    W = {"f.gate": torch.tensor([[1.0]], dtype=F64), "f.gate.b": torch.tensor([0.2], dtype=F64), "f.up": torch.tensor([[2.0]], dtype=F64),
         "f.up.b": torch.tensor([-1.0], dtype=F64), "f.down": torch.tensor([[3.0]], dtype=F64), "f.down.b": torch.tensor([0.5], dtype=F64)}
    assert abs(float(P.feed_forward(torch.tensor([[0.5]], dtype=F64), W, "f.")) - 0.5) < 1e-12      # the up row is 0: the bias alone
    got = float(P.feed_forward(torch.tensor([[1.0]], dtype=F64), W, "f."))
    assert abs(got - (3 * float(P.gelu_tanh(torch.tensor(1.2, dtype=F64))) * 1.0 + 0.5)) < 1e-12


# ------------------------------------------------------------------ every option changes the result

def test_every_option_matters(vononex_dirs):
    for name in ("A", "B", "C"):
        d, _page, raw = vononex_dirs[name]
        _raw, W = vm.load(d)
        toks = vm.requests_for(raw, [40], 9)["r0"]
        base = P.forward(raw, W, toks)

        def differs(other_raw=None, other_W=None):
            return float((P.forward(other_raw or raw, other_W or W, toks) - base).abs().max())

        def edit(path, f):
            """config.json with every mixer entry at `path` changed by f."""
            r = copy.deepcopy(raw)
            hit = 0
            for lay in r["layers"]:
                m = lay["mixer"]
                for key in path[:-1]:
                    m = m.get(key) or {}
                if path[-1] in m:
                    m[path[-1]] = f(m[path[-1]])
                    hit += 1
            assert hit, path
            return r
        for n in sorted({n.split(".", 1)[1] if n[0] == "l" and "." in n else n for n in W}):
            # (a single key head's norm weight and the like: roll changes what scaling would not)
            some = {k: (v.roll(1, 0) + 0.01 if k == n or k.endswith("." + n) else v) for k, v in W.items()}
            assert differs(other_W=some) > 1e-7, (name, n)
        assert differs({**raw, "postln_alpha": raw["postln_alpha"] + 0.1}) > 1e-6 and differs({**raw, "norm": {"eps": raw["norm"]["eps"] * 30}}) > 1e-9
        for path, f in ((("left", "scale"), lambda v: v * 1.1), (("left", "rot", "base"), lambda v: v * 1.5), (("right", "rot", "base"), lambda v: v * 1.5),
                        (("right", "decay"), lambda v: [x * 0.97 for x in v]), (("left_scale",), lambda v: v * 1.1),
                        (("right_scale",), lambda v: v * 1.1)):
            if path == ("right", "rot", "base") and all(l["mixer"]["right"]["rot"]["dims"] == 2 for l in raw["layers"] if l["type"] == "parallel"):
                continue                                   # one frequency, which no base changes
            assert differs(edit(path, f)) > 1e-6, (name, path)


# ------------------------------------------------------------------ configuration and plan

def test_config_round_trip_and_plan(vononex_dirs):
    from inferflux_b200.config import ConfigError, VononexConfig, config_from_dict, load_config
    from inferflux_b200.models.model import Model
    d, _page, raw = vononex_dirs["A"]
    cfg = load_config(d)
    assert isinstance(cfg, VononexConfig) and cfg.to_dict() == raw
    plan = cfg.to_plan()
    assert [l.block.kind for l in plan.layers] == ["norm_of_sum"] * 4
    assert [l.mixer.kind for l in plan.layers] == ["pair", "min_gru", "pair", "min_gru"]
    model = Model(plan)
    exp = model.expected_tensors()
    assert set(exp) == set(vm.load(d)[1])
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.left.q.b", "l0.mix.left.q.norm", "l0.mix.left.temp",
            "l0.mix.left.o.b", "l0.mix.right.g", "l0.mlp.down.b", "l1.mix.z.b", "l1.mix.o"} <= set(exp)
    assert not {"l2.norm2", "l2.mlp.gate", "l3.norm2", "l0.mix.right.q.b", "l1.mix.g.b", "l1.mix.o.b"} & set(exp)
    assert exp["l0.mix.left.q.norm"].shape == (64,) and exp["l0.mix.left.k.norm"].shape == (32,) and exp["l0.mix.left.temp"].shape == (4,)
    specs = model.cache_specs()
    kv, st = specs[0]
    assert (kv.num_kv_heads, kv.head_dim, kv.window) == (2, 16, None) and st.shape == (3 * 12 * 20,)
    assert specs[1][0] is None and specs[1][1].shape == (104,)
    lay = raw["layers"][0]

    def with_mixer(**kw):
        return {**raw, "layers": [{**lay, "mixer": {**lay["mixer"], **kw}}]}
    left, right = lay["mixer"]["left"], lay["mixer"]["right"]
    for bad in ({**raw, "layers": []}, {**raw, "layers": [{**lay, "type": "other"}]}, {k: v for k, v in raw.items() if k != "postln_alpha"},
                {k: v for k, v in raw.items() if k != "width"}, with_mixer(right=None), with_mixer(left={**left, "kv_heads": 3}),
                with_mixer(left={**left, "rot": {"base": 100.0, "dims": 7}}), with_mixer(left={**left, "vdim": 7}),
                with_mixer(left={k: v for k, v in left.items() if k != "rot"}), with_mixer(right={**right, "decay": [0.5]}),
                with_mixer(right={**right, "dim": 600, "rot": {"base": 9.0, "dims": 4}}), with_mixer(left_scale=None),
                {**raw, "layers": [{**lay, "mlp": {"kind": "moe", "ff": 3}}]}, {**raw, "layers": [{"type": "mingru", "mixer": {}, "mlp": None}]}):
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_wrong_weights_are_refused(vononex_dirs, tmp_path):
    from inferflux_b200.models import load_model
    from inferflux_b200.weights import WeightError, write_safetensors
    d, _page, _raw = vononex_dirs["A"]
    _raw, W = vm.load(d)
    (tmp_path / "config.json").write_text((d / "config.json").read_text())
    W2 = {k: v for k, v in W.items() if k not in ("l0.mix.left.temp", "l1.mlp.gate.b")}
    W2["l0.mix.left.q.norm"] = W["l0.mix.left.q.norm"][:-1].contiguous()
    W2["l1.mix.g.b"] = W["l1.mix.z.b"].clone()
    write_safetensors(tmp_path / "model.safetensors", W2)
    with pytest.raises(WeightError) as e:
        load_model(tmp_path, dtype="float32", device="cpu")
    assert e.value.missing == ["l0.mix.left.temp", "l1.mlp.gate.b"] and e.value.unexpected == ["l1.mix.g.b"]
    assert [w[0] for w in e.value.wrong_shape] == ["l0.mix.left.q.norm"]


# ------------------------------------------------------------------ the engine's host logic on plain kernels

LENS = [40, 33, 50, 61, 97, 70, 25, 64, 1, 2]


def _plain_runner(d, page, pages=None, max_seqs=4, max_seq_len=512):
    from inferflux_b200.engine import ModelRunner
    from inferflux_b200.models import load_model
    _c, model = load_model(d, dtype="float32", device="cpu")
    return ModelRunner(model, PlainKernels(wide=True), page_size=page, num_pages=pages or 256 // page, max_seqs=max_seqs,
                       max_seq_len=max_seq_len)


@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("cutting", ["whole", "tail", "portions", "mixed"])
def test_engine_host_logic_on_plain_kernels(name, cutting, vononex_dirs):
    d, page, raw = vononex_dirs[name]
    reqs = vm.requests_for(raw, LENS, 100)
    want = vm.plain_logits(d, reqs)
    steps = {"whole": helpers.trace_whole, "tail": helpers.trace_tail, "portions": helpers.trace_portions,
             "mixed": lambda r: helpers.trace_mixed(r, 256)}[cutting](reqs)
    runner = _plain_runner(d, page)
    got = helpers.collect(steps, helpers.run_steps_in_process(runner, steps), raw["vocab"])
    bad = helpers.first_bad(got, want, 2e-4)
    assert bad is None, f"first wrong row (request, position, diff): {bad}"
    pools = [256 // page] * len(runner.cache.groups)
    assert not runner.cache.live_requests() and runner.cache.free_pages() == pools


def test_portions_down_to_two_tokens_and_the_first_tokens(vononex_dirs):
    """Portions of 2, 1, 3, 2, 2, 5 ... tokens from the first token on: the recurrences read the state that the portion
    before left (and zeros before the sequence's start), attention its pages."""
    from inferflux_b200.engine import StepEntry
    for name in ("A", "C"):
        d, page, raw = vononex_dirs[name]
        toks = vm.requests_for(raw, [60], 3)["r0"]
        want = vm.plain_logits(d, {"r0": toks})["r0"]
        runner = _plain_runner(d, page)
        got, pos, sizes, i = [], 0, [2, 1, 3, 2, 2, 5, 1, 1, 2, 17], 0
        while pos < len(toks):
            n = min(sizes[i % len(sizes)], len(toks) - pos)
            i += 1
            got += list(runner.step([StepEntry("r0", toks[pos:pos + n], list(range(n)))]).double().numpy())
            pos += n
        runner.end_request("r0")
        assert float(np.abs(np.stack(got) - want).max()) < 2e-4, name


def test_a_slot_and_pages_that_are_used_again_start_clean(vononex_dirs):
    from inferflux_b200.engine import StepEntry
    d, page, raw = vononex_dirs["A"]
    reqs = vm.requests_for(raw, [9, 1, 3, 2, 30, 5], 7)
    want = vm.plain_logits(d, reqs)
    runner = _plain_runner(d, page, pages=4, max_seqs=1, max_seq_len=32)
    for rid, toks in reqs.items():                         # one slot, four pages: everybody inherits them
        got = runner.step([StepEntry(rid, toks, list(range(len(toks))))]).double().numpy()
        assert float(np.abs(got - want[rid]).max()) < 2e-4, rid
        assert all(float(s[0].double().abs().max()) > 0 for s in runner.cache.state if s is not None)
        runner.end_request(rid)
        runner.cache.check()
    assert all(g.alloc.allocations > 4 for g in runner.cache.groups)


def test_greedy_generation_through_engine_and_scheduler(vononex_dirs):
    from inferflux_b200 import Engine, SamplingParams
    d, page, raw = vononex_dirs["A"]
    _raw, W = vm.load(d)
    prompts = list(vm.requests_for(raw, [7, 19, 33, 4, 1], 40).values())

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


def test_command_line_info_and_random_model(vononex_dirs, tmp_path, capsys):
    import json
    from inferflux_b200.cli.main import main
    _d, _page, raw = vononex_dirs["B"]
    (tmp_path / "config.json").write_text(json.dumps(raw))
    assert main(["random-model", "--config", str(tmp_path / "config.json"), "--seed", "3", "--out", str(tmp_path / "m")]) == 0
    capsys.readouterr()
    assert main(["info", "--model", str(tmp_path / "m")]) == 0
    assert "Vononex" in capsys.readouterr().out
