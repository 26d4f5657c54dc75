"""Small Vononex models for the tests: configurations that differ in every size and option, random weights made sharp,
and the plain implementation's logits for a set of requests."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from plain import plain_vononex


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _parallel(left, right, scales, mlp):
    """left: (heads, kv_heads, dim, vdim, scale, rot base, rot dims); right: (dim, vdim, rot base, rot dims, decays)."""
    h, g, d, dv, scale, base, dims = left
    rd, rv, rbase, rdims, decay = right
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": h, "kv_heads": g, "dim": d, "vdim": dv, "scale": scale, "rot": {"base": base, "dims": dims}},
        "right": {"heads": len(decay), "dim": rd, "vdim": rv, "rot": {"base": rbase, "dims": rdims}, "decay": list(decay)},
        "left_scale": scales[0], "right_scale": scales[1]}}


def _mingru(width, mlp):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def configs():
    """name -> (config.json as a dict, page size).  Between them: both layer kinds first, last, alone and repeated; grouped,
    ungrouped and single key heads; values longer and shorter than keys and of the same size; rotation of the whole head
    and of a part of it, by bases of their own on either side; recurrent heads whose key and value sizes are no
    multiples of anything, one head and several, decays from fast to none at all; gated recurrences narrower and wider
    than the model; layers without feed-forward; alphas above, below and at one; eps small and large."""
    a = {"architecture": "Vononex", "vocab": 310, "width": 72, "norm": {"eps": 1e-6}, "postln_alpha": 2.2, "layers": [
        _parallel((4, 2, 16, 8, 0.3, 500.0, 16), (12, 20, 3000.0, 12, [0.9, 0.999, 0.5]), (0.8, 1.4), _dense(88)),
        _mingru(104, _dense(40)),
        _parallel((2, 2, 24, 24, 0.21, 40.0, 8), (8, 8, 100.0, 4, [1.0]), (1.3, 0.7), None),
        _mingru(24, None)]}
    b = {"architecture": "Vononex", "vocab": 259, "width": 96, "norm": {"eps": 2e-4}, "postln_alpha": 1.0, "layers": [
        _mingru(96, None), _mingru(160, _dense(64)),
        _parallel((6, 1, 8, 32, 0.5, 2000.0, 4), (24, 6, 50.0, 24, [0.97, 0.75]), (1.0, 1.0), _dense(200))]}
    c = {"architecture": "Vononex", "vocab": 151, "width": 50, "norm": {"eps": 1e-5}, "postln_alpha": 0.6, "layers": [
        _parallel((3, 3, 10, 6, 0.45, 90.0, 10), (5 * 2, 7, 900.0, 6, [0.98, 0.6, 0.9995, 0.8, 0.99]), (-0.7, 1.1), _dense(33)),
        _parallel((5, 1, 14, 14, 0.27, 25.0, 2), (6, 3, 10.0, 2, [0.9]), (0.5, 2.0), _dense(75))]}
    return {"A": (a, 8), "B": (b, 4), "C": (c, 16)}


def medium_config():
    """A model of a few hundred columns whose prompts are long enough for the kernels of many rows: attention heads of 64
    and 128 with equal key and value sizes on pages of 16 (the tiled attention kernels), a head size that only the
    mma.sync tiles take, recurrent heads of 32 to 128 key channels, a gated recurrence wider than a block's channels."""
    return {"architecture": "Vononex", "vocab": 705, "width": 320, "norm": {"eps": 1e-6}, "postln_alpha": 1.7, "layers": [
        _parallel((4, 2, 64, 64, 0.14, 10000.0, 64), (64, 48, 5000.0, 64, [0.99, 0.9999, 0.7]), (1.1, 0.6), _dense(448)),
        _mingru(456, _dense(320)),
        _parallel((6, 3, 128, 128, 0.1, 700.0, 64), (128, 64, 20000.0, 96, [0.95, 0.995]), (0.9, 0.8), None),
        _parallel((8, 2, 32, 32, 0.2, 300.0, 16), (32, 128, 60.0, 32, [0.9, 0.98, 0.999, 0.5]), (1.2, 0.5), _dense(192))]}, 16


def write_model(raw, out_dir, seed):
    """Random weights for `raw`, then made sharp: norm weights and factors per head are spread (and queries and keys large
    through them, so that attention is peaked), the embedding's rows differ, biases are not small, gates of the
    recurrences spread from shut to open."""
    from inferflux_b200.config import config_from_dict
    from inferflux_b200.weights import SafetensorsFile, write_random_model, write_safetensors
    cfg = config_from_dict(raw)
    write_random_model(cfg, out_dir, seed=seed, dtype=torch.float32, std=0.08, norm_jitter=0.2)
    path = Path(out_dir) / "model.safetensors"
    with SafetensorsFile(path) as f:
        tensors = {n: f.tensor(n).clone() for n in f.names()}
    g = torch.Generator().manual_seed(seed)
    for n, t in tensors.items():
        if n.endswith(".left.q.norm") or n.endswith(".left.k.norm"):
            tensors[n] = t * 2.0
        elif n.endswith(".left.temp"):
            tensors[n] = 0.5 + torch.rand(t.shape, generator=g)
        elif n == "embed":
            tensors[n] = t * 12.0
        elif n == "head":
            tensors[n] = t * 3.0
        elif n.endswith(".mix.z.b"):
            tensors[n] = 2.0 * torch.randn(t.shape, generator=g) - 1.0
        elif n.endswith(".b"):
            tensors[n] = 0.4 * torch.randn(t.shape, generator=g)
        elif n.endswith((".mlp.gate", ".mlp.up", ".mlp.down", ".mix.o", ".left.o", ".right.o", ".mix.x", ".mix.g", ".right.q", ".right.k")):
            tensors[n] = t * 2.5
    write_safetensors(path, tensors, metadata={"format": "pt"})
    (Path(out_dir) / "config.json").write_text(json.dumps(raw, indent=1))
    return Path(out_dir)


def load(model_dir):
    return plain_vononex.load_model_dir(model_dir)


def plain_logits(model_dir, requests, weights_as=None, dtype=torch.float64):
    raw, W = load(model_dir)
    if weights_as is not None:
        W = {k: (v.to(weights_as) if v.is_floating_point() else v) for k, v in W.items()}
    return {rid: plain_vononex.forward(raw, W, toks, dtype=dtype).double().numpy() for rid, toks in requests.items()}


def requests_for(raw, lens, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lens)}
