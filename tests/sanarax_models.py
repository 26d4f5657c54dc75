"""Small Sanarax models for the tests: configurations that differ in every size and option, random weights made sharp,
and the plain implementation's logits for a set of requests."""
from __future__ import annotations

import copy
import json
from pathlib import Path

import torch

from plain import plain_sanarax


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _attention(heads, kv_heads, dim, scale, base, dims, size, keep, mlp):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": {"base": base, "dims": dims},
        "mask": {"size": size, "keep_first": keep}}}


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, mlp):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
        "rot": {"base": base, "dims": rot_dim}}}


def _lightning(decay, dim, vdim, mlp):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def _again(layers, j):
    return {**copy.deepcopy(layers[j]), "weights_of": j}


def _config(vocab, width, eps, embedding, logit, layers):
    return {"architecture": "Sanarax", "vocab": vocab, "width": width, "embedding": {"scale": embedding}, "norm": {"eps": eps},
            "logit_scale": logit, "layers": layers}


def configs():
    """name -> (config.json as a dict, page size).  Between them: every layer kind first, last, alone and run again with the
    same weights; feed-forwards present and absent on each kind; grouped, ungrouped and single key heads; whole heads,
    parts of them and single pairs rotated; windows longer and shorter than a page, of one token, and longer than most
    prompts; no first tokens kept, a few, a page of them, more than the window holds; latents and head sizes that are no
    multiples of anything; recurrent heads from fast decay to none; scales at and away from one; eps small and large."""
    a = [_attention(4, 2, 16, 0.3, 500.0, 8, 24, 5, _dense(88)), _latent(3, 12, 4, 10, 20, 24, 0.25, 300.0, _dense(40)),
         _lightning([0.9, 0.999, 0.5], 12, 20, None)]
    a += [_again(a, 0), _attention(2, 2, 24, 0.21, 40.0, 24, 7, 0, None), _again(a, 2), _again(a, 1)]
    b = [_lightning([0.97], 24, 26, _dense(64)), _attention(6, 1, 8, 0.5, 2000.0, 4, 1, 33, _dense(200)),
         _latent(1, 16, 16, 8, 32, 16, 0.3, 50.0, None), _lightning([0.999, 0.3, 1.0, 0.6, 0.9], 8, 8, _dense(24))]
    b += [_again(b, 1), _again(b, 3)]
    c = [_latent(2, 7, 6, 5, 9, 11, 0.4, 90.0, _dense(33)), _attention(3, 3, 10, 0.45, 25.0, 2, 16, 16, None)]
    c += [_again(c, 0), _attention(5, 1, 14, 0.27, 700.0, 10, 90, 3, _dense(75)), _lightning([0.98, 0.6, 0.995], 11, 9, _dense(21))]
    return {"A": (_config(310, 72, 1e-6, 3.0, 0.7, a), 8), "B": (_config(259, 96, 2e-4, 1.0, 1.0, b), 4),
            "C": (_config(151, 50, 1e-5, 0.6, 2.5, c), 16)}


def medium_config():
    """A model of a few hundred columns whose prompts are long enough for the kernels of many rows: attention heads of 64
    and 128 on pages of 16 (the tcgen05 and TMA attention kernels), one size that only the mma.sync tiles take, kept first
    tokens inside one key tile, past one and next to the window; a latent of the tiles' sizes."""
    m = [_attention(4, 2, 64, 0.14, 10000.0, 32, 200, 37, _dense(448)), _latent(6, 32, 32, 40, 96, 64, 0.15, 5000.0, _dense(320)),
         _lightning([0.99, 0.9999, 0.7], 64, 48, None), _attention(6, 3, 128, 0.1, 700.0, 128, 150, 140, None),
         _attention(8, 2, 80, 0.12, 300.0, 40, 170, 9, _dense(192))]
    m += [_again(m, 1), _again(m, 0)]
    return _config(705, 320, 1e-6, 4.0, 1.5, m), 16


def write_model(raw, out_dir, seed):
    """Random weights for `raw`, then made sharp: queries and keys large (peaked attention), biases and sinks not small,
    gates spread from shut to open, norm weights spread around their one."""
    from inferflux_b200.config import config_from_dict
    from inferflux_b200.weights import SafetensorsFile, write_random_model, write_safetensors
    cfg = config_from_dict(raw)
    write_random_model(cfg, out_dir, seed=seed, dtype=torch.float32, std=0.08, norm_jitter=0.2)
    path = Path(out_dir) / "model.safetensors"
    with SafetensorsFile(path) as f:
        tensors = {n: f.tensor(n).clone() for n in f.names()}
    g = torch.Generator().manual_seed(seed)
    for n, t in tensors.items():
        if ".norm" in n or n == "final.norm":
            base = 1.0 if n.endswith((".dq.norm", ".dkv.norm", ".mix.norm")) else 0.0
            tensors[n] = base + 0.3 * torch.randn(t.shape, generator=g)
        elif n.endswith((".mix.q.b", ".mix.k.b")):
            tensors[n] = 0.5 * torch.randn(t.shape, generator=g)
        elif n.endswith(".mix.sink"):
            tensors[n] = 1.0 + torch.randn(t.shape, generator=g)
        elif n == "embed":
            tensors[n] = t * 6.0
        elif n == "head":
            tensors[n] = t * 4.0
        elif n.endswith((".mix.q", ".mix.k", ".mix.uq", ".mix.uk", ".mix.dkv", ".mix.g", ".mix.v", ".mlp.up")):
            tensors[n] = t * 2.5
    write_safetensors(path, tensors, metadata={"format": "pt"})
    (Path(out_dir) / "config.json").write_text(json.dumps(raw, indent=1))
    return Path(out_dir)


def load(model_dir):
    return plain_sanarax.load_model_dir(model_dir)


def plain_logits(model_dir, requests, weights_as=None, dtype=torch.float64):
    raw, W = load(model_dir)
    if weights_as is not None:
        W = {k: (v.to(weights_as) if v.is_floating_point() else v) for k, v in W.items()}
    return {rid: plain_sanarax.forward(raw, W, toks, dtype=dtype).double().numpy() for rid, toks in requests.items()}


def requests_for(raw, lens, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lens)}
