"""The Vononex decoder stated plainly: one function per mechanism, whole sequences at once, no cache, no
batching, nothing shared with the package.  Slow on purpose; the tests hold the engine to it.

A model is (raw, W): config.json as a dict and name -> tensor.  Every function computes in the dtype of
its inputs (the tests use float64).

    x = embed[tokens]
    per layer:  x = rms_norm(alpha x + mixer(x)) * norm1;   x = rms_norm(alpha x + ff(x)) * norm2   (ff may be absent)
    logits = head . (rms_norm(x) * final.norm)

Mixer `parallel`: left_scale * left(x) + right_scale * right(x).  The left one is causal attention with biases,
queries and keys normed over their whole rows and then turned, a factor per head on the scores, and values turned by
their own position whose weighted sum is turned back by the query's.  The right one is a retention: a matrix of state
per head with a fixed decay.  Mixer `mingru`: a gated recurrence, element by element, whose gates read the present
token only.  Feed-forward: a gated product with the tanh form of gelu and biases.
"""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch


# ------------------------------------------------------------------------------ small pieces

def unit_rms(x, eps):
    """x divided by its root mean square over the last axis, eps under the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sum_norm(x, y, alpha, w, eps):
    """The norm behind a sublayer: of alpha times its input plus its output."""
    return unit_rms(alpha * x + y, eps) * w


# ------------------------------------------------------------------------------ positions

def rotate_halves(x, positions, dims, base, direction=1.0):
    """x: [n, H, d]; elements i and i + dims/2 of the first `dims` turn by direction * position * base^(-2i/dims)."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = direction * torch.tensor(list(positions), dtype=torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[:, :, :half], x[:, :, half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[:, :, dims:]], dim=-1)


# ------------------------------------------------------------------------------ attention

def attend(q, k, v, scale, temp):
    """q: [n, H, d], k: [n, G, d], v: [n, G, dv]: softmax over every key up to the query's own position, the scores
    multiplied by scale and by the head's temp."""
    n, H = q.shape[0], q.shape[1]
    per = H // k.shape[1]
    seen = torch.tril(torch.ones(n, n, dtype=torch.bool))
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale * temp[h]
        s = s.masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out.append((e / e.sum(dim=-1, keepdim=True)) @ v[:, h // per])
    return torch.stack(out, dim=1)


def attention(h, W, p, m, eps, positions):
    n = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    q, k, v = (h @ W[p + s].T + W[p + s + ".b"] for s in ("q", "k", "v"))
    q = (unit_rms(q, eps) * W[p + "q.norm"]).reshape(n, H, d)              # the mean runs over all heads' elements
    k = (unit_rms(k, eps) * W[p + "k.norm"]).reshape(n, G, d)
    q, k = rotate_halves(q, positions, dims, base), rotate_halves(k, positions, dims, base)
    v = rotate_halves(v.reshape(n, G, dv), positions, dv, base)
    o = attend(q, k, v, float(m["scale"]), W[p + "temp"])
    o = rotate_halves(o, positions, dv, base, direction=-1.0)
    return o.reshape(n, H * dv) @ W[p + "o"].T + W[p + "o.b"]


# ------------------------------------------------------------------------------ retention

def retention_scan(q, k, v, decay):
    """q, k: [n, H, d]; v: [n, H, dv]; decay: [H].  S <- decay S + k_t v_t^T; o_t = S^T q_t with the new S."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def retention(h, W, p, m, eps, positions):
    n = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    q = rotate_halves((h @ W[p + "q"].T).reshape(n, H, d), positions, dims, base)
    k = rotate_halves((h @ W[p + "k"].T).reshape(n, H, d), positions, dims, base) * d ** -0.5
    v = (h @ W[p + "v"].T).reshape(n, H, dv)
    o = retention_scan(q, k, v, torch.tensor([float(x) for x in m["decay"]], dtype=h.dtype))
    o = unit_rms(o, eps).reshape(n, H * dv)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------ minGRU

def gated_scan(z, candidate):
    """[n, width] each: S_t = (1 - z_t) S_(t-1) + z_t candidate_t, from zero."""
    S = torch.zeros(z.shape[1], dtype=z.dtype)
    out = []
    for t in range(z.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * candidate[t]
        out.append(S)
    return torch.stack(out)


def mingru(h, W, p):
    z = torch.sigmoid(h @ W[p + "z"].T + W[p + "z.b"])
    u = h @ W[p + "x"].T + W[p + "x.b"]
    candidate = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    return (gated_scan(z, candidate) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------ the layer

def mixer(h, W, p, layer, eps, positions):
    m = layer["mixer"]
    if layer["type"] == "parallel":
        return (float(m["left_scale"]) * attention(h, W, p + "left.", m["left"], eps, positions)
                + float(m["right_scale"]) * retention(h, W, p + "right.", m["right"], eps, positions))
    if layer["type"] == "mingru":
        return mingru(h, W, p)
    raise ValueError(layer["type"])


def feed_forward(h, W, p):
    a = gelu_tanh(h @ W[p + "gate"].T + W[p + "gate.b"]) * (h @ W[p + "up"].T + W[p + "up.b"])
    return a @ W[p + "down"].T + W[p + "down.b"]


# ------------------------------------------------------------------------------ the model

def forward(raw, W, tokens, dtype=torch.float64, streams=None):
    """Logits [n, vocab] of one sequence.  `streams`: a list that receives the residual stream after every layer."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in W.items()}
    eps, alpha = float(raw["norm"]["eps"]), float(raw["postln_alpha"])
    positions = list(range(len(tokens)))
    x = W["embed"][list(tokens)]
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i}."
        x = sum_norm(x, mixer(x, W, p + "mix.", layer, eps, positions), alpha, W[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = sum_norm(x, feed_forward(x, W, p + "mlp."), alpha, W[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.clone())
    return (unit_rms(x, eps) * W["final.norm"]) @ W["head"].T


def load_model_dir(model_dir):
    """(config.json as a dict, name -> tensor) of a model folder, read without the package."""
    import numpy as np
    model_dir = Path(model_dir)
    raw = json.loads((model_dir / "config.json").read_text())
    blob = (model_dir / "model.safetensors").read_bytes()
    n = int.from_bytes(blob[:8], "little")
    header = json.loads(blob[8:8 + n])
    W = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        data = blob[8 + n + lo:8 + n + hi]
        if info["dtype"] == "BF16":
            u = np.frombuffer(data, dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(u.view(np.float32).copy())
        elif info["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(data, dtype="<f4").copy())
        elif info["dtype"] == "F64":
            t = torch.from_numpy(np.frombuffer(data, dtype="<f8").copy())
        elif info["dtype"] == "I32":
            t = torch.from_numpy(np.frombuffer(data, dtype="<i4").copy())
        else:
            raise ValueError(f"{name}: dtype {info['dtype']}")
        W[name] = t.reshape(info["shape"])
    return raw, W
