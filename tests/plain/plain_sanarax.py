"""The Sanarax decoder stated plainly: one function per mechanism, whole sequences at once, no cache, no
batching, nothing shared with the package.  Slow on purpose; the tests hold the engine to it.

A model is (raw, W): config.json as a dict and name -> tensor.  Every function computes in the dtype of
its inputs (the tests use float64).  In bfloat16, what the design keeps in 32 bits is float32 here too: the residual
stream, norms, rotations, scores and softmax, gates, the recurrence; such a run is the yardstick for what rounding the
rest does.

    x = scale * embed[tokens]
    per layer run:  x += n(mixer(n(x)));   x += n(ff(n(x)))   (ff may be absent; every n has a weight 1 + w of its own)
    logits = logit_scale * head . n(x)

A layer may run with another layer's weights; it then has its own history.  Mixer `attention`: grouped queries, values
that are the keys before rotation, a window beside which the first tokens stay visible, a learned unit in the softmax's
denominator, a gate per head.  Mixer `latent_attention`: queries through a normed latent, keys and values from another
one, one rotated key part for all heads, a gate per head.  Mixer `lightning`: a matrix of state per head with a fixed
decay, one norm over all heads, an elementwise gate.  Feed-forward: two products with a squared ReLU between them.
"""
from __future__ import annotations

import math

import torch

from .plain_vononex import load_model_dir            # noqa: F401  (reads config.json and model.safetensors, nothing else)


# ------------------------------------------------------------------------------ small pieces

def wide(x):
    """Float32 for bfloat16, anything else as it is."""
    return x.to(torch.float32) if x.dtype == torch.bfloat16 else x


def unit_rms(x, eps):
    """x divided by its root mean square over the last axis, eps under the root."""
    x = wide(x)
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x, w, eps):
    """The model's norm: the stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + wide(w))


def silu(z):
    return z * torch.sigmoid(z)


def squared_relu(z):
    return torch.clamp(z, min=0.0) ** 2


def gate_heads(o, logits):
    """o: [n, H, dv] heads' outputs, logits: [n, H]."""
    return (wide(o) * torch.sigmoid(wide(logits))[:, :, None]).to(logits.dtype)


# ------------------------------------------------------------------------------ positions

def _angles(positions, dims, base, dtype):
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.tensor(list(positions), dtype=torch.float64)[:, None] * f[None, :]
    return torch.cos(a).to(dtype)[:, None, :], torch.sin(a).to(dtype)[:, None, :]


def rotate_halves(x, positions, dims, base):
    """x: [n, H, d]; elements i and i + dims/2 of the first `dims` turn by position * base^(-2i/dims)."""
    dtype, x = x.dtype, wide(x)
    c, s = _angles(positions, dims, base, x.dtype)
    u, v = x[:, :, :dims // 2], x[:, :, dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[:, :, dims:]], dim=-1).to(dtype)


def rotate_neighbours(x, positions, dims, base):
    """The same for elements 2i and 2i + 1."""
    dtype, x = x.dtype, wide(x)
    c, s = _angles(positions, dims, base, x.dtype)
    out = x.clone()
    u, v = x[:, :, 0:dims:2], x[:, :, 1:dims:2]
    out[:, :, 0:dims:2] = u * c - v * s
    out[:, :, 1:dims:2] = v * c + u * s
    return out.to(dtype)


# ------------------------------------------------------------------------------ masks and softmax

def visible(n, size=None, keep_first=0):
    """[n, n] bool: row i sees column j.  Not later than itself; with `size`, also less than that far back or among the
    first `keep_first`."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def softmax_rows(s, seen, sink=None):
    """Weights over the visible columns of every row; `sink`: a score that joins the denominator alone."""
    s = s.masked_fill(~seen, -math.inf)
    m = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink.reshape(1, 1))
    e = torch.exp(s - m)
    total = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink.reshape(1, 1) - m)
    return e / total


# ------------------------------------------------------------------------------ attention

def attend(q, k, v, scale, seen, sinks):
    """q: [n, H, d], k: [n, G, d], v: [n, G, dv]; query head h reads key head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (wide(q[:, h]) @ wide(k[:, g]).T) * scale
        w = softmax_rows(s, seen, None if sinks is None else wide(sinks[h]))
        out.append((w.to(q.dtype) @ v[:, g]))
    return torch.stack(out, dim=1)


def attention(h, W, p, m, positions):
    n = h.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(n, H, d)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(n, G, d)
    v = k                                                                    # before the rotation
    q, k = rotate_halves(q, positions, dims, base), rotate_halves(k, positions, dims, base)
    seen = visible(n, int(m["mask"]["size"]), int(m["mask"]["keep_first"]))
    o = attend(q, k, v, float(m["scale"]), seen, W[p + "sink"])
    return gate_heads(o, h @ W[p + "g"].T).reshape(n, H * d) @ W[p + "o"].T


# ------------------------------------------------------------------------------ latent attention

def latent_attention(h, W, p, m, eps, positions):
    n = h.shape[0]
    H, d, dr, dv, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    base = float(m["rot"]["base"])
    cq = (unit_rms(h @ W[p + "dq"].T, eps) * wide(W[p + "dq.norm"])).to(h.dtype)
    q = (cq @ W[p + "uq"].T).reshape(n, H, d + dr)
    down = h @ W[p + "dkv"].T
    c = (unit_rms(down[:, :r], eps) * wide(W[p + "dkv.norm"])).to(h.dtype)
    k = (c @ W[p + "uk"].T).reshape(n, H, d)
    v = (c @ W[p + "uv"].T).reshape(n, H, dv)
    kr = rotate_neighbours(down[:, r:].reshape(n, 1, dr), positions, dr, base)
    qr = rotate_neighbours(q[:, :, d:], positions, dr, base)
    q = torch.cat([q[:, :, :d], qr], dim=-1)
    k = torch.cat([k, kr.expand(n, H, dr)], dim=-1)
    o = attend(q, k, v, float(m["scale"]), visible(n), None)
    return gate_heads(o, h @ W[p + "g"].T).reshape(n, H * dv) @ W[p + "o"].T


# ------------------------------------------------------------------------------ lightning attention

def decay_scan(q, k, v, decay):
    """q, k: [n, H, d]; v: [n, H, dv]; decay: [H].  S <- decay S + k_t v_t^T; o_t = S^T q_t with the new S."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def lightning(h, W, p, m, eps):
    n = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k = (silu(wide(h @ W[p + s].T)).reshape(n, H, d) for s in ("q", "k"))
    v = silu(wide(h @ W[p + "v"].T)).reshape(n, H, dv)
    o = decay_scan(q, k, v, torch.tensor([float(x) for x in m["decay"]], dtype=q.dtype)).reshape(n, H * dv)
    o = unit_rms(o, eps) * wide(W[p + "norm"])
    return (o * torch.sigmoid(wide(h @ W[p + "g"].T))).to(h.dtype) @ W[p + "o"].T


# ------------------------------------------------------------------------------ the layer

def mixer(h, W, p, layer, eps, positions):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return attention(h, W, p, m, positions)
    if layer["type"] == "latent_attention":
        return latent_attention(h, W, p, m, eps, positions)
    if layer["type"] == "lightning":
        return lightning(h, W, p, m, eps)
    raise ValueError(layer["type"])


def feed_forward(h, W, p):
    return squared_relu(h @ W[p + "up"].T) @ W[p + "down"].T


# ------------------------------------------------------------------------------ the model

def forward(raw, W, tokens, dtype=torch.float64, streams=None):
    """Logits [n, vocab] of one sequence.  `streams`: a list that receives the residual stream after every layer run."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in W.items()}
    eps = float(raw["norm"]["eps"])
    positions = list(range(len(tokens)))
    x = wide(W["embed"][list(tokens)]) * float(raw["embedding"]["scale"])
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i if layer.get('weights_of') is None else layer['weights_of']}."
        y = mixer(norm(x, W[p + "norm1"], eps).to(dtype), W, p + "mix.", layer, eps, positions)
        x = x + norm(y, W[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(norm(x, W[p + "norm2"], eps).to(dtype), W, p + "mlp.")
            x = x + norm(y, W[p + "norm2b"], eps)
        if streams is not None:
            streams.append(x.clone())
    return float(raw["logit_scale"]) * wide(norm(x, W["final.norm"], eps).to(dtype) @ W["head"].T)
