"""A plain, slow implementation of the Lulisun decoder in float64: the oracle of the Lulisun tests.

One function per mechanism, written from the formulas.  It reads a model folder with its own safetensors reader
and shares no code with `liteinfer_b200`.  A whole sequence goes in, logits of every position come out; there is
no cache, no batch and no cut.
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np
import torch

F = torch.float64


def read_model(model_dir):
    """(config.json as a dict, {tensor name: float64 tensor})."""
    model_dir = Path(model_dir)
    config = json.loads((model_dir / "config.json").read_text())
    blob = (model_dir / "model.safetensors").read_bytes()
    (header_len,) = struct.unpack("<Q", blob[:8])
    data = blob[8 + header_len:]
    tensors = {}
    for name, meta in json.loads(blob[8:8 + header_len]).items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = np.frombuffer(data[lo:hi], dtype=np.uint8)
        if meta["dtype"] == "BF16":
            value = torch.from_numpy((raw.view(np.uint16).astype(np.uint32) << 16).view(np.float32).copy())
        elif meta["dtype"] == "F32":
            value = torch.from_numpy(raw.view(np.float32).copy())
        else:
            raise ValueError(f"{name}: dtype {meta['dtype']}")
        tensors[name] = value.to(F).reshape(meta["shape"])
    return config, tensors


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """A root-mean-square norm whose stored weight lies around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def rotate(x, dims, base):
    """x [T, heads, n]: dimensions i and i + dims / 2 of every head turn by position * base^(-2 i / dims)."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=F)
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + dims // 2]
        out[:, :, i] = u * c - v * s
        out[:, :, i + dims // 2] = v * c + u * s
    return out


def chunk_start(position, size):
    """The first position that `position` reads: the start of its chunk (None: of the sequence)."""
    return 0 if size is None else (position // size) * size


def chunked_attention(q, k, v, scale, size):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: position i reads the keys of its own chunk up to itself;
    query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            lo = chunk_start(i, size)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[lo:i + 1, g]
    return out


def left_mixer(h, w, p, mixer):
    """Grouped-query attention within chunks, half-split rotation of the first dimensions."""
    T = h.shape[0]
    H, G, D, V = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D)
    k = (h @ w[p + "k"].T).view(T, G, D)
    v = (h @ w[p + "v"].T).view(T, G, V)
    if mixer.get("rot"):
        q, k = (rotate(x, mixer["rot"]["dims"], float(mixer["rot"]["base"])) for x in (q, k))
    size = mixer["mask"]["size"] if mixer.get("mask") else None
    return chunked_attention(q, k, v, mixer["scale"], size).reshape(T, H * V) @ w[p + "o"].T


def forget_memory(q, f, v):
    """q, f [T, H, D], v [T, H, V] -> [T, H, V]: per head a matrix S [D, V] from zero; row d keeps f[d] of itself and
    takes (1 - f[d]) of the token's value; the read-out is S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def forget_gate(z, lower):
    """The forget gate: between its lower bound and 1."""
    return lower + (1.0 - lower) * sigmoid(z)


def right_mixer(h, w, p, mixer, eps):
    T = h.shape[0]
    H, D, V = mixer["heads"], mixer["dim"], mixer["vdim"]
    q = silu(h @ w[p + "q"].T).view(T, H, D)
    f = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    o = unit_rms(forget_memory(q, f, v), eps) * w[p + "norm"]
    return o.reshape(T, H * V) @ w[p + "o"].T


def both_mixers(h, w, p, mixer, eps):
    return (mixer["left_scale"] * left_mixer(h, w, p + "left.", mixer["left"])
            + mixer["right_scale"] * right_mixer(h, w, p + "right.", mixer["right"], eps))


def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route_scores(scores, correction, router):
    """scores [T, E] -> (chosen experts [T, top], their weights [T, top]).  Choice: scores + correction, within the
    groups of neighbours whose two best choice scores sum highest.  Weights: the scores, divided by their sum."""
    T, E = scores.shape
    choice = scores + correction
    groups = router.get("groups")
    if groups:
        per = E // groups["count"]
        masked = torch.full_like(choice, -math.inf)
        for t in range(T):
            ranks = []
            for g in range(groups["count"]):
                best = sorted(choice[t, g * per:(g + 1) * per].tolist(), reverse=True)
                ranks.append((-sum(best[:2]), g))
            for _, g in sorted(ranks)[:groups["keep"]]:
                masked[t, g * per:(g + 1) * per] = choice[t, g * per:(g + 1) * per]
        choice = masked
    chosen = torch.argsort(-choice, dim=-1, stable=True)[:, :router["top"]]
    picked = scores.gather(1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20)


def moe_ff(h, w, p, mlp):
    chosen, weights = route_scores(sigmoid(h @ w[p + "router"].T), w[p + "correction"], mlp["router"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        at, slot = torch.nonzero(chosen == e, as_tuple=True)
        if len(at):
            out[at] += weights[at, slot][:, None] * dense_ff(h[at], w, f"{p}e{e}.")
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * dense_ff(h, w, p + "shared.")
    return out


def forward(config, w, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence.  `trace`: a list that receives the stream after every layer."""
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        j = i
        while config["layers"][j].get("weights_of") is not None:
            j = config["layers"][j]["weights_of"]
        p = f"l{j}."
        y = both_mixers(offset_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + moe_ff(offset_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return offset_norm(x, w["final.norm"], eps) @ w["head"].T
