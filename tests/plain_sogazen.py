"""A plain, slow implementation of the Sogazen decoder in float64: the oracle of the Sogazen tests.

One function per mechanism, written from the formulas.  It reads a model folder with its own safetensors reader
and shares no code with `liteinfer_b200`.  A whole sequence goes in, logits of every position come out; there is
no cache, no batch and no cut.
"""

from __future__ import annotations

import json
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


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def cap(x, limit):
    return limit * torch.tanh(x / limit) if limit else x


# ------------------------------------------------------------------ attention
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


def quiet_attention(q, k, v, scale, softcap):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: causal, scores capped, and one more than the exponentials in
    the denominator, so that a query none of whose keys score much reads next to nothing."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            s = cap((k[:i + 1, g] @ q[i, h]) * scale, softcap)
            top = max(float(s.max()), 0.0)
            e = torch.exp(s - top)
            out[i, h] = (e @ v[:i + 1, g]) / (np.exp(-top) + e.sum())
    return out


def left_mixer(h, w, p, mixer, eps):
    """Grouped-query attention whose values are its unnormalised, unrotated keys."""
    T = h.shape[0]
    H, G, D = mixer["heads"], mixer["kv_heads"], mixer["dim"]
    q, k = (h @ w[p + n].T + w[p + n + ".b"] for n in "qk")
    v = k.view(T, G, D)
    q, k = (unit_rms(x, eps) * w[p + n + ".norm"] for x, n in ((q, "q"), (k, "k")))
    q, k = q.view(T, H, D), k.view(T, G, D)
    if mixer.get("rot"):
        q, k = (rotate(x, mixer["rot"]["dims"], float(mixer["rot"]["base"])) for x in (q, k))
    return quiet_attention(q, k, v, mixer["scale"], mixer.get("softcap")).reshape(T, H * D) @ w[p + "o"].T


# ------------------------------------------------------------------ the state space
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K]: per channel, the last tap on the token itself, zeros before the first."""
    T, K = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=F), x])
    return sum(padded[j:j + T] * taps[:, j] for j in range(K)) + bias


def state_space(x, b, c, dt, a_log, skip):
    """x [T, H, V], b, c [T, G, N], dt [T, H], a_log, skip [H] -> [T, H, V]: per head a matrix S [N, V] from zero, kept
    by exp(-exp(a_log) dt) and given dt b x^T; read as S^T c, plus skip x."""
    T, H, V = x.shape
    G, N = b.shape[1:]
    out = torch.zeros(T, H, V, dtype=F)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(N, V, dtype=F)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * torch.outer(b[t, g], x[t, h])
            out[t, h] = S.T @ c[t, g] + skip[h] * x[t, h]
    return out


def gated_group_norm(y, z, weight, groups, eps):
    """The gate silu(z) first, then each of `groups` equal parts by its own root mean square."""
    y = y * silu(z)
    return unit_rms(y.unflatten(1, (groups, -1)), eps).flatten(1) * weight


def right_mixer(h, w, p, mixer, eps):
    T = h.shape[0]
    H, V, N, G = mixer["heads"], mixer["vdim"], mixer["state"], mixer["groups"]
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [H * V, H * V + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, b, c = torch.split(xbc, [H * V, G * N, G * N], dim=1)
    y = state_space(x.reshape(T, H, V), b.reshape(T, G, N), c.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]),
                    w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, H * V), z, w[p + "norm"], mixer["norm_groups"], eps) @ w[p + "o"].T


def both_mixers(h, w, p, mixer, eps):
    """The mean of the two, each normalised over the width by a weight of its own."""
    left = unit_rms(left_mixer(h, w, p + "left.", mixer["left"], eps), eps) * w[p + "left.out"]
    right = unit_rms(right_mixer(h, w, p + "right.", mixer["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


# ------------------------------------------------------------------ the time mixer
def token_shift(h, mu):
    """Every token's own mix of itself and the token before it (zeros before the first)."""
    before = torch.cat([torch.zeros(1, h.shape[1], dtype=F), h[:-1]])
    return h + (before - h) * mu


def bonus_memory(r, k, v, decay, u):
    """r, k, decay [T, H, D], v [T, H, D], u [H, D] -> [T, H, D]: per head a matrix S [D, D] from zero; a token reads what
    the tokens before it left, plus u-weighted what it brings itself; then the rows decay and take k v^T."""
    T, H, D = r.shape
    out = torch.zeros(T, H, D, dtype=F)
    for h in range(H):
        S = torch.zeros(D, D, dtype=F)
        for t in range(T):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S + u[h][:, None] * kv).T @ r[t, h]
            S = decay[t, h][:, None] * S + kv
    return out


def time_mixer(h, w, p, mixer, eps):
    T = h.shape[0]
    H, D = mixer["heads"], mixer["dim"]
    mix = {n: token_shift(h, w[p + "mu." + n]) for n in "rkvgw"}
    r, k, v, g = (mix[n] @ w[p + n].T for n in "rkvg")
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))
    o = bonus_memory(*(x.view(T, H, D) for x in (r, k, v, decay)), w[p + "u"])
    return (unit_rms(o, eps).reshape(T, H * D) * w[p + "norm"] * silu(g)) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward
def capped_gate(gate, up, limit):
    gate, up = torch.clamp(gate, max=limit), torch.clamp(up, -limit, limit)
    return gate * sigmoid(1.702 * gate) * (up + 1.0)


def dense_ff(h, w, p, mlp):
    return capped_gate(h @ w[p + "gate"].T, h @ w[p + "up"].T, mlp["limit"]) @ w[p + "down"].T


def route(logits, correction, top):
    """(chosen outputs [T, top], their weights): softmax scores; the choice goes by score + correction, the weight is the
    score."""
    scores = torch.softmax(logits, dim=-1)
    chosen = torch.argsort(-(scores + correction), dim=-1, stable=True)[:, :top]
    return chosen, scores.gather(1, chosen)


def moe_ff(h, w, p, mlp):
    experts = mlp["router"]["experts"]
    chosen, weights = route(h @ w[p + "router"].T, w[p + "correction"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(w[p + "router"].shape[0]):
        at, slot = torch.nonzero(chosen == e, as_tuple=True)
        if len(at):
            y = h[at] if e >= experts else torch.relu(h[at] @ w[f"{p}e{e}.up"].T).pow(2) @ w[f"{p}e{e}.down"].T
            out[at] += weights[at, slot][:, None] * y
    return out


def forward(config, w, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence.  `trace`: a list that receives the stream after every layer."""
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        mixer = both_mixers if layer["type"] == "parallel" else time_mixer
        x = x + unit_rms(mixer(x, w, p + "mix.", layer["mixer"], eps), eps) * w[p + "norm1"]
        if layer.get("mlp") is not None:
            ff = dense_ff if layer["mlp"]["kind"] == "dense" else moe_ff
            x = x + unit_rms(ff(x, w, p + "mlp.", layer["mlp"]), eps) * w[p + "norm2"]
        if trace is not None:
            trace.append(x.clone())
    return cap((unit_rms(x, eps) * w["final.norm"]) @ w["head"].T, config.get("logit_softcap"))
