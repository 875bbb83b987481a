"""A plain, slow implementation of the Zebovik decoder: one function per mechanism, 64-bit, whole sequences, no cache.

It shares no code with the library: tensors come as a ``{name: tensor}`` mapping, sizes and constants from the nested
configuration (a dict shaped like config.json). Every function works on ONE sequence given from its first token on;
the recurrences are loops over the tokens, attention is a loop over the queries, each reduced over its visible keys.

Notation: ``h`` is a mixer's or feed-forward's input ``[T, width]``; linear weights are ``[out, in]``; ``p`` is the
prefix of the tensors' names.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Mapping, Optional

import torch

F64 = torch.float64


def load_model(model_dir: str):
    """(the JSON object of config.json, {name: tensor}) of a model folder"""
    from safetensors.torch import load_file
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, load_file(os.path.join(model_dir, "model.safetensors"))


def _w(t: Mapping[str, torch.Tensor], name: str) -> torch.Tensor:
    return t[name].to(F64)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x: float) -> float:
    return max(x, 0.0) + math.log1p(math.exp(-abs(x)))


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis"""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(x / cap)


# ----------------------------------------------------------------------------------------------- matrix memory
def mlstm_gates(zi: List[float], zf: List[float], cap: float):
    """the log input gates, the log forget gates and the running maxima of one head, from the gates' projections"""
    i = [cap * math.tanh(z / cap) for z in zi]
    f = [-softplus(-cap * math.tanh(z / cap)) for z in zf]
    m, ms = 0.0, []
    for t in range(len(i)):
        m = max(f[t] + m, i[t])
        ms.append(m)
    return i, f, ms


def mlstm_head(q, k, v, i, f) -> torch.Tensor:
    """one head's matrix memory: q, k [T, d], v [T, dv]; i, f: log gates. Row t is S^T q / max(|n . q|, e^-m)"""
    T, d = q.shape
    S = torch.zeros((d, v.shape[1]), dtype=F64)
    n = torch.zeros(d, dtype=F64)
    m = 0.0
    out = torch.zeros((T, v.shape[1]), dtype=F64)
    for t in range(T):
        new = max(f[t] + m, i[t])
        keep, write = math.exp(f[t] + m - new), math.exp(i[t] - new)
        S = keep * S + write * torch.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm(t, p: str, c: Mapping, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, d, dv, cap = int(c["heads"]), int(c["dim"]), int(c["vdim"]), float(c["gate_cap"])
    T = h.shape[0]
    q = (h @ _w(t, p + "q").T).view(T, H, d) * d ** -0.5
    k = (h @ _w(t, p + "k").T).view(T, H, d)
    v = (h @ _w(t, p + "v").T).view(T, H, dv)
    zi = h @ _w(t, p + "i").T + _w(t, p + "i.b")
    zf = h @ _w(t, p + "f").T + _w(t, p + "f.b")
    heads = []
    for a in range(H):
        i, f, _ = mlstm_gates(zi[:, a].tolist(), zf[:, a].tolist(), cap)
        heads.append(rms(mlstm_head(q[:, a], k[:, a], v[:, a], i, f), eps))
    o = torch.cat(heads, dim=1) * _w(t, p + "norm")
    return (o * sigmoid(h @ _w(t, p + "g").T)) @ _w(t, p + "o").T


# ----------------------------------------------------------------------------------------------- state-space duality
def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x [T, C], w [C, taps]: y[t] = b + sum_j w[:, j] x[t - (taps - 1) + j], zeros before the start"""
    T, taps = x.shape[0], w.shape[1]
    y = b.expand(T, -1).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * x[:T - back]
    return y


def ssd_head(x, B, C, dt, a_log: float, D: float) -> torch.Tensor:
    """one head: x [T, dv], B, C [T, N], dt: step sizes. S_t = exp(-e^a_log dt) S_(t-1) + dt B x^T; y = S^T C + D x"""
    T = x.shape[0]
    S = torch.zeros((B.shape[1], x.shape[1]), dtype=F64)
    out = torch.zeros_like(x)
    for t in range(T):
        S = math.exp(-math.exp(a_log) * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        out[t] = S.T @ C[t] + D * x[t]
    return out


def mamba2(t, p: str, c: Mapping, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, dv, N, G = int(c["heads"]), int(c["vdim"]), int(c["state"]), int(c["groups"])
    parts = int(c["norm_groups"])
    T, inner = h.shape[0], H * dv
    row = h @ _w(t, p + "in").T
    z, xbc, zdt = row[:, :inner], row[:, inner:2 * inner + 2 * G * N], row[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, _w(t, p + "conv"), _w(t, p + "conv.b")))
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    bias, a_log, D = (_w(t, p + n).tolist() for n in ("dt_bias", "A_log", "D"))
    heads = []
    for a in range(H):
        g = a // (H // G)
        dt = [softplus(float(u) + bias[a]) for u in zdt[:, a]]
        heads.append(ssd_head(x[:, a], B[:, g], C[:, g], dt, a_log[a], D[a]))
    y = torch.cat(heads, dim=1) * silu(z)
    y = rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * _w(t, p + "norm")
    return y @ _w(t, p + "o").T


# ----------------------------------------------------------------------------------------------- attention
def rotate_half(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, n, d]: the pair (i, i + dims / 2) at position p turns by p base^(-2i / dims); the rest passes"""
    T = x.shape[0]
    out = x.clone()
    pos = torch.arange(T, dtype=F64)
    for i in range(dims // 2):
        a = pos * (base ** (-2.0 * i / dims))
        c, s = torch.cos(a).view(T, 1), torch.sin(a).view(T, 1)
        u, w = x[:, :, i], x[:, :, i + dims // 2]
        out[:, :, i] = u * c - w * s
        out[:, :, i + dims // 2] = w * c + u * s
    return out


def chunk_start(i: int, size: Optional[int]) -> int:
    """the first position that position i sees"""
    return 0 if not size else i // size * size


def capped_attention(q, k, v, scale: float, cap: Optional[float], size: Optional[int]) -> torch.Tensor:
    """one head: q, k [T, d], v [T, dv]; scores capped, keys of the query's chunk, one added to the denominator"""
    T = q.shape[0]
    out = torch.zeros((T, v.shape[1]), dtype=F64)
    for i in range(T):
        lo = chunk_start(i, size)
        s = (k[lo:i + 1] @ q[i]) * scale
        if cap:
            s = softcap(s, cap)
        m = max(float(s.max()), 0.0)
        e = torch.exp(s - m)
        out[i] = (e / (math.exp(-m) + e.sum())) @ v[lo:i + 1]
    return out


def attention_kv(t, p: str, c: Mapping, h: torch.Tensor, eps: float):
    """keys [T, G, d] after rotation and norm, values [T, G, dv]"""
    G, d, dv = int(c["kv_heads"]), int(c["dim"]), int(c["vdim"])
    T = h.shape[0]
    k = (h @ _w(t, p + "k").T + _w(t, p + "k.b")).view(T, G, d)
    v = (h @ _w(t, p + "v").T + _w(t, p + "v.b")).view(T, G, dv)
    return rms(rotate_half(k, float(c["rot"]["base"]), int(c["rot"]["dims"])), eps), v


def attention(t, p: str, c: Mapping, h: torch.Tensor, eps: float, k, v) -> torch.Tensor:
    H, G, d = int(c["heads"]), int(c["kv_heads"]), int(c["dim"])
    T = h.shape[0]
    q = (h @ _w(t, p + "q").T + _w(t, p + "q.b")).view(T, H, d)
    q = rms(rotate_half(q, float(c["rot"]["base"]), int(c["rot"]["dims"])), eps)
    size = None if c.get("mask") is None else int(c["mask"]["size"])
    heads = [capped_attention(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], float(c["scale"]), c.get("softcap"),
                              size) for a in range(H)]
    return torch.cat(heads, dim=1) @ _w(t, p + "o").T


# ----------------------------------------------------------------------------------------------- feed-forward, model
def feed_forward(t, p: str, h: torch.Tensor) -> torch.Tensor:
    u = torch.clamp(h @ _w(t, p + "up").T + _w(t, p + "up.b"), min=0.0)
    return (u * u) @ _w(t, p + "down").T + _w(t, p + "down.b")


def layers(cfg: Mapping, t: Mapping[str, torch.Tensor], tokens: List[int]):
    """the residual stream after every layer: a list of [T, width]"""
    eps = float(cfg["norm"]["eps"])
    x = _w(t, "embed")[torch.tensor(tokens, dtype=torch.long)]
    kept: Dict[int, tuple] = {}
    out = []
    for i, layer in enumerate(cfg["layers"]):
        p, c = "l%d." % i, layer["mixer"]
        h = rms(x, eps) * _w(t, p + "norm1")
        if layer["type"] == "mlstm":
            y = mlstm(t, p + "mix.", c, h, eps)
        elif layer["type"] == "mamba2":
            y = mamba2(t, p + "mix.", c, h, eps)
        else:
            if c.get("kv_from") is None:
                kept[i] = attention_kv(t, p + "mix.", c, h, eps)
            y = attention(t, p + "mix.", c, h, eps, *kept[i if c.get("kv_from") is None else int(c["kv_from"])])
        x = x + rms(y, eps) * _w(t, p + "norm1b")
        if layer.get("mlp") is not None:
            h = rms(x, eps) * _w(t, p + "norm2")
            x = x + rms(feed_forward(t, p + "mlp.", h), eps) * _w(t, p + "norm2b")
        out.append(x)
    return out


def logits(cfg: Mapping, t: Mapping[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """[T, vocab] of one sequence"""
    y = rms(layers(cfg, t, tokens)[-1], float(cfg["norm"]["eps"])) * _w(t, "final.norm")
    z = y @ _w(t, "head").T
    return softcap(z, float(cfg["logit_softcap"])) if cfg.get("logit_softcap") else z
