"""A plain, slow implementation of the Basitar decoder: one function per mechanism, 64-bit, whole sequences, no cache.

It shares no code with the library: tensors come as a ``{name: tensor}`` mapping, sizes and constants from the nested
configuration (a dict shaped like config.json). Every function works on ONE sequence given from its first token on; the
recurrence is a loop over the tokens, attention a loop over the queries, each reduced over its visible keys, with keys and
values expanded from the latents.

Notation: ``h`` is a mixer's or feed-forward's input ``[T, width]``; linear weights are ``[out, in]``; ``p`` is the
prefix of the tensors' names.
"""
from __future__ import annotations

import json
import math
import os
from typing import List, Mapping, Optional

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


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis"""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """the layers' norm: the gain is one more than the stored weight"""
    return rms(x, eps) * (1.0 + w)


# ----------------------------------------------------------------------------------------------- embedding
def bigram_rows(tokens: List[int], buckets: int, mul_prev: int, mul_cur: int) -> List[int]:
    """the row of the pair table for every token; the first token has no predecessor and takes the last row"""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + tokens[i] * mul_cur) % buckets for i in range(len(tokens))]


def embedding(cfg: Mapping, t, tokens: List[int]) -> torch.Tensor:
    b = cfg["embedding"]["bigram"]
    x = _w(t, "embed")[torch.tensor(tokens, dtype=torch.long)]
    rows = bigram_rows(tokens, int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]))
    x = x + _w(t, "bigram")[torch.tensor(rows, dtype=torch.long)]
    return x + _w(t, "pos")[:len(tokens)]


# ----------------------------------------------------------------------------------------------- time mixing
def shifted(h: torch.Tensor) -> torch.Tensor:
    """the row before, zeros for the first"""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)


def token_mix(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    return h + (shifted(h) - h) * mu


def wkv_head(r, k, v, w, u) -> torch.Tensor:
    """one head: r, k, w [T, d], v [T, dv], u [d]. Row t reads the state before it and, with the bonus u, its own token"""
    T, d = k.shape
    S = torch.zeros((d, v.shape[1]), dtype=F64)
    out = torch.zeros((T, v.shape[1]), dtype=F64)
    for t in range(T):
        kv = torch.outer(k[t], v[t])
        out[t] = (S + u[:, None] * kv).T @ r[t]
        S = w[t][:, None] * S + kv
    return out


def decay(t, p: str, mixed: torch.Tensor) -> torch.Tensor:
    """exp(-exp(.)) of the low-rank projection: a number in (0, 1) per key channel"""
    return torch.exp(-torch.exp(torch.tanh(mixed @ _w(t, p + "w1").T) @ _w(t, p + "w2").T + _w(t, p + "w0")))


def wkv(t, p: str, c: Mapping, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, d = int(c["heads"]), int(c["dim"])
    T = h.shape[0]
    mix = {s: token_mix(h, _w(t, p + "mu." + s)) for s in "rkvgw"}
    r, k, v = ((mix[s] @ _w(t, p + s).T).view(T, H, d) for s in "rkv")
    gate = silu(mix["g"] @ _w(t, p + "g").T)
    w = decay(t, p, mix["w"]).view(T, H, d)
    u = _w(t, p + "u").view(H, d)
    o = torch.cat([rms(wkv_head(r[:, a], k[:, a], v[:, a], w[:, a], u[a]), eps) for a in range(H)], dim=1)
    return (o * _w(t, p + "norm") * gate) @ _w(t, p + "o").T


# ----------------------------------------------------------------------------------------------- latent attention
def frequencies(rot: Mapping):
    """([rot / 2] angles per position, the factor on cosines and sines)"""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s is None:
        return f, 1.0
    factor, original = float(s["factor"]), float(s["original"])

    def dim(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim(float(s["fast"]))), 0), min(math.ceil(dim(float(s["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, rot: Mapping, interleaved: bool) -> torch.Tensor:
    """x [T, n, dims]; pairs are neighbours (2i, 2i + 1) or half the size apart (i, i + dims / 2)"""
    T, dims = x.shape[0], int(rot["dims"])
    f, mult = frequencies(rot)
    out = x.clone()
    pos = torch.arange(T, dtype=F64)
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        c, s = (torch.cos(pos * f[i]) * mult).view(T, 1), (torch.sin(pos * f[i]) * mult).view(T, 1)
        out[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
        out[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return out


def causal_attention(q, k, v, scale: float) -> torch.Tensor:
    """one head: q, k [T, d], v [T, dv]"""
    T = q.shape[0]
    out = torch.zeros((T, v.shape[1]), dtype=F64)
    for i in range(T):
        s = (k[:i + 1] @ q[i]) * scale
        e = torch.exp(s - s.max())
        out[i] = (e / e.sum()) @ v[:i + 1]
    return out


def latent_attention(t, p: str, c: Mapping, h: torch.Tensor, eps: float, interleaved: bool) -> torch.Tensor:
    H, d, r, dv, kr = (int(c[n]) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    T = h.shape[0]
    cq = rms(h @ _w(t, p + "dq").T, eps) * _w(t, p + "dq.norm")
    q = (cq @ _w(t, p + "uq").T).view(T, H, d + r)
    q_rot = rotate(q[:, :, d:], c["rot"], interleaved)
    down = h @ _w(t, p + "dkv").T
    lat = rms(down[:, :kr], eps) * _w(t, p + "dkv.norm")
    k_rot = rotate(down[:, None, kr:], c["rot"], interleaved)[:, 0]
    k = (lat @ _w(t, p + "uk").T).view(T, H, d)
    v = (lat @ _w(t, p + "uv").T).view(T, H, dv)
    heads = [causal_attention(torch.cat([q[:, a, :d], q_rot[:, a]], dim=1), torch.cat([k[:, a], k_rot], dim=1), v[:, a],
                              float(c["scale"])) for a in range(H)]
    return torch.stack(heads, dim=1)


def head_gate(t, p: str, h: torch.Tensor, o: torch.Tensor) -> torch.Tensor:
    """o [T, H, dv]: one number a head and row"""
    return o * sigmoid(h @ _w(t, p + "g").T)[:, :, None]


def mixer(t, p: str, kind: str, c: Mapping, h: torch.Tensor, eps: float) -> torch.Tensor:
    if kind == "wkv":
        return wkv(t, p, c, h, eps)
    o = latent_attention(t, p, c, h, eps, interleaved=kind == "latent_attention_2")
    if kind == "latent_attention_2":
        o = head_gate(t, p, h, o)
    return o.reshape(h.shape[0], -1) @ _w(t, p + "o").T


# ----------------------------------------------------------------------------------------------- feed-forward
def gated_unit(t, p: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ _w(t, p + "gate").T) * (h @ _w(t, p + "up").T)) @ _w(t, p + "down").T


def route(z: torch.Tensor, top: int):
    """z [E] logits of one row: (the picked experts, their weights)"""
    idx = torch.argsort(z, descending=True, stable=True)[:top]
    e = torch.exp(z[idx] - z[idx].max())
    return idx.tolist(), (e / e.sum()).tolist()


def experts(t, p: str, c: Mapping, h: torch.Tensor) -> torch.Tensor:
    z = h @ _w(t, p + "router").T + _w(t, p + "router.b")
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        for e, w in zip(*route(z[i], int(c["router"]["top"]))):
            out[i] += w * gated_unit(t, p + "e%d." % e, h[i:i + 1])[0]
    return out


# ----------------------------------------------------------------------------------------------- model
def owner(cfg: Mapping, i: int) -> int:
    """the layer whose tensors layer i uses"""
    j = cfg["layers"][i].get("weights_of")
    return i if j is None else owner(cfg, int(j))


def layers(cfg: Mapping, t: Mapping[str, torch.Tensor], tokens: List[int]):
    """the residual stream after every layer: a list of [T, width]"""
    eps = float(cfg["norm"]["eps"])
    x = embedding(cfg, t, tokens)
    out = []
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % owner(cfg, i)
        y = mixer(t, p + "mix.", layer["type"], layer["mixer"], norm(x, _w(t, p + "norm1"), eps), eps)
        x = x + norm(y, _w(t, p + "norm1b"), eps)
        mlp: Optional[Mapping] = layer.get("mlp")
        if mlp is not None:
            h = norm(x, _w(t, p + "norm2"), eps)
            y = gated_unit(t, p + "mlp.", h) if mlp["kind"] == "dense" else experts(t, p + "mlp.", mlp, h)
            x = x + norm(y, _w(t, p + "norm2b"), eps)
        out.append(x)
    return out


def logits(cfg: Mapping, t: Mapping[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """[T, vocab] of one sequence"""
    y = norm(layers(cfg, t, tokens)[-1], _w(t, "final.norm"), float(cfg["norm"]["eps"]))
    return y @ _w(t, "embed").T
