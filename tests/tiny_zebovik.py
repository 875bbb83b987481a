"""Small Zebovik configurations with seeded random weights for the tests, with one token that stands out.

The configurations differ in every size and option: the order of the mixers, head counts and groups, values wider and
narrower than keys, head sizes the tensor-core attention kernels take and sizes no vector load takes, rotations of the whole
head, of a part and of nothing, chunks smaller and larger than a cache page and no chunks at all, a layer that reads another
one's keys and values under a larger or a smaller chunk, caps that bend the scores and caps that hardly touch them, one
convolution tap and many, one group of states and several, norms in one part and in several, layers without a feed-forward.
"""
from __future__ import annotations

import json
import os
import random
from typing import List

NEEDLE, PROBE = 3, 4            # token ids: the needle stands out for every probe
CODE = 3.0                      # the size of the planted embedding features, far above the random ones
KEPT = 2                        # the stream's first columns keep the token's own features through all layers


def _att(heads, kv, dim, vdim, chunk, softcap, base, dims, ff=None, kv_from=None, scale=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 12.0 / dim,
         "softcap": softcap, "rot": {"base": base, "dims": dims}, "mask": None if chunk is None else {"size": chunk}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _mem(heads, dim, vdim, cap, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _ssd(heads, vdim, state, groups, conv, parts, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": parts}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _config(vocab, width, eps, cap, layers):
    return {"architecture": "Zebovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": layers}


# A: small everything; chunks smaller than a page, the second layer reads the first one's keys under a larger chunk with a
#    cap and a scale of its own; values wider than keys; a layer without a feed-forward
ZE_A = _config(211, 64, 1e-5, 15.0, [
    _att(4, 2, 16, 24, 40, 20.0, 10000.0, 8, 48),
    _att(8, 2, 16, 24, 56, 35.0, 10000.0, 8, kv_from=0, scale=0.6),
    _mem(2, 16, 24, 8.0, 40), _ssd(4, 16, 24, 1, 4, 2, 56)])
# B: head size 64 (the tensor-core attention kernels run in bfloat16), whole heads rotated, a chunk that is no multiple of a
#    page, the reader's chunk smaller than the owner's; several groups of states; the recurrent layers first
ZE_B = _config(300, 128, 1e-6, 40.0, [
    _ssd(8, 16, 64, 4, 2, 4, 96), _att(6, 2, 64, 64, 150, 30.0, 500000.0, 64, 96), _mem(3, 64, 32, 15.0, 96),
    _att(6, 2, 64, 64, 96, 30.0, 500000.0, 64, 64, kv_from=1), _ssd(6, 32, 32, 2, 4, 1)])
# C: head size 128 with values of 64 (widened in the cache), one key/value head, a cap below the scores (they are bent), a
#    chunk of exactly a page, a width that is no power of two, one convolution tap, a group per head, one head of memory
ZE_C = _config(257, 200, 2e-6, 10.0, [
    _att(4, 1, 128, 64, 64, 6.0, 10000.0, 32, 136), _mem(1, 128, 80, 12.0, 72), _ssd(3, 40, 128, 3, 1, 1, 40),
    _att(3, 1, 128, 64, 128, 8.0, 10000.0, 32, kv_from=0)])
# D: sizes that no vector load or tensor-core tile takes, a key/value head per query head, chunks of 17, eight taps
ZE_D = _config(131, 72, 1e-5, 25.0, [
    _mem(3, 10, 7, 5.0, 20), _att(5, 5, 24, 10, 17, 12.0, 30000.0, 6), _ssd(2, 9, 5, 2, 8, 3, 36),
    _att(3, 1, 9, 24, 100, 50.0, 100.0, 2, 20)])
# E: attention without chunks, without a cap and without a rotation, no cap on the logits, keys of the memory wider than 128,
#    heads of 80 (widened to 128)
ZE_E = _config(401, 160, 1e-5, None, [
    _mem(2, 200, 72, 10.0, 64), _att(4, 2, 80, 80, None, None, 10000.0, 0, 64), _ssd(4, 48, 16, 2, 3, 2, 96)])
TINY = {"A": (ZE_A, 41), "B": (ZE_B, 42), "C": (ZE_C, 43), "D": (ZE_D, 44), "E": (ZE_E, 45)}


def plant(cfg: dict, t: dict, seed: int) -> None:
    """random weights made sharp, in place.

    The needle's embedding row has one large feature (column 0), a probe's another (column 1), and no branch writes into those
    columns. Attention: the keys of the first key/value head read column 0 into their last element with a weight far above the
    random ones, the queries of that group's heads read column 1 into theirs: after the unit norms both are about sqrt(dim)
    there, and the layer's scale makes the score stand out. Matrix memory: the same with the first head's keys and queries,
    the input gate reads column 0 (the needle is written strongly) and forget gates lie near one (it is still there hundreds
    of tokens later). State space: the first group's B reads column 0 and its C column 1, decays are slow. Queries of the
    memory are correlated with its keys, so that a token's own score is not a small difference of large numbers. Convolutions,
    gains and biases are drawn large enough to matter."""
    import torch
    g = torch.Generator().manual_seed(seed + 1)

    def randn(*shape):
        return torch.randn(*shape, generator=g)
    emb = t["embed"]
    emb[:, :KEPT] = 0.0
    emb[:, KEPT:] = randn(emb.shape[0], emb.shape[1] - KEPT)
    emb[NEEDLE, 0] = CODE * emb.shape[1] ** 0.5 / 4
    emb[PROBE, 1] = CODE * emb.shape[1] ** 0.5 / 4
    for n in list(t):
        if n.endswith(("norm1", "norm2", "norm1b", "norm2b", "final.norm", "mix.norm")):
            t[n] = 1.0 + 0.2 * randn(*t[n].shape)
        elif n.endswith((".q.b", ".k.b", ".v.b", ".up.b", ".down.b")):
            t[n] = 0.3 * randn(*t[n].shape)
        elif n.endswith((".q", ".k", ".v", ".g", ".in", ".up", ".down", ".mix.o", ".mix.i", ".mix.f")) or n == "head":
            t[n] = randn(*t[n].shape) / t[n].shape[1] ** 0.5
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], "l%d.mix." % i
        if layer["type"] == "attention":
            H, G, dim = m["heads"], m["kv_heads"], m["dim"]
            at = dim - 1
            if m.get("kv_from") is None:
                t[p + "k"][at, :] = 0.0
                t[p + "k"][at, 0] = 8.0
                t[p + "v"][:, 0] = torch.sign(t[p + "v"][:, 5])
            for h in range(H // G):
                t[p + "q"][h * dim + at, :] = 0.0
                t[p + "q"][h * dim + at, 1] = 8.0
        elif layer["type"] == "mlstm":
            d = m["dim"]
            t[p + "q"] = 0.8 * t[p + "k"] + 0.3 * t[p + "q"]
            for n, col in (("k", 0), ("q", 1)):
                t[p + n][d - 1, :] = 0.0
                t[p + n][d - 1, col] = 4.0
            t[p + "v"][:, 0] = torch.sign(t[p + "v"][:, 5])
            t[p + "i"][:, 0] = 2.0
            t[p + "i.b"] = 0.5 * randn(*t[p + "i.b"].shape)
            t[p + "f"] *= 0.5
            t[p + "f.b"] = 3.0 + randn(*t[p + "f.b"].shape)
        else:
            H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            inner = H * dv
            t[p + "conv"] = 0.4 * randn(*t[p + "conv"].shape)
            t[p + "conv"][:, -1] += 0.8
            t[p + "conv.b"] = 0.3 * randn(*t[p + "conv.b"].shape)
            t[p + "in"][inner + inner + N - 1, :] = 0.0
            t[p + "in"][inner + inner + N - 1, 0] = 6.0                                   # B of the first group
            t[p + "in"][inner + inner + G * N + N - 1, :] = 0.0
            t[p + "in"][inner + inner + G * N + N - 1, 1] = 6.0                           # C of the first group
            t[p + "in"][inner:2 * inner, 0] = torch.sign(t[p + "in"][inner:2 * inner, 5])     # the needle's x
            t[p + "dt_bias"] = -2.0 + 0.7 * randn(H)
            t[p + "A_log"] = -2.5 + 0.5 * randn(H)
            t[p + "D"] = 1.0 + 0.3 * randn(H)
    for n in list(t):
        if n.endswith((".mix.o", ".down", ".down.b")):
            t[n][:KEPT] = 0.0


def make_model(tmp_path, name: str, dtype: str = "bfloat16") -> str:
    """a model folder with the configuration's planted random weights (``plant``)"""
    import torch
    from kindi_b200.config.registry import model_from_config
    from kindi_b200.parts.model import expected_tensors, tensor_inits
    from kindi_b200.weights.random_init import random_tensors
    from kindi_b200.weights.safetensors_io import write_file
    cfg, seed = TINY[name]
    cfg = json.loads(json.dumps(cfg))
    d = os.path.join(str(tmp_path), "ze_%s_%s" % (name, dtype))
    if os.path.isfile(os.path.join(d, "model.safetensors")):
        return d
    os.makedirs(d, exist_ok=True)
    _, spec = model_from_config(cfg)
    t = random_tensors(expected_tensors(spec), seed, dtype=torch.float32, inits=tensor_inits(spec))
    plant(cfg, t, seed)
    tdt = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
    t = {n: v.to(tdt) for n, v in t.items()}
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_file(os.path.join(d, "model.safetensors"), t, metadata={"format": "pt"})
    return d


def needle_request(vocab: int, length: int, needle_at: int, probes: List[int], rng: random.Random) -> List[int]:
    """random tokens (neither needle nor probe) with the needle at `needle_at` and probes at the listed places"""
    toks = []
    for i in range(length):
        t = rng.randrange(vocab)
        while t in (NEEDLE, PROBE):
            t = rng.randrange(vocab)
        toks.append(NEEDLE if i == needle_at else PROBE if i in probes else t)
    return toks


def edge_places(cfg: dict, length: int) -> List[int]:
    """positions around the borders of every chunk size of the configuration and of the cache's pages"""
    sizes = {64} | {l["mixer"]["mask"]["size"] for l in cfg["layers"]
                    if l["type"] == "attention" and l["mixer"].get("mask")}
    out = set()
    for s in sizes:
        for c in range(s, length, s):
            out |= {c - 1, c, c + 1}
    return sorted(p for p in out if 0 < p < length)
