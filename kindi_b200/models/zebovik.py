"""The Zebovik decoder: its config.json keys, its typed configuration and its ``ModelSpec``.

What the architecture is. ``x = embed[token]``; a list of layers, each with a norm before and after every sub-layer,
``x += norm1b(mixer(norm1(x)))``, then ``x += norm2b(ff(norm2(x)))``, all RMS norms; a final norm of the same kind, an untied
head and capped logits. ``layers[i].type`` names the layer's mixer:

* ``attention``: grouped-query softmax attention with biases on q, k and v, a rotation of (a part of) every head, a unit RMS
  norm per head after the rotation, capped scores, one added to the softmax denominator, and chunks: a position sees the
  earlier positions of its own chunk of ``mask.size`` positions. ``kv_from``: the layer has no key and value projections and
  attends, with its own queries and its own chunk size, to what an earlier attention layer has cached.
* ``mlstm``: matrix memory with exponential gates.
* ``mamba2``: state-space duality.

The feed-forward (``mlp.kind`` = ``dense``) is ``W_down relu(W_up h + b)^2 + b``; a layer may have none (``mlp``: null).

config.json is nested: ``layers[i] = {"type", "mixer": {...}, "mlp": {...} | null}``, ``norm.eps``, ``logit_softcap``,
``vocab``, ``width``. Tensors: ``embed``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.*``,
``l<i>.mlp.{up,down}`` with ``.b``, ``final.norm``, ``head``. Every size and constant comes from the configuration; nothing
here knows a particular model.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..config.model_config import ConfigError, ConfigReader
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

NULL_SCORE = 0.0                # the score without key or value in every softmax: exp(0) joins the denominator


@dataclass(frozen=True)
class ZebovikAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    rot_base: float
    rot_dims: int
    chunk: Optional[int]
    kv_from: Optional[int]


@dataclass(frozen=True)
class ZebovikMLSTM:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ZebovikMamba2:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class ZebovikLayer:
    kind: str                   # "attention" | "mlstm" | "mamba2"
    mixer: Any
    ff: Optional[int]           # the feed-forward's intermediate size, None without one


@dataclass(frozen=True)
class ZebovikConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    logit_softcap: Optional[float]
    layers: Tuple[ZebovikLayer, ...]

    def to_dict(self) -> dict:
        """the config.json that reads back as this configuration"""
        layers = []
        for l in self.layers:
            m = l.mixer
            if l.kind == "attention":
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                         "softcap": m.softcap, "rot": {"base": m.rot_base, "dims": m.rot_dims},
                         "mask": None if m.chunk is None else {"size": m.chunk}}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            elif l.kind == "mlstm":
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
            else:
                mixer = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.conv,
                         "norm_groups": m.norm_groups}
            layers.append({"type": l.kind, "mixer": mixer, "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "logit_softcap": self.logit_softcap, "layers": layers}


def _positive(what: str, v):
    if not (v > 0):
        raise ConfigError("%s must be positive, found %r" % (what, v))
    return v


def _count(r: ConfigReader, key: str, where: str, *default) -> int:
    return _positive("%s.%s" % (where, key), r.integer(key, *default))


def _optional_positive(r: ConfigReader, key: str, where: str) -> Optional[float]:
    v = r.number(key, None)
    return None if v is None else float(_positive("%s.%s" % (where, key), v))


def _read_attention(raw: Mapping[str, Any], where: str) -> ZebovikAttention:
    r = ConfigReader(raw, where)
    heads = _count(r, "heads", where)
    kv = _count(r, "kv_heads", where, heads)
    if heads % kv:
        raise ConfigError("%s: heads %d is not a multiple of kv_heads %d" % (where, heads, kv))
    dim = _count(r, "dim", where)
    vdim = _count(r, "vdim", where, dim)
    scale = float(_positive(where + ".scale", r.number("scale", dim ** -0.5)))
    cap = _optional_positive(r, "softcap", where)
    base, dims = 10000.0, 0
    rraw = r.any("rot")
    if rraw is not None:
        rr = ConfigReader(rraw, where + ".rot")
        dims = rr.integer("dims")
        base = float(_positive(where + ".rot.base", rr.number("base")))
        rr.finish(())
        if dims < 0 or dims % 2 or dims > dim:
            raise ConfigError("%s.rot: dims must be even and lie between 0 and dim %d, found %d" % (where, dim, dims))
    chunk = None
    mraw = r.any("mask")
    if mraw is not None:
        mr = ConfigReader(mraw, where + ".mask")
        chunk = _count(mr, "size", where + ".mask")
        mr.finish(())
    kv_from = r.integer("kv_from", None)
    r.finish(())
    return ZebovikAttention(heads, kv, dim, vdim, scale, cap, base, dims, chunk, kv_from)


def _read_mlstm(raw: Mapping[str, Any], where: str) -> ZebovikMLSTM:
    r = ConfigReader(raw, where)
    heads, dim = _count(r, "heads", where), _count(r, "dim", where)
    vdim = _count(r, "vdim", where, dim)
    cap = float(_positive(where + ".gate_cap", r.number("gate_cap")))
    r.finish(())
    return ZebovikMLSTM(heads, dim, vdim, cap)


def _read_mamba2(raw: Mapping[str, Any], where: str) -> ZebovikMamba2:
    r = ConfigReader(raw, where)
    heads, vdim, state = (_count(r, k, where) for k in ("heads", "vdim", "state"))
    groups, conv, parts = _count(r, "groups", where, 1), _count(r, "conv", where), _count(r, "norm_groups", where, 1)
    r.finish(())
    if heads % groups:
        raise ConfigError("%s: heads %d is not a multiple of groups %d" % (where, heads, groups))
    if conv > 8:
        raise ConfigError("%s: conv must lie between 1 and 8 taps, found %d" % (where, conv))
    if heads * vdim % parts:
        raise ConfigError("%s: %d elements cannot be normed in %d equal parts" % (where, heads * vdim, parts))
    return ZebovikMamba2(heads, vdim, state, groups, conv, parts)


_MIXERS = {"attention": _read_attention, "mlstm": _read_mlstm, "mamba2": _read_mamba2}


def read_config(raw: Mapping[str, Any]) -> ZebovikConfig:
    r = ConfigReader(raw)
    arch = r.string("architecture")
    vocab, width = _count(r, "vocab", "config.json"), _count(r, "width", "config.json")
    norm = ConfigReader(r.any("norm") or {}, "config.json: norm")
    eps = float(_positive("config.json: norm.eps", norm.number("eps")))
    norm.finish(())
    cap = _optional_positive(r, "logit_softcap", "config.json")
    lraw = r.any("layers")
    if not isinstance(lraw, (list, tuple)) or not lraw:
        raise ConfigError("config.json: layers must be a non-empty list")
    layers = []
    for i, l in enumerate(lraw):
        where = "config.json: layers[%d]" % i
        lr = ConfigReader(l, where)
        kind = lr.string("type")
        if kind not in _MIXERS:
            raise ConfigError("%s: type %r is not a mixer of this architecture (%s)" % (where, kind, ", ".join(_MIXERS)))
        mixer = _MIXERS[kind](lr.any("mixer") or {}, where + ".mixer")
        ff = None
        fraw = lr.any("mlp")
        if fraw is not None:
            fr = ConfigReader(fraw, where + ".mlp")
            how = fr.string("kind", "dense")
            if how != "dense":
                raise ConfigError("%s.mlp: kind %r is not a feed-forward of this architecture (dense)" % (where, how))
            ff = _count(fr, "ff", where + ".mlp")
            fr.finish(())
        lr.finish(())
        layers.append(ZebovikLayer(kind, mixer, ff))
    r.finish()
    for i, l in enumerate(layers):
        if l.kind == "attention" and l.mixer.kv_from is not None:
            _check_shared(layers, i)
    return ZebovikConfig(arch, vocab, width, eps, cap, tuple(layers))


def _check_shared(layers, i: int) -> None:
    """layer i attends to another layer's keys and values: that layer runs earlier, is an attention layer with
    projections of its own, and its heads fit"""
    m, j = layers[i].mixer, layers[i].mixer.kv_from
    where = "config.json: layers[%d].mixer.kv_from" % i
    if not (0 <= j < i) or layers[j].kind != "attention" or layers[j].mixer.kv_from is not None:
        raise ConfigError("%s: %r is not an earlier attention layer with keys and values of its own" % (where, j))
    o = layers[j].mixer
    if (o.kv_heads, o.dim, o.vdim) != (m.kv_heads, m.dim, m.vdim):
        raise ConfigError("%s: layer %d caches %d heads of %d and %d, this layer reads %d heads of %d and %d"
                          % (where, j, o.kv_heads, o.dim, o.vdim, m.kv_heads, m.dim, m.vdim))


EMBEDDING, HEAD, FINAL_NORM = "embed", "head", "final.norm"


def _cache_window(cfg: ZebovikConfig, i: int):
    """how many positions the cache keeps of attention layer i: the largest chunk among the layers that read it"""
    sizes = [l.mixer.chunk for n, l in enumerate(cfg.layers)
             if l.kind == "attention" and (n == i or l.mixer.kv_from == i)]
    return "all" if any(s is None for s in sizes) else max(sizes)


def build_spec(cfg: ZebovikConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"eps": cfg.eps, "weight": ""})
    layers, schedule = [], []
    for i, l in enumerate(cfg.layers):
        m = l.mixer
        source = None
        if l.kind == "attention":
            source = m.kv_from
            position = PartSpec("rotary", {"base": m.rot_base, "rotary_dim": m.rot_dims}) if m.rot_dims \
                else PartSpec("none", {})
            mixer = PartSpec("headnorm_attention", {
                "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "scale": m.scale,
                "position": position, "head_norm": {"eps": cfg.eps, "when": "after"}, "bias": "%s.b", "chunk": m.chunk,
                "softcap": m.softcap, "null_score": NULL_SCORE, "shares_kv": source is not None,
                "cache_window": _cache_window(cfg, i), "widen_heads": True,
                "names": {"q": "q", "k": "k", "v": "v", "o": "o"}})
        elif l.kind == "mlstm":
            mixer = PartSpec("mlstm", {"n_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "cap": m.gate_cap,
                                       "eps": cfg.eps})
        else:
            mixer = PartSpec("mamba2", {"n_heads": m.heads, "n_groups": m.groups, "state": m.state, "v_head_dim": m.vdim,
                                        "conv": m.conv, "norm_groups": m.norm_groups, "eps": cfg.eps})
        ff = None
        if l.ff is not None:
            ff = PartSpec("dense", {"intermediate": l.ff, "activation": "relu2", "bias": True})
        block = PartSpec("sandwich", {
            "norm1": norm, "mixer": mixer, "norm1b": norm, "norm2": norm, "feed_forward": ff, "norm2b": norm,
            "names": {"norm1": "norm1", "mixer": "mix.", "norm1b": "norm1b", "norm2": "norm2", "feed_forward": "mlp.",
                      "norm2b": "norm2b"}})
        layers.append(LayerSpec(block, "l%d." % i))
        schedule.append(ScheduleEntry(layer=i, cache=i, reads_cache_of=source))
    spec = ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, width=cfg.width, layers=tuple(layers),
        schedule=tuple(schedule), final_norm=norm, final_norm_prefix=FINAL_NORM,
        embedding=PartSpec("table", {"name": EMBEDDING, "vocab": cfg.vocab}),
        head=PartSpec("linear", {"name": HEAD, "vocab": cfg.vocab, "softcap": cfg.logit_softcap}),
        # a layer without a feed-forward has no use for its norms: a folder that stores them all the same is accepted
        may_ignore=tuple("l%d.%s" % (i, n) for i, l in enumerate(cfg.layers) if l.ff is None for n in ("norm2", "norm2b")))
    spec.validate()
    return spec


register_architecture("Zebovik", build_spec, read_config)
