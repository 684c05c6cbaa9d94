"""Typed configuration of the Biguzen design, read from its own ``config.json``.

Top level: ``architecture``, ``vocab``, ``width``, ``streams`` (residual streams beside each
other), ``norm.eps`` and ``layers``: one object per layer with ``type`` ("mlstm": a matrix
memory with exponential gates; "attention": grouped-query attention over a window, with
biases, short convolutions, a rotation of neighbouring pairs, a learned sink and a gate per
head), ``mixer`` (its sizes and constants) and ``mlp`` (``kind`` "dense" or "moe", or null for
none).  An attention layer with ``kv_from`` names an earlier attention layer whose keys and
values it reads in the place of its own.  Every size and constant a model of the design can
vary is read from there; what has a natural "off" may be absent (no window, no convolution,
no rotation, no scaling of its frequencies, no groups, no shared expert, no feed-forward).  A
key of the wrong JSON type, an unknown layer type or feed-forward kind, or sizes that do not
fit are refused with the place named.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .mapovik_config import _object
from .model_config import ConfigError, _Reader

ARCHITECTURE = "Biguzen"
MLSTM, ATTENTION = "mlstm", "attention"
DENSE, MOE = "dense", "moe"


@dataclass(frozen=True)
class BiguzenMemory:
    heads: int
    dim: int                  # query / key entries per head
    vdim: int                 # value entries per head
    gate_cap: float           # gates' pre-activations are squashed to cap * tanh(z / cap)


@dataclass(frozen=True)
class BiguzenRotation:
    dims: int
    base: float
    factor: float = 1.0       # every frequency is divided by it


@dataclass(frozen=True)
class BiguzenAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0           # mask.size: a query sees itself and the window - 1 before it; 0: all
    conv: int = 0             # taps of the convolutions after the projections; 0: none
    rot: Optional[BiguzenRotation] = None
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class BiguzenMlp:
    kind: str
    ff: int                   # dense: inner width; moe: an expert's inner width
    experts: int = 0
    top: int = 0
    scale: float = 1.0        # the chosen experts' weights are multiplied by it
    group_count: int = 0      # 0: no groups
    group_keep: int = 0
    shared_ff: int = 0        # 0: no shared expert


@dataclass(frozen=True)
class BiguzenLayer:
    type: str
    memory: Optional[BiguzenMemory] = None
    attention: Optional[BiguzenAttention] = None
    mlp: Optional[BiguzenMlp] = None


@dataclass(frozen=True)
class BiguzenConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[BiguzenLayer, ...]
    torch_dtype: str = "bfloat16"
    architecture: str = ARCHITECTURE
    eos_token_ids: tuple = ()

    ARCHITECTURE = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_json(cls, obj: Mapping[str, Any], where: str = "config.json") -> "BiguzenConfig":
        r = _Reader(obj, where)
        name = r.string("architecture")
        if name != ARCHITECTURE:
            raise ConfigError(f"{where}: architecture {name!r} is not {ARCHITECTURE!r}")
        norm = _Reader(_object(obj, "norm", where), f"{where}: norm")
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = tuple(_layer(lo, f"{where}: layers[{i}]") for i, lo in enumerate(raw_layers))
        cfg = cls(vocab=r.integer("vocab"), width=r.integer("width"),
                  streams=r.integer("streams", 1), norm_eps=norm.number("eps"), layers=layers,
                  torch_dtype=r.string("torch_dtype", "bfloat16"))
        cfg.validate(where)
        return cfg

    def validate(self, where: str = "config") -> None:
        def need(ok, msg):
            if not ok:
                raise ConfigError(f"{where}: {msg}")

        need(self.vocab > 0 and self.width > 0, "'vocab' and 'width' must be positive")
        need(self.streams > 0, f"'streams' {self.streams} must be positive")
        need(self.norm_eps > 0, "'norm.eps' must be positive")
        for i, layer in enumerate(self.layers):
            at = f"layers[{i}].mixer"
            if layer.type == MLSTM:
                m = layer.memory
                need(min(m.heads, m.dim, m.vdim) > 0,
                     f"{at}: {m.heads} heads of {m.dim} / {m.vdim}")
                need(m.gate_cap > 0, f"{at}: 'gate_cap' {m.gate_cap} must be positive")
            else:
                a = layer.attention
                need(min(a.heads, a.kv_heads, a.dim, a.vdim) > 0 and a.heads % a.kv_heads == 0,
                     f"{at}: {a.heads} heads of {a.dim} / {a.vdim} over {a.kv_heads} key/value "
                     "heads")
                need(a.window >= 0, f"{at}.mask: size {a.window} must not be negative")
                need(a.conv >= 0, f"{at}: conv {a.conv} must not be negative")
                if a.rot is not None:
                    need(0 <= a.rot.dims <= a.dim and a.rot.dims % 2 == 0 and a.rot.base > 0,
                         f"{at}.rot: {a.rot.dims} rotated entries of {a.dim}, base {a.rot.base}")
                    need(a.rot.factor > 0, f"{at}.rot.scaling: factor {a.rot.factor}")
                if a.kv_from is not None:
                    src = (self.layers[a.kv_from].attention if 0 <= a.kv_from < i else None)
                    need(src is not None and src.kv_from is None,
                         f"{at}: 'kv_from' {a.kv_from} is not an earlier attention layer with "
                         "keys and values of its own")
                    need((src.kv_heads, src.dim, src.vdim, src.rot)
                         == (a.kv_heads, a.dim, a.vdim, a.rot),
                         f"{at}: keys and values of layer {a.kv_from} have other sizes or another "
                         "rotation")
            f = layer.mlp
            if f is not None:
                at = f"layers[{i}].mlp"
                need(f.ff > 0, f"{at}: inner width {f.ff}")
                if f.kind == MOE:
                    need(0 < f.top <= f.experts,
                         f"{at}.router: {f.top} of {f.experts} experts")
                    if f.group_count:
                        need(f.group_count > 0 and f.experts % f.group_count == 0
                             and 0 < f.group_keep <= f.group_count
                             and f.group_keep * (f.experts // f.group_count) >= f.top,
                             f"{at}.router.groups: {f.group_keep} of {f.group_count} groups over "
                             f"{f.experts} experts, {f.top} chosen")
                    need(f.shared_ff >= 0, f"{at}.shared: inner width {f.shared_ff}")

    def to_json(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "streams": self.streams, "norm": {"eps": self.norm_eps}, "layers": [],
               "torch_dtype": self.torch_dtype}
        for layer in self.layers:
            if layer.type == MLSTM:
                m = layer.memory
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
            else:
                a = layer.attention
                mixer = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim,
                         "scale": a.scale, "conv": a.conv}
                if a.window:
                    mixer["mask"] = {"size": a.window}
                if a.rot is not None:
                    mixer["rot"] = {"dims": a.rot.dims, "base": a.rot.base}
                    if a.rot.factor != 1.0:
                        mixer["rot"]["scaling"] = {"factor": a.rot.factor}
                if a.kv_from is not None:
                    mixer["kv_from"] = a.kv_from
            mlp = None
            f = layer.mlp
            if f is not None and f.kind == DENSE:
                mlp = {"kind": DENSE, "ff": f.ff}
            elif f is not None:
                router = {"experts": f.experts, "top": f.top, "scale": f.scale}
                if f.group_count:
                    router["groups"] = {"count": f.group_count, "keep": f.group_keep}
                mlp = {"kind": MOE, "expert": {"ff": f.ff}, "router": router}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            out["layers"].append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        return out


def _attention(m, at) -> BiguzenAttention:
    mask = _Reader(_object(m.obj, "mask", at, default={}), f"{at}.mask")
    rot = None
    if m.obj.get("rot") is not None:
        ro = _Reader(_object(m.obj, "rot", at), f"{at}.rot")
        sc = _Reader(_object(ro.obj, "scaling", f"{at}.rot", default={}), f"{at}.rot.scaling")
        rot = BiguzenRotation(dims=ro.integer("dims"), base=ro.number("base"),
                              factor=sc.number("factor", 1.0))
    heads, dim = m.integer("heads"), m.integer("dim")
    return BiguzenAttention(
        heads=heads, kv_heads=m.integer("kv_heads", heads), dim=dim, vdim=m.integer("vdim", dim),
        scale=m.number("scale"), window=mask.integer("size", 0), conv=m.integer("conv", 0),
        rot=rot, kv_from=m.integer("kv_from") if m.obj.get("kv_from") is not None else None)


def _mlp(obj, where) -> BiguzenMlp:
    f = _Reader(obj, where)
    kind = f.string("kind")
    if kind == DENSE:
        return BiguzenMlp(kind=DENSE, ff=f.integer("ff"))
    if kind != MOE:
        raise ConfigError(f"{where}: unknown kind {kind!r} (known: {DENSE!r}, {MOE!r})")
    ex = _Reader(_object(obj, "expert", where), f"{where}.expert")
    ro = _Reader(_object(obj, "router", where), f"{where}.router")
    count = keep = shared = 0
    if ro.obj.get("groups") is not None:
        gr = _Reader(_object(ro.obj, "groups", f"{where}.router"), f"{where}.router.groups")
        count, keep = gr.integer("count"), gr.integer("keep")
    if obj.get("shared") is not None:
        shared = _Reader(_object(obj, "shared", where), f"{where}.shared").integer("ff")
    return BiguzenMlp(kind=MOE, ff=ex.integer("ff"), experts=ro.integer("experts"),
                      top=ro.integer("top"), scale=ro.number("scale", 1.0), group_count=count,
                      group_keep=keep, shared_ff=shared)


def _layer(obj, where) -> BiguzenLayer:
    if not isinstance(obj, Mapping):
        raise ConfigError(f"{where}: must be an object")
    kind = _Reader(obj, where).string("type")
    if kind not in (MLSTM, ATTENTION):
        # an unknown kind of layer is refused, never run as another
        raise ConfigError(f"{where}: unknown layer type {kind!r} "
                          f"(known: {MLSTM!r}, {ATTENTION!r})")
    at = f"{where}.mixer"
    m = _Reader(_object(obj, "mixer", where), at)
    memory = attention = None
    if kind == MLSTM:
        dim = m.integer("dim")
        memory = BiguzenMemory(heads=m.integer("heads"), dim=dim, vdim=m.integer("vdim", dim),
                               gate_cap=m.number("gate_cap"))
    else:
        attention = _attention(m, at)
    mlp = None
    if obj.get("mlp") is not None:
        mlp = _mlp(_object(obj, "mlp", where), f"{where}.mlp")
    return BiguzenLayer(type=kind, memory=memory, attention=attention, mlp=mlp)
