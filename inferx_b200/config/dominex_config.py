"""Typed configuration of the Dominex design, read from its own ``config.json``.

Top level: ``architecture``, ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``,
``logit_softcap`` and ``layers`` (one object per layer: ``type`` is "parallel" - chunked
attention with a distance penalty beside a gated recurrence - or "latent_attention",
``mixer`` holds the sizes and constants, ``mlp`` the feed-forward, kind "moe", or null for
none).  A latent layer with ``kv_from`` names an earlier latent layer whose cached records
it reads in place of its own.  Every size and constant a model of the design can vary is
read from there; what has a natural "off" may be absent (no chunks, no rotation, no soft cap,
scales of one).  ``q_rank`` may be left to the checkpoint's tensors.  A key of the wrong
JSON type, an unknown layer type or feed-forward kind, or sizes that do not fit are refused
with the place named.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .model_config import ConfigError, _Reader

ARCHITECTURE = "Dominex"
PARALLEL, LATENT = "parallel", "latent_attention"
MOE = "moe"


@dataclass(frozen=True)
class DominexAttention:
    heads: int
    kv_heads: int
    dim: int                  # query / key entries per head
    vdim: int                 # value entries per head
    scale: float              # factor on q . k
    chunk: int = 0            # positions a run of visible keys spans; 0: every earlier key


@dataclass(frozen=True)
class DominexParallel:
    left: DominexAttention
    gru_width: int
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass(frozen=True)
class DominexLatent:
    heads: int
    dim: int                  # plain query/key entries per head
    rot_dim: int              # rotated query/key entries per head
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    q_rank: int = 0           # 0: the checkpoint's
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class DominexMoe:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class DominexLayer:
    type: str
    pair: Optional[DominexParallel] = None
    latent: Optional[DominexLatent] = None
    mlp: Optional[DominexMoe] = None


@dataclass(frozen=True)
class DominexConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    logit_softcap: float
    layers: Tuple[DominexLayer, ...]
    torch_dtype: str = "bfloat16"
    architecture: str = ARCHITECTURE
    eos_token_ids: tuple = ()

    ARCHITECTURE = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_json(cls, obj: Mapping[str, Any], where: str = "config.json") -> "DominexConfig":
        r = _Reader(obj, where)
        name = r.string("architecture")
        if name != ARCHITECTURE:
            raise ConfigError(f"{where}: architecture {name!r} is not {ARCHITECTURE!r}")
        emb = _Reader(_object(obj, "embedding", where, {}), f"{where}: embedding")
        norm = _Reader(_object(obj, "norm", where), f"{where}: norm")
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = tuple(_layer(lo, f"{where}: layers[{i}]") for i, lo in enumerate(raw_layers))
        cap = r.number("logit_softcap", 0.0) if obj.get("logit_softcap") is not None else 0.0
        cfg = cls(vocab=r.integer("vocab"), width=r.integer("width"),
                  embedding_scale=emb.number("scale", 1.0), norm_eps=norm.number("eps"),
                  logit_softcap=cap, layers=layers,
                  torch_dtype=r.string("torch_dtype", "bfloat16"))
        cfg.validate(where)
        return cfg

    def validate(self, where: str = "config") -> None:
        def need(ok, msg):
            if not ok:
                raise ConfigError(f"{where}: {msg}")

        need(self.vocab > 0 and self.width > 0, "'vocab' and 'width' must be positive")
        need(self.norm_eps > 0, "'norm.eps' must be positive")
        need(self.logit_softcap >= 0, "'logit_softcap' must not be negative")
        for i, layer in enumerate(self.layers):
            at = f"layers[{i}].mixer"
            if layer.type == PARALLEL:
                a = layer.pair.left
                need(min(a.heads, a.kv_heads, a.dim, a.vdim) > 0 and a.heads % a.kv_heads == 0,
                     f"{at}.left: {a.heads} heads of {a.dim} / {a.vdim} over {a.kv_heads} "
                     "key/value heads")
                need(a.chunk >= 0, f"{at}.left: 'mask.size' must not be negative")
                need(layer.pair.gru_width > 0, f"{at}.right: 'width' must be positive")
            else:
                m = layer.latent
                need(min(m.heads, m.vdim, m.kv_rank) > 0 and m.dim >= 0 and m.rot_dim >= 0
                     and m.dim + m.rot_dim > 0 and m.q_rank >= 0,
                     f"{at}: sizes must be positive")
                need(m.rot_dims % 2 == 0 and 0 <= m.rot_dims <= m.rot_dim,
                     f"{at}: 'rot.dims' {m.rot_dims} must be even and at most rot_dim "
                     f"{m.rot_dim}")
                need(m.rot_base > 0, f"{at}: 'rot.base' must be positive")
                if m.kv_from is not None:
                    src = (self.layers[m.kv_from].latent if 0 <= m.kv_from < i else None)
                    need(src is not None and src.kv_from is None,
                         f"{at}: 'kv_from' {m.kv_from} is not an earlier latent layer with "
                         "records of its own")
                    need((src.kv_rank, src.rot_dim, src.rot_dims, src.rot_base)
                         == (m.kv_rank, m.rot_dim, m.rot_dims, m.rot_base),
                         f"{at}: records of layer {m.kv_from} have other sizes or another "
                         "rotation")
            f = layer.mlp
            if f is not None:
                need(f.ff > 0 and 0 < f.top <= f.experts,
                     f"layers[{i}].mlp: {f.top} of {f.experts} experts of {f.ff}")

    def to_json(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
               "layers": [], "torch_dtype": self.torch_dtype}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        for layer in self.layers:
            if layer.type == PARALLEL:
                p, a = layer.pair, layer.pair.left
                left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim,
                        "scale": a.scale}
                if a.chunk:
                    left["mask"] = {"size": a.chunk}
                mixer = {"left": left, "right": {"width": p.gru_width},
                         "left_scale": p.left_scale, "right_scale": p.right_scale}
            else:
                m = layer.latent
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim,
                         "kv_rank": m.kv_rank, "scale": m.scale,
                         "rot": {"base": m.rot_base, "dims": m.rot_dims}}
                if m.q_rank:
                    mixer["q_rank"] = m.q_rank
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            f = layer.mlp
            out["layers"].append({
                "type": layer.type, "mixer": mixer,
                "mlp": None if f is None else {
                    "kind": MOE, "expert": {"ff": f.ff},
                    "router": {"experts": f.experts, "top": f.top}}})
        return out


def _object(obj, key, where, default=None):
    v = obj.get(key) if isinstance(obj, Mapping) else None
    if v is None:
        if default is None:
            raise ConfigError(f"{where}: required object '{key}' is missing")
        return default
    if not isinstance(v, Mapping):
        raise ConfigError(f"{where}: '{key}' must be an object, got {v!r}")
    return v


def _parallel(mixer, where) -> DominexParallel:
    m = _Reader(mixer, where)
    a = _Reader(_object(mixer, "left", where), f"{where}.left")
    heads, dim = a.integer("heads"), a.integer("dim")
    mask = _Reader(_object(a.obj, "mask", f"{where}.left", {}), f"{where}.left.mask")
    left = DominexAttention(heads=heads, kv_heads=a.integer("kv_heads", heads), dim=dim,
                            vdim=a.integer("vdim", dim), scale=a.number("scale"),
                            chunk=mask.integer("size", 0))
    right = _Reader(_object(mixer, "right", where), f"{where}.right")
    return DominexParallel(left=left, gru_width=right.integer("width"),
                           left_scale=m.number("left_scale", 1.0),
                           right_scale=m.number("right_scale", 1.0))


def _latent(mixer, where) -> DominexLatent:
    m = _Reader(mixer, where)
    rot_dim, dim = m.integer("rot_dim"), m.integer("dim")
    rot_obj = _object(mixer, "rot", where, {})
    rot = _Reader(rot_obj, f"{where}.rot")
    return DominexLatent(
        heads=m.integer("heads"), dim=dim, rot_dim=rot_dim, vdim=m.integer("vdim", dim),
        kv_rank=m.integer("kv_rank"), scale=m.number("scale"),
        rot_base=rot.number("base", 10000.0),
        rot_dims=rot.integer("dims", rot_dim if rot_obj else 0), q_rank=m.integer("q_rank", 0),
        kv_from=m.integer("kv_from") if mixer.get("kv_from") is not None else None)


def _layer(obj, where) -> DominexLayer:
    if not isinstance(obj, Mapping):
        raise ConfigError(f"{where}: must be an object")
    kind = _Reader(obj, where).string("type")
    mixer = _object(obj, "mixer", where)
    pair = latent = None
    if kind == PARALLEL:
        pair = _parallel(mixer, f"{where}.mixer")
    elif kind == LATENT:
        latent = _latent(mixer, f"{where}.mixer")
    else:
        # an unknown kind of layer is refused, never run as another
        raise ConfigError(f"{where}: unknown layer type {kind!r} "
                          f"(known: {PARALLEL!r}, {LATENT!r})")
    mlp = None
    if obj.get("mlp") is not None:
        f = _Reader(_object(obj, "mlp", where), f"{where}.mlp")
        fk = f.string("kind")
        if fk != MOE:
            raise ConfigError(f"{where}.mlp: unknown kind {fk!r} (known: {MOE!r})")
        ex = _Reader(_object(f.obj, "expert", f"{where}.mlp"), f"{where}.mlp.expert")
        ro = _Reader(_object(f.obj, "router", f"{where}.mlp"), f"{where}.mlp.router")
        mlp = DominexMoe(experts=ro.integer("experts"), top=ro.integer("top"),
                         ff=ex.integer("ff"))
    return DominexLayer(type=kind, pair=pair, latent=latent, mlp=mlp)
