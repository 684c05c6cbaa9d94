"""Biguzen: from the typed config to a ``ModelSpec``.

The only file that knows how this design chooses its parts.  The stream is several streams
beside each other, all equal to the embedding's row at the start; every sublayer reads a
weighted sum of them through a norm that is a tanh entry by entry, and its output enters all of
them through learned weights (the arrangement "hyper_connected").  A layer of type "mlstm"
keeps a matrix memory with exponential gates; one of type "attention" is grouped-query
attention over a window whose q, k and v have biases and pass short convolutions, with a
rotation of neighbouring pairs whose frequencies are divided by a factor, a learned sink per
head and a gate per head; with ``kv_from`` it reads an earlier layer's keys and values (a
schedule entry that names that layer's cache) and has projections for the queries alone.  The
feed-forward is a dense one with the square of relu, or a mixture of plain experts (exact
gelu, no gate): sigmoid scores, a correction used for the choice alone, groups valued by their
two best choice scores, weights normed and scaled, and a shared expert behind a sigmoid; or
none.  The last norm reads the sum of the streams; the head is the embedding table.  Tensor
names: ``embed``, ``final.norm``, and per layer i ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.hc1.*``, ``l<i>.hc2.*``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from ..config.biguzen_config import DENSE, MLSTM, BiguzenConfig
from ..parts.specs import (ActivatedMlpSpec, DynamicTanhSpec, HyperConnectionSpec, LayerSpec,
                           MatrixMemorySpec, ModelSpec, MoeSpec, PreparedAttentionSpec, RunEntry,
                           ScaledRopeSpec, StreamCopiesSpec)

RENORM_EPS = 1e-20            # fixed by the design: chosen weights over (their sum + 1e-20)
DENOMINATOR_EPS = 1e-6        # fixed by the design: added to the memory's normaliser

_ATTENTION_NAMES = tuple((n, n) for n in ("q", "k", "v", "o", "g", "sink")) + tuple(
    (f"{n}_conv", f"{n}.conv") for n in "qkv") + tuple((f"{n}_bias", f"{n}.b") for n in "qkv")


def _kept_window(cfg: BiguzenConfig, i: int) -> int:
    """How many tokens layer i's keys and values are kept for: the widest window of the
    layers that read them (0: all)."""
    windows = [layer.attention.window for j, layer in enumerate(cfg.layers)
               if layer.attention is not None and (j == i or layer.attention.kv_from == i)]
    return 0 if 0 in windows else max(windows)


def _mixer(cfg: BiguzenConfig, i: int):
    layer = cfg.layers[i]
    if layer.type == MLSTM:
        m = layer.memory
        return MatrixMemorySpec(hidden=cfg.width, heads=m.heads, dim=m.dim, vdim=m.vdim,
                                gate_cap=m.gate_cap, q_scale=float(m.dim) ** -0.5,
                                norm_eps=cfg.norm_eps, den_eps=DENOMINATOR_EPS)
    a = layer.attention
    position = None
    if a.rot is not None and a.rot.dims:
        scaling = ("linear", a.rot.factor) if a.rot.factor != 1.0 else None
        position = ScaledRopeSpec(head_dim=a.dim, rotary_dim=a.rot.dims, theta=a.rot.base,
                                  layout="interleaved", scaling=scaling)
    return PreparedAttentionSpec(
        hidden=cfg.width, heads=a.heads, kv_heads=a.kv_heads, head_dim=a.dim, value_dim=a.vdim,
        scale=a.scale, window=a.window, position=position, norm_eps=cfg.norm_eps,
        conv_taps=a.conv, bias=True, learned_sink=True, head_gate=True,
        own_kv=a.kv_from is None,
        cache_window=_kept_window(cfg, i) if a.kv_from is None else None,
        names=_ATTENTION_NAMES)


def _ffn(cfg: BiguzenConfig, f):
    if f is None:
        return None
    if f.kind == DENSE:
        return ActivatedMlpSpec(hidden=cfg.width, intermediate=f.ff, activation="relu_squared")
    shared = (ActivatedMlpSpec(hidden=cfg.width, intermediate=f.shared_ff, activation="gelu")
              if f.shared_ff else None)
    return MoeSpec(
        hidden=cfg.width, num_experts=f.experts, top_k=f.top, expert_intermediate=f.ff,
        renormalize=True, routed_scale=f.scale, shared=shared, shared_gated=shared is not None,
        shared_name="shared", shared_gate_name="shared.sg", shared_gate_suffix="",
        router_name="router", expert_names=("e{e}.up", "e{e}.down"), expert_activation="gelu",
        correction_name="correction", group_count=f.group_count, group_keep=f.group_keep,
        group_value="pair_sum", renorm_eps=RENORM_EPS, score="sigmoid")


def build_spec(cfg: BiguzenConfig) -> ModelSpec:
    norm = DynamicTanhSpec(size=cfg.width)
    connection = HyperConnectionSpec(streams=cfg.streams)
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        layers.append(LayerSpec(
            prefix=f"l{i}", input_norm=norm, mixer=_mixer(cfg, i), post_norm=norm,
            ffn=_ffn(cfg, layer.mlp), input_norm_name="norm1", mixer_name="mix",
            post_norm_name="norm2", ffn_name="mlp", kind="hyper_connected",
            connection=connection))
        schedule.append(RunEntry(
            i, cache_of=layer.attention.kv_from if layer.attention is not None else None))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden=cfg.width,
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, tied_head=True,
        embed_name="embed", final_norm_name="final.norm", head_name="embed",
        embedding=StreamCopiesSpec(streams=cfg.streams))
