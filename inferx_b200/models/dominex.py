"""Dominex: from the typed config to a ``ModelSpec``.

The only file that knows how this design chooses its parts.  Every layer is the pre-norm
arrangement on an fp32 stream, x += mixer(norm1(x)); x += ffn(norm2(x)), with RMS norms
whose weights are stored around zero.  A "parallel" layer's mixer is left_scale * left +
right_scale * right: attention confined to runs of positions whose scores carry a
temperature per head and lose a logarithm of the distance, and a gated recurrence whose
gates read the current token alone.  A "latent_attention" layer keeps one latent and one
rotated key part per token, its queries going through a latent of their own; with
``kv_from`` it reads an earlier layer's records instead (a schedule entry that names that
layer's cache).  The feed-forward is a mixture of gated experts: sigmoid scores, the
largest chosen, each score multiplying its expert's input; or none.  The stream starts as
embed[token] * embedding.scale; the head is the embedding table itself, unscaled, its
logits squashed to softcap * tanh(logits / softcap).  Tensor names: ``embed``,
``final.norm``, and per layer i ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` (``.left.*``
and ``.right.*`` of a pair), ``l<i>.mlp.*``.
"""
from __future__ import annotations

from ..config.dominex_config import PARALLEL, DominexConfig
from ..parts.specs import (DistanceAttentionSpec, InterleavedRopeSpec, LatentAttentionSpec,
                           LayerSpec, MinGruSpec, ModelSpec, MoeSpec, RmsNormSpec, RunEntry,
                           ScaledPairSpec)

CANDIDATE_SHIFT = 0.5         # fixed by the design: the recurrence's candidate is u + 1/2 above 0


def _mixer(cfg: DominexConfig, layer):
    if layer.type == PARALLEL:
        p, a = layer.pair, layer.pair.left
        left = DistanceAttentionSpec(hidden=cfg.width, heads=a.heads, kv_heads=a.kv_heads,
                                     head_dim=a.dim, value_dim=a.vdim, scale=a.scale,
                                     chunk=a.chunk)
        right = MinGruSpec(hidden=cfg.width, width=p.gru_width, shift=CANDIDATE_SHIFT)
        return ScaledPairSpec(hidden=cfg.width, left=left, right=right,
                              left_scale=p.left_scale, right_scale=p.right_scale)
    m = layer.latent
    rope = None
    if m.rot_dims > 0:
        rope = InterleavedRopeSpec(head_dim=m.rot_dim, rotary_dim=m.rot_dims, theta=m.rot_base)
    return LatentAttentionSpec(
        hidden=cfg.width, heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim,
        kv_rank=m.kv_rank, scale=m.scale, window=0, position=rope, latent_eps=cfg.norm_eps,
        output_gate=False, q_rank=m.q_rank or -1, own_records=m.kv_from is None,
        fp32_weights=True, out_float32=False)


def _ffn(cfg: DominexConfig, f):
    if f is None:
        return None
    return MoeSpec(hidden=cfg.width, num_experts=f.experts, top_k=f.top,
                   expert_intermediate=f.ff, renormalize=False, routed_scale=1.0, shared=None,
                   shared_gated=False, router_name="router",
                   expert_names=("e{e}.gate", "e{e}.up", "e{e}.down"), score="sigmoid",
                   weight_input=True)


def build_spec(cfg: DominexConfig) -> ModelSpec:
    norm = RmsNormSpec(size=cfg.width, eps=cfg.norm_eps, gain_offset=1.0, suffix="")
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        ffn = _ffn(cfg, layer.mlp)
        layers.append(LayerSpec(
            prefix=f"l{i}", input_norm=norm, mixer=_mixer(cfg, layer),
            post_norm=norm if ffn is not None else None, ffn=ffn, input_norm_name="norm1",
            mixer_name="mix", post_norm_name="norm2", ffn_name="mlp", kind="pre_norm"))
        src = layer.latent.kv_from if layer.latent is not None else None
        schedule.append(RunEntry(i, cache_of=src))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden=cfg.width,
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, tied_head=True,
        embed_name="embed", final_norm_name="final.norm", head_name="embed",
        embed_scale=cfg.embedding_scale, logit_softcap=cfg.logit_softcap)
