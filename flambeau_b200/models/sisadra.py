"""Sisadra: configuration -> ModelSpec.

A decoder of pre-norm blocks whose norms take the mean off (a weight, no bias).  The embedding is the token's row, scaled,
plus a row of a second table that a hash of the token before it and the token itself picks.  The mixer is, layer by layer,
differential attention within chunks of positions ('attention': biases on all four maps, a norm and a rotation with slowed
long waves on every map of q and k), attention over cached latents without positions, with a sink ('latent_attention'), or
a gated delta rule with a decay per key channel and an output gate, both made through narrow middles ('channel_delta').
The feed-forward, where a layer has one, is plain (the exact GELU).  The logits pass a soft cap.  Tensor names are the
checkpoint's: embed, bigram, l<i>.norm1 / norm2, l<i>.mix.*, l<i>.mlp.up / down, final.norm, head.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sisadra import ARCHITECTURE, SisadraConfig
from ..parts.spec import LayerCall, ModelSpec, PartSpec

UNIT_EPS = 1e-6                      # in the root of the recurrence's unit vectors


def _mixer(kind: str, m, D: int, eps: float, prefix: str) -> PartSpec:
    if kind == "attention":
        position = PartSpec("position", "rotary_half", dict(head_dim=m.dim, theta=m.rot.base, rotary_dim=m.rot.dims,
                                                            stretch=m.rot.scaling)) if m.rot is not None else None
        return PartSpec("mixer", "diff_attention", dict(
            width=D, num_heads=m.heads, num_kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, chunk=m.chunk,
            scale=m.scale, diff=m.diff, eps=eps, bias=True, out_bias=True, head_gate=False, qk_norm=True,
            position=position), prefix)
    if kind == "latent_attention":
        return PartSpec("mixer", "latent_attention", dict(
            width=D, num_heads=m.heads, head_dim=m.dim, rot_dim=0, value_dim=m.vdim, kv_rank=m.kv_rank, q_rank=None,
            window=0, scale=m.scale, eps=eps, gate=False, sink=True), prefix)
    return PartSpec("mixer", "gated_delta", dict(
        width=D, num_heads=m.heads, num_qk_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, conv=m.conv, eps=eps,
        unit_eps=UNIT_EPS, decay="channel", gate="sigmoid", low_rank_gate=True, rank=m.dim), prefix)


def build_spec(cfg: SisadraConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps

    def norm(prefix, name):
        return PartSpec("norm", "layernorm", dict(width=D, eps=eps, init=("one_plus_normal", 0.1), weight_name=name), prefix)

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        params = dict(mixer=_mixer(layer.type, layer.mixer, D, eps, p + "mix."), mixer_norm=norm(p, "norm1"))
        if layer.ff:
            params.update(feed_forward=PartSpec("feed_forward", "mlp", dict(width=D, inner=layer.ff, activation="gelu"),
                                                p + "mlp."),
                          feed_forward_norm=norm(p, "norm2"))
        layers.append(PartSpec("block", "pre_norm", params, p))
    pairs = dict(cfg.bigram.to_dict(), weight_name="bigram") if cfg.bigram is not None else None
    return ModelSpec(
        hidden_size=D, vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", "token_embedding", dict(vocab=cfg.vocab, width=D, scale=cfg.embedding_scale,
                                                                weight_name="embed", pairs=pairs), ""),
        layers=layers, order=[LayerCall(i) for i in range(len(cfg.layers))], final_norm=norm("final.", "norm"),
        head=PartSpec("head", "lm_head", dict(vocab=cfg.vocab, width=D, weight_name="head", softcap=cfg.logit_softcap), ""))


register_architecture(ARCHITECTURE, SisadraConfig, build_spec, replace=True)
