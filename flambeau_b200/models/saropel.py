"""Saropel: configuration -> ModelSpec.

A decoder of parallel blocks (one "1 + w" RMS norm, whose rows mixer and feed-forward both read).  The embedding is the
token's row plus a row of a second table that a hash of the token before it and the token itself picks.  The mixer is,
layer by layer, grouped-query attention under a sliding window without rotation whose scores pass a soft cap
('attention'), or one whose values are the projected keys, with a norm per head, a rotation with stretched frequencies
on part of a head and a sigmoid gate per head ('attention_2').  The feed-forward is dense (SiLU-gated) or a mixture of
experts whose operands are cut off (softmax over all experts, a choice within the best groups, weights as they are)
beside a shared expert behind a sigmoid gate per token.  Behind every layer the token's id gives the stream something
of its own (`side.*`).  A stretch of layers [loop.start, loop.stop) runs loop.times times in a row on the same weights,
every pass with a cache of its own; before every pass but the first the embedding output joins the stream, and before
every pass the pass's learned vector (`loop.step`).  Tensor names are the checkpoint's: embed, bigram, side.embed,
loop.step, l<i>.norm1, l<i>.mix.*, l<i>.mlp.*, l<i>.side.*, final.norm, head.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.saropel import ARCHITECTURE, VALUES_FROM_KEYS, SaropelConfig
from ..parts.spec import LayerCall, ModelSpec, PartSpec

NORM_INIT = ("normal", 0.1)          # the stored weight is the deviation from one
PLAIN_NORM_INIT = ("one_plus_normal", 0.1)
ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "g": "g"}
EXPERT_SLOPE = 1.702                 # an expert's gate is g sigmoid(1.702 g)


def build_spec(cfg: SaropelConfig) -> ModelSpec:
    D, eps, n = cfg.width, cfg.norm_eps, len(cfg.layers)

    def norm(prefix, name):
        return PartSpec("norm", "rmsnorm", dict(width=D, eps=eps, init=NORM_INIT, weight_offset=1.0, weight_name=name),
                        prefix)

    def feed_forward(f, prefix):
        if f is None:
            return None
        names = ("gate", "up", "down")
        if f.kind == "dense":
            return PartSpec("feed_forward", "gated_mlp", dict(width=D, inner=f.ff, activation="silu", names=names), prefix)
        shared = None
        if f.shared is not None:
            shared = PartSpec("feed_forward", "gated_mlp", dict(
                width=D, inner=f.shared.ff, activation="limited", limit=f.shared.limit, slope=EXPERT_SLOPE,
                names=names), prefix + "shared.")
        return PartSpec("feed_forward", "routed_experts", dict(
            width=D, inner=f.expert.ff, experts=f.experts, top=f.top, activation="limited", limit=f.expert.limit,
            slope=EXPERT_SLOPE, gated=True, rule="softmax_of_all", renormalize=False, groups=f.groups,
            keep_groups=f.keep_groups, router_bias=False, shared=shared, shared_gate=shared is not None), prefix)

    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        params = dict(width=D, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                      window=m.window, scale=m.scale, names=ATTENTION_NAMES, weights_float32=True)
        if VALUES_FROM_KEYS[layer.type]:
            params.update(
                values_from_keys=True, gate="head",
                qk_norm=PartSpec("norm", "rmsnorm", dict(width=m.dim, eps=eps, init=PLAIN_NORM_INIT)),
                position=PartSpec("position", "rotary_half", dict(
                    head_dim=m.dim, theta=m.rot.base, rotary_dim=m.rot.dims, stretch=m.rot.scaling))
                if m.rot is not None else None)
        else:
            params.update(softcap=m.softcap)
        block = PartSpec("block", "parallel", dict(
            mixer=PartSpec("mixer", "attention", params, p + "mix."), norm=norm(p, "norm1"),
            feed_forward=feed_forward(layer.mlp, p + "mlp.")), p)
        if cfg.side_dim:
            block = PartSpec("block", "token_input", dict(
                block=block, width=D, dim=cfg.side_dim, offset=i * cfg.side_dim, vocab=cfg.vocab, table="side.embed",
                table_width=n * cfg.side_dim,
                norm=PartSpec("norm", "rmsnorm", dict(width=D, eps=eps, init=PLAIN_NORM_INIT, weight_name="norm"),
                              p + "side.")), p + "side.")
        layers.append(block)

    reentry = None
    if cfg.loop is None:
        order = [LayerCall(i) for i in range(n)]
    else:
        lp = cfg.loop
        order = [LayerCall(i) for i in range(lp.start)]
        for t in range(lp.times):
            order += [LayerCall(i, reenter=(i == lp.start), pass_index=t) for i in range(lp.start, lp.stop)]
        order += [LayerCall(i) for i in range(lp.stop, n)]
        reentry = PartSpec("reentry", "add", dict(width=D, step_name="step", passes=lp.times), "loop.")
    pairs = dict(cfg.bigram.to_dict(), weight_name="bigram") if cfg.bigram is not None else None
    return ModelSpec(
        hidden_size=D, vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", "token_embedding", dict(vocab=cfg.vocab, width=D, weight_name="embed",
                                                                pairs=pairs), ""),
        layers=layers, order=order, final_norm=norm("final.", "norm"),
        head=PartSpec("head", "lm_head", dict(vocab=cfg.vocab, width=D, weight_name="head"), ""),
        reentry=reentry)


register_architecture(ARCHITECTURE, SaropelConfig, build_spec, replace=True)
