"""The Bafilorn decoder written out in parts.

s residual streams start as scale * E[token] + P[hash of (token before, token)].  Every sublayer reads an RMSNorm (weight
1 + w) of a weighted sum of the streams, and its output joins all streams through a learned connection.  Mixers:
`latent_attention` (queries and keys/values through latents, a rotated part in pairs, a sigmoid gate per element), `lightning`
(fixed decays, one norm over all heads), `parallel` (attention over chunks whose values are its keys, with biases, one added
to the softmax's denominator and a sigmoid gate per element, beside a gated linear unit; half the sum of the two, each normed
over the width).  Feed-forwards: down relu(up)^2.  `loop` repeats some layers, each run with a cache and state of its own.
Then the norm of the streams' sum and the head.
Tensor names: `embed`, `bigram`, `l<i>.norm1|norm2`, `l<i>.hc1|hc2.in|out|mix`, `l<i>.mix.dq|dq.norm|uq|dkv|dkv.norm|uk|uv|g|o`
(latent_attention), `l<i>.mix.q|k|v|g|norm|o` (lightning), `l<i>.mix.left.q|q.b|k|k.b|g|o|o.b|out` and
`l<i>.mix.right.y|y.b|x|x.b|conv|conv.b|ra|ra.b|ri|ri.b|lam|o|out` (parallel), `l<i>.mlp.up|down`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..parts.base import PartSpec
from ..parts.spec import ModelSpec, ScheduleEntry
from .bafilorn import RAMP_KEYS, BafilornConfig
from .registry import register_architecture


def build_bafilorn_spec(cfg: BafilornConfig) -> ModelSpec:
    def norm(weight: str, read: str | None = None) -> PartSpec:
        return PartSpec("streams_rmsnorm", dict(width=cfg.width, eps=cfg.norm_eps, weight=weight, streams=cfg.streams, read=read,
                                                one_plus=True))

    def connection(name: str) -> PartSpec:
        return PartSpec("hyper", dict(streams=cfg.streams, mix=name + ".mix", out=name + ".out"))

    blocks, encodings, tolerated = [], {}, []

    def rotation(l, layout: str) -> str | None:
        if l.rot_dims == 0:
            return None
        name = f"rope_{layout}_{l.rot_dims}_{l.rot_base!r}_{l.ramp!r}"
        encodings[name] = PartSpec("rope", dict(
            rotary_dim=l.rot_dims, theta=l.rot_base, layout=layout, precise=True, exact_angles=True,
            ramp=dict(zip(RAMP_KEYS, l.ramp)) if l.ramp is not None else None))
        return name

    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        m = p + "mix."
        if l.type == "latent_attention":
            mixer = PartSpec("latent_attention", dict(
                width=cfg.width, n_heads=l.heads, head_dim=l.dim, rot_dim=l.rot_dim, v_head_dim=l.vdim, q_rank=l.q_rank,
                kv_rank=l.kv_rank, position_encoding=rotation(l, "pairs"), eps=cfg.norm_eps, scale=l.scale, gate=m + "g",
                gate_per_head=False,
                names={"dq": m + "dq", "dq_norm": m + "dq.norm", "uq": m + "uq", "dkv": m + "dkv", "dkv_norm": m + "dkv.norm",
                       "uk": m + "uk", "uv": m + "uv", "o": m + "o"}))
        elif l.type == "lightning":
            mixer = PartSpec("lightning", dict(
                width=cfg.width, n_heads=l.heads, head_dim=l.dim, v_head_dim=l.vdim, decay=l.decay, eps=cfg.norm_eps,
                names={s: m + s for s in ("q", "k", "v", "g", "norm", "o")}))
        else:
            lm, rm = m + "left.", m + "right."
            left = PartSpec("gqa_attention", dict(
                width=cfg.width, n_q_heads=l.heads, n_kv_heads=l.kv_heads, head_dim=l.dim, position_encoding=rotation(l, "halves"),
                qk_norm=False, eps=cfg.norm_eps, scale=l.scale, chunk=l.chunk, values_are_keys=True, sink_logit=0.0, gate=lm + "g",
                names={s: lm + s for s in ("q", "k", "o")}, biases={s: lm + s + ".b" for s in ("q", "k", "o")}))
            right = PartSpec("gated_linear_unit", dict(
                width=cfg.width, inner=l.inner, blocks=l.blocks, taps=l.conv,
                names={"conv": rm + "conv", "conv_bias": rm + "conv.b", "lam": rm + "lam", "o": rm + "o",
                       **{s + t: rm + s + u for s in ("y", "x", "ra", "ri") for t, u in (("", ""), ("_bias", ".b"))}}))
            mixer = PartSpec("side_by_side", dict(left=left, right=right, width=cfg.width, left_scale=0.5, right_scale=0.5,
                                                  norms={"left": lm + "out", "right": rm + "out"}, eps=cfg.norm_eps))
        ffn = None
        if l.ff:
            ffn = PartSpec("activated", dict(width=cfg.width, inner=l.ff, activation="relu2",
                                             names={"up": p + "mlp.up", "down": p + "mlp.down"}))
        else:
            tolerated += [p + n for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix")]   # a layer without feed-forward reads none
        blocks.append(PartSpec("prenorm", dict(
            mixer=mixer, feed_forward=ffn, norm_mixer=norm(p + "norm1", p + "hc1.in"), connect_mixer=connection(p + "hc1"),
            norm_feed_forward=norm(p + "norm2", p + "hc2.in") if ffn is not None else None,
            connect_feed_forward=connection(p + "hc2") if ffn is not None else None)))
    pair = None
    if cfg.bigram is not None:
        pair = {"weight": "bigram", "buckets": cfg.bigram[0], "mul_prev": cfg.bigram[1], "mul_cur": cfg.bigram[2]}
    return ModelSpec(
        width=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_table", dict(vocab_size=cfg.vocab, width=cfg.width, weight="embed", scale=cfg.embedding_scale,
                                               pair=pair, streams=cfg.streams)),
        position_encodings=encodings,
        layers=tuple(blocks),
        schedule=tuple(ScheduleEntry(i) for i in cfg.layer_runs()),
        final_norm=norm("final.norm"),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, width=cfg.width, weight="head")),
        tolerated_tensors=tuple(tolerated),
    )


register_architecture("Bafilorn", BafilornConfig, build_bafilorn_spec)
