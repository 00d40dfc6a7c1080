"""The Fugavik decoder written out in parts.

x = E[token].  Sublayers read x as it is and a layer norm with a learned scale stands on their outputs:
x += s1 * ln1(mixer(x)), x += s2 * ln2(feed_forward(x)).  Mixers: `attention` (heads normed, then rotated in halves with
frequencies slowed down by one factor, a sink logit, values mixed with those of the first layer that says v_mix),
`latent_attention` (one normed key/value latent per token, no positions, a sink, a sigmoid gate per head), `delta` (the gated
delta rule behind a short convolution).  Feed-forwards: down relu(up)^2, or gated experts with the largest sigmoid scores, each
reading its score times its input.  Then a layer norm and the head.
Tensor names: `embed`, `l<i>.norm1|norm1.b|ls1|norm2|norm2.b|ls2`, `l<i>.mix.q|k|v|o|q.norm|k.norm|vmix|sink` (attention),
`l<i>.mix.q|dkv|dkv.norm|uk|uv|sink|g|o` (latent_attention), `l<i>.mix.q|k|v|q.conv|k.conv|v.conv|b|a|A_log|dt_bias|norm|g|o`
(delta), `l<i>.mlp.up|down`, `l<i>.mlp.router`, `l<i>.mlp.e<n>.gate|up|down`, `final.norm|final.norm.b`, `head`.
"""
from __future__ import annotations

from ..parts.base import PartSpec
from ..parts.spec import ModelSpec, ScheduleEntry
from .fugavik import FugavikConfig
from .registry import register_architecture


def build_fugavik_spec(cfg: FugavikConfig) -> ModelSpec:
    def norm(name: str, scale: str | None = None) -> PartSpec:
        return PartSpec("layernorm", dict(width=cfg.width, eps=cfg.norm_eps, weight=name, bias=name + ".b", scale=scale))

    as_it_is = PartSpec("none", dict(width=cfg.width))
    blocks, encodings, tolerated = [], {}, []
    first_mixing = next((i for i, l in enumerate(cfg.layers) if l.v_mix), None)
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        m = p + "mix."
        if l.type == "attention":
            pe, mix = None, None
            if l.rot_dims > 0:
                pe = f"rope_{l.rot_dims}_{l.rot_base!r}_{l.rot_factor!r}"
                encodings[pe] = PartSpec("rope", dict(rotary_dim=l.rot_dims, theta=l.rot_base, slowdown=l.rot_factor,
                                                      precise=True, exact_angles=True))
            if l.v_mix:
                mix = {"key": "first values", "lambda": m + "vmix" if i != first_mixing else None}
                if i == first_mixing:
                    tolerated.append(m + "vmix")   # the first such layer has nothing to mix with
            mixer = PartSpec("gqa_attention", dict(
                width=cfg.width, n_q_heads=l.heads, n_kv_heads=l.kv_heads, head_dim=l.dim, v_head_dim=l.vdim,
                position_encoding=pe, eps=cfg.norm_eps, scale=l.scale, sink=m + "sink", value_mix=mix,
                names={"q": m + "q", "k": m + "k", "v": m + "v", "o": m + "o", "q_norm": m + "q.norm", "k_norm": m + "k.norm"}))
        elif l.type == "latent_attention":
            mixer = PartSpec("latent_attention", dict(
                width=cfg.width, n_heads=l.heads, head_dim=l.dim, rot_dim=0, v_head_dim=l.vdim, q_rank=0, kv_rank=l.kv_rank,
                position_encoding=None, eps=cfg.norm_eps, scale=l.scale, sink=m + "sink", gate=m + "g",
                names={"q": m + "q", "dkv": m + "dkv", "dkv_norm": m + "dkv.norm", "uk": m + "uk", "uv": m + "uv", "o": m + "o"}))
        else:
            mixer = PartSpec("gated_delta_rule", dict(
                width=cfg.width, n_heads=l.heads, n_groups=l.kv_heads, head_dim=l.dim, v_head_dim=l.vdim, taps=l.conv,
                eps=cfg.norm_eps,
                names={"q": m + "q", "k": m + "k", "v": m + "v", "q_conv": m + "q.conv", "k_conv": m + "k.conv",
                       "v_conv": m + "v.conv", "g": m + "g", "b": m + "b", "a": m + "a", "A_log": m + "A_log",
                       "dt_bias": m + "dt_bias", "norm": m + "norm", "o": m + "o"}))
        ffn = None
        f = p + "mlp."
        if l.mlp_kind == "dense":
            ffn = PartSpec("activated", dict(width=cfg.width, inner=l.ff, activation="relu2",
                                             names={"up": f + "up", "down": f + "down"}))
        elif l.mlp_kind == "moe":
            ffn = PartSpec("routed_experts", dict(
                width=cfg.width, inner=l.ff, n_experts=l.experts, top=l.top, activation="silu", score="sigmoid_as_is",
                weigh_input=True,
                names={"router": f + "router", "gate": f + "e{e}.gate", "up": f + "e{e}.up", "down": f + "e{e}.down"}))
        else:
            tolerated += [p + "norm2", p + "norm2.b", p + "ls2"]   # a layer without feed-forward reads none of them
        blocks.append(PartSpec("prenorm", dict(
            mixer=mixer, feed_forward=ffn, norm_mixer=as_it_is, norm_feed_forward=as_it_is if ffn is not None else None,
            post_norm_mixer=norm(p + "norm1", p + "ls1"),
            post_norm_feed_forward=norm(p + "norm2", p + "ls2") if ffn is not None else None)))
    return ModelSpec(
        width=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_table", dict(vocab_size=cfg.vocab, width=cfg.width, weight="embed")),
        position_encodings=encodings,
        layers=tuple(blocks),
        schedule=tuple(ScheduleEntry(i) for i in range(len(blocks))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, width=cfg.width, weight="head")),
        tolerated_tensors=tuple(tolerated),
    )


register_architecture("Fugavik", FugavikConfig, build_fugavik_spec)
