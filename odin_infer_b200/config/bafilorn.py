"""Configuration of the Bafilorn decoder: several residual streams joined by learned connections, some layers run more than
once, token embeddings plus a hashed table of token pairs; mixers are attention through latents (gated per element), linear
attention with fixed decays, or attention whose values are its keys beside a gated linear unit; feed-forwards are
down relu(up)^2.

config.json keys: "architecture", "vocab", "width", "streams", "norm" {"eps"}, "embedding" {"scale" (absent: 1), "bigram"
{"buckets", "mul_prev", "mul_cur"} (absent: no pair table)}, "loop" {"start", "stop", "times"} (absent: every layer runs once)
and "layers": a list of

    {"type": "latent_attention" | "lightning" | "parallel", "mixer": {...}, "mlp": null | {"kind": "dense", "ff"}}

latent_attention: mixer {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {dims, base}} (dims = rot_dim).
lightning:        mixer {heads, dim, vdim, decay: a list of one number per head}.
parallel:         mixer {left {heads, kv_heads, dim, vdim (= dim), scale, rot {dims, base, scaling {factor, original, fast, slow}
                  (absent: none)}, mask {size}}, right {width, blocks, conv}}.
"""
from __future__ import annotations

import dataclasses

from .base import KeyReader, ModelConfig

LAYER_TYPES = ("latent_attention", "lightning", "parallel")
RAMP_KEYS = ("factor", "original", "fast", "slow")


@dataclasses.dataclass(frozen=True)
class BafilornLayer:
    type: str
    heads: int = 0                     # every attention and the recurrence over heads
    dim: int = 0
    vdim: int = 0
    scale: float = 0.0                 # latent_attention, parallel
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_dim: int = 0                   # latent_attention
    q_rank: int = 0
    kv_rank: int = 0
    decay: tuple[float, ...] = ()      # lightning
    kv_heads: int = 0                  # parallel: the attention ...
    chunk: int = 0
    ramp: tuple | None = None          # (factor, original, fast, slow)
    inner: int = 0                     # ... and the gated unit
    blocks: int = 1
    conv: int = 0
    ff: int = 0                        # 0: no feed-forward

    def mixer_dict(self) -> dict:
        if self.type == "lightning":
            return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        rot = {"dims": self.rot_dims, "base": self.rot_base}
        if self.type == "latent_attention":
            return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                    "kv_rank": self.kv_rank, "scale": self.scale, "rot": rot}
        if self.ramp is not None:
            rot["scaling"] = dict(zip(RAMP_KEYS, self.ramp))
        return {"left": {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                         "rot": rot, "mask": {"size": self.chunk}},
                "right": {"width": self.inner, "blocks": self.blocks, "conv": self.conv}}


def _sub(reader: KeyReader, key: str, where: str) -> KeyReader:
    raw = reader.raw.get(key)
    if not isinstance(raw, dict):
        reader.problems.append(f"missing key '{key}'")
        raw = {}
    return KeyReader(raw, where)


def _take(into: KeyReader, sub: KeyReader, label: str) -> None:
    into.problems += [f"{label}: {p}" for p in sub.problems]


def _sizes(r: KeyReader, *keys: str) -> dict:
    size = {k: r.get(k, int) for k in keys}
    r.require(min(size.values()) > 0, f"{', '.join(size)} must be positive, got {', '.join(str(v) for v in size.values())}")
    return size


def _rotation(r: KeyReader, at_most: int) -> dict:
    rot = _sub(r, "rot", "rot")
    dims, base = rot.get("dims", int), rot.get("base", float)
    rot.require(dims >= 0 and dims % 2 == 0 and dims <= at_most, f"dims ({dims}) must be even and at most {at_most}")
    rot.require(base > 0 and base != 1, f"base must be positive and not 1, got {base}")
    ramp = None
    if rot.raw.get("scaling") is not None:
        sc = _sub(rot, "scaling", "scaling")
        ramp = tuple(sc.get(k, float) for k in RAMP_KEYS)
        sc.require(min(ramp) > 0, f"{', '.join(RAMP_KEYS)} must be positive, got {', '.join(str(v) for v in ramp)}")
        _take(rot, sc, "scaling")
    _take(r, rot, "rot")
    return {"rot_dims": dims, "rot_base": base, "ramp": ramp}


@dataclasses.dataclass(frozen=True)
class BafilornConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    streams: int = 1
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    bigram: tuple | None = None       # (buckets, mul_prev, mul_cur)
    loop: tuple | None = None         # (start, stop, times)
    layers: tuple[BafilornLayer, ...] = ()

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "BafilornConfig":
        r = KeyReader(raw, where)
        vocab, width, streams = r.get("vocab", int), r.get("width", int), r.get("streams", int)
        norm = _sub(r, "norm", "norm")
        eps = norm.get("eps", float)
        _take(r, norm, "norm")
        r.require(vocab > 0 and width > 0, f"'vocab' and 'width' must be positive, got {vocab} and {width}")
        r.require(1 <= streams <= 16, f"'streams' must lie between 1 and 16, got {streams}")
        r.require(eps > 0, f"norm eps must be positive, got {eps}")
        emb = KeyReader(raw.get("embedding") if isinstance(raw.get("embedding"), dict) else {}, "embedding")
        scale, bigram = emb.get("scale", float, 1.0), None
        if emb.raw.get("bigram") is not None:
            b = _sub(emb, "bigram", "bigram")
            bigram = (b.get("buckets", int), b.get("mul_prev", int), b.get("mul_cur", int))
            b.require(bigram[0] > 0, f"buckets must be positive, got {bigram[0]}")
            _take(emb, b, "bigram")
        _take(r, emb, "embedding")
        raw_layers = raw.get("layers")
        if not (isinstance(raw_layers, list) and raw_layers):
            r.problems.append("key 'layers' must be a list with a layer in it")
            raw_layers = []
        layers = [cls._layer(r, i, e if isinstance(e, dict) else {}) for i, e in enumerate(raw_layers)]
        loop = None
        if raw.get("loop") is not None:
            lo = _sub(r, "loop", "loop")
            loop = tuple(lo.get(k, int) for k in ("start", "stop", "times"))
            lo.require(0 <= loop[0] < loop[1] <= len(raw_layers) and loop[2] >= 1,
                       f"start {loop[0]}, stop {loop[1]}, times {loop[2]} do not name layers to repeat")
            _take(r, lo, "loop")
        r.finish()
        return cls(architecture=str(raw.get("architecture", "Bafilorn")), vocab=vocab, width=width, streams=streams, norm_eps=eps,
                   embedding_scale=scale, bigram=bigram, loop=loop, layers=tuple(layers))

    @staticmethod
    def _layer(r: KeyReader, i: int, entry: dict) -> BafilornLayer:
        kind = entry.get("type")
        if kind not in LAYER_TYPES:
            r.problems.append(f"layer {i}: type must be one of {', '.join(LAYER_TYPES)}, got {kind!r}")
            return BafilornLayer(type="lightning")
        m = KeyReader(entry.get("mixer") if isinstance(entry.get("mixer"), dict) else {}, f"layer {i} mixer")
        if kind == "lightning":
            more = _sizes(m, "heads", "dim", "vdim")
            decay = m.get("decay", list)
            ok = isinstance(decay, list) and all(isinstance(d, (int, float)) and not isinstance(d, bool) for d in decay)
            m.require(ok and len(decay or []) == more["heads"], f"decay must be a list of {more['heads']} numbers, one per head")
            more["decay"] = tuple(float(d) for d in decay) if ok else ()
        elif kind == "latent_attention":
            more = _sizes(m, "heads", "dim", "vdim", "q_rank", "kv_rank", "rot_dim")
            more["scale"] = m.get("scale", float)
            more.update(_rotation(m, more["rot_dim"]))
            m.require(more["rot_dims"] == more["rot_dim"], f"rot dims ({more['rot_dims']}) must be rot_dim ({more['rot_dim']})")
        else:
            a = _sub(m, "left", "left")
            more = _sizes(a, "heads", "kv_heads", "dim", "vdim")
            more["scale"] = a.get("scale", float)
            more.update(_rotation(a, more["dim"]))
            a.require(more["heads"] % max(more["kv_heads"], 1) == 0,
                      f"heads ({more['heads']}) must be a multiple of kv_heads ({more['kv_heads']})")
            a.require(more["vdim"] == more["dim"], f"values are keys: vdim ({more['vdim']}) must be dim ({more['dim']})")
            mask = _sub(a, "mask", "mask")
            more["chunk"] = _sizes(mask, "size")["size"]
            _take(a, mask, "mask")
            _take(m, a, "left")
            g = _sub(m, "right", "right")
            size = _sizes(g, "width", "blocks", "conv")
            g.require(size["width"] % max(size["blocks"], 1) == 0, f"width ({size['width']}) must be a multiple of blocks ({size['blocks']})")
            _take(m, g, "right")
            more.update(inner=size["width"], blocks=size["blocks"], conv=size["conv"])
        if "scale" in more:
            m.require(more["scale"] > 0, f"scale must be positive, got {more['scale']}")
        r.problems += [f"layer {i} mixer: {p}" for p in m.problems]
        mlp = entry.get("mlp")
        if mlp is not None:
            k = KeyReader(mlp if isinstance(mlp, dict) else {}, f"layer {i} mlp")
            k.require(k.raw.get("kind") == "dense", f"kind must be 'dense', got {k.raw.get('kind')!r}")
            more["ff"] = _sizes(k, "ff")["ff"]
            r.problems += [f"layer {i} mlp: {p}" for p in k.problems]
        return BafilornLayer(type=kind, **more)

    def layer_runs(self) -> list[int]:
        """The layers in the order in which they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return [*range(start), *list(range(start, stop)) * times, *range(stop, n)]

    def to_dict(self) -> dict:
        layers = [{"type": l.type, "mixer": l.mixer_dict(), "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None} for l in self.layers]
        emb: dict = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
               "norm": {"eps": self.norm_eps}, "embedding": emb, "layers": layers}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out
