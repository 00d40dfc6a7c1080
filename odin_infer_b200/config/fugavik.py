"""Configuration of the Fugavik decoder: sublayers that read the residual stream itself, with a layer norm and a learned
scale on their outputs; mixers are attention (normed and rotated heads, a sink, values mixed with the first such layer's),
attention through one key/value latent per token (no positions, a sink, a gate per head) or a gated delta rule; feed-forwards
are down relu(up)^2 or experts that read their input times their own sigmoid score.

config.json keys: "architecture", "vocab", "width", "norm" {"eps"} and "layers": a list of

    {"type": "attention" | "latent_attention" | "delta", "mixer": {...}, "mlp": null | {...}}

attention:        mixer {heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor} (absent: 1)} (absent: no
                  rotation), v_mix (absent: false)}.
latent_attention: mixer {heads, dim, vdim, kv_rank, scale}.
delta:            mixer {heads, kv_heads, dim, vdim, conv}.
mlp: {"kind": "dense", "ff"} or {"kind": "moe", "expert" {"ff"}, "router" {"experts", "top"}}.
"""
from __future__ import annotations

import dataclasses

from .base import KeyReader, ModelConfig

LAYER_TYPES = ("attention", "latent_attention", "delta")


@dataclasses.dataclass(frozen=True)
class FugavikLayer:
    type: str
    heads: int = 0
    dim: int = 0
    vdim: int = 0
    kv_heads: int = 0                 # attention, delta
    scale: float = 0.0                # attention, latent_attention
    # attention
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_factor: float = 1.0
    v_mix: bool = False
    kv_rank: int = 0                  # latent_attention
    conv: int = 0                     # delta
    # feed-forward
    mlp_kind: str | None = None       # None, "dense", "moe"
    ff: int = 0
    experts: int = 0
    top: int = 0

    def mixer_dict(self) -> dict:
        if self.type == "latent_attention":
            return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "kv_rank": self.kv_rank, "scale": self.scale}
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim}
        if self.type == "delta":
            return {**out, "conv": self.conv}
        out["scale"] = self.scale
        if self.rot_dims:
            out["rot"] = {"dims": self.rot_dims, "base": self.rot_base, "scaling": {"factor": self.rot_factor}}
        out["v_mix"] = self.v_mix
        return out

    def mlp_dict(self):
        if self.mlp_kind is None:
            return None
        if self.mlp_kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


def _sub(reader: KeyReader, key: str, where: str) -> KeyReader:
    raw = reader.raw.get(key)
    if not isinstance(raw, dict):
        reader.problems.append(f"missing key '{key}'")
        raw = {}
    return KeyReader(raw, where)


def _take(into: KeyReader, sub: KeyReader, label: str) -> None:
    into.problems += [f"{label}: {p}" for p in sub.problems]


@dataclasses.dataclass(frozen=True)
class FugavikConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-5
    layers: tuple[FugavikLayer, ...] = ()

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "FugavikConfig":
        r = KeyReader(raw, where)
        vocab, width = r.get("vocab", int), r.get("width", int)
        norm = _sub(r, "norm", "norm")
        eps = norm.get("eps", float)
        _take(r, norm, "norm")
        r.require(vocab > 0 and width > 0, f"'vocab' and 'width' must be positive, got {vocab} and {width}")
        r.require(eps > 0, f"norm eps must be positive, got {eps}")
        raw_layers = raw.get("layers")
        if not (isinstance(raw_layers, list) and raw_layers):
            r.problems.append("key 'layers' must be a list with a layer in it")
            raw_layers = []
        layers = [cls._layer(r, i, e if isinstance(e, dict) else {}) for i, e in enumerate(raw_layers)]
        # values are mixed element by element with those of the first layer that says so: equal sizes
        sizes = {(l.kv_heads, l.vdim) for l in layers if l.v_mix}
        r.require(len(sizes) <= 1, f"layers with v_mix must have equal kv_heads and vdim, got {sorted(sizes)}")
        r.finish()
        return cls(architecture=str(raw.get("architecture", "Fugavik")), vocab=vocab, width=width, norm_eps=eps,
                   layers=tuple(layers))

    @staticmethod
    def _layer(r: KeyReader, i: int, entry: dict) -> FugavikLayer:
        kind = entry.get("type")
        if kind not in LAYER_TYPES:
            r.problems.append(f"layer {i}: type must be one of {', '.join(LAYER_TYPES)}, got {kind!r}")
            return FugavikLayer(type="delta")
        m = KeyReader(entry.get("mixer") if isinstance(entry.get("mixer"), dict) else {}, f"layer {i} mixer")
        size = {k: m.get(k, int) for k in ("heads", "dim", "vdim")}
        if kind != "latent_attention":
            size["kv_heads"] = m.get("kv_heads", int)
        if kind == "latent_attention":
            size["kv_rank"] = m.get("kv_rank", int)
        if kind == "delta":
            size["conv"] = m.get("conv", int)
        m.require(min(size.values()) > 0, f"{', '.join(size)} must be positive, got {', '.join(str(v) for v in size.values())}")
        if "kv_heads" in size:
            m.require(size["heads"] % max(size["kv_heads"], 1) == 0,
                      f"heads ({size['heads']}) must be a multiple of kv_heads ({size['kv_heads']})")
        more = {}
        if kind != "delta":
            more["scale"] = m.get("scale", float)
            m.require(more["scale"] > 0, f"scale must be positive, got {more['scale']}")
        if kind == "attention":
            more["v_mix"] = m.get("v_mix", bool, False)
            if m.raw.get("rot") is not None:
                rot = _sub(m, "rot", "rot")
                dims, base, factor = rot.get("dims", int), rot.get("base", float), 1.0
                if rot.raw.get("scaling") is not None:
                    sc = _sub(rot, "scaling", "scaling")
                    factor = sc.get("factor", float)
                    sc.require(factor > 0, f"factor must be positive, got {factor}")
                    _take(rot, sc, "scaling")
                rot.require(dims >= 0 and dims % 2 == 0 and dims <= max(size["dim"], 0),
                            f"dims ({dims}) must be even and at most {size['dim']}")
                rot.require(base > 0, f"base must be positive, got {base}")
                _take(m, rot, "rot")
                more.update(rot_dims=dims, rot_base=base, rot_factor=factor)
        r.problems += [f"layer {i} mixer: {p}" for p in m.problems]
        layer = FugavikLayer(type=kind, **size, **more)
        mlp = entry.get("mlp")
        if mlp is None:
            return layer
        k = KeyReader(mlp if isinstance(mlp, dict) else {}, f"layer {i} mlp")
        mk = k.raw.get("kind")
        if mk == "dense":
            ff = k.get("ff", int)
            k.require(ff > 0, f"ff must be positive, got {ff}")
            layer = dataclasses.replace(layer, mlp_kind="dense", ff=ff)
        elif mk == "moe":
            ex, ro = _sub(k, "expert", "expert"), _sub(k, "router", "router")
            ff, n, top = ex.get("ff", int), ro.get("experts", int), ro.get("top", int)
            _take(k, ex, "expert")
            _take(k, ro, "router")
            k.require(ff > 0 and n > 0 and 0 < top <= max(n, 1),
                      f"needs ff > 0, experts > 0 and 0 < top <= experts, got ff {ff}, experts {n}, top {top}")
            layer = dataclasses.replace(layer, mlp_kind="moe", ff=ff, experts=n, top=top)
        else:
            k.problems.append(f"kind must be 'dense' or 'moe', got {mk!r}")
        r.problems += [f"layer {i} mlp: {p}" for p in k.problems]
        return layer

    def to_dict(self) -> dict:
        layers = [{"type": l.type, "mixer": l.mixer_dict(), "mlp": l.mlp_dict()} for l in self.layers]
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "layers": layers}
