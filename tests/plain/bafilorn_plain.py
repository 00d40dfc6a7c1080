"""Plain, slow implementation of the Bafilorn decoder: the oracle of its tests.

Whole sequences, no cache, one function per mechanism, float64 on the CPU.  It shares no code with the product
package (only the oracles' reader of a model folder, which is test code too).

In this file's notation (n tokens, width d, s residual streams X[0] .. X[s-1], each [n, d]):

    X[i] = scale * E[token] + P[pair of (token before, token)]          for every i
    for every layer run (the runs of `loop` repeat some layers):
        X = hyper(X, hc1, y) with y = mixer(rms(sum_i in_i X[i]) * (1 + w))
        X = hyper(X, hc2, y) with y = W_down relu(W_up rms(..) * (1 + w'))^2          (if the layer has a feed-forward)
    logits = H rms(sum_i X[i]) * (1 + w_final)

hyper(X, hc, y)[j] = sum_i mix[i, j] X[i] + out[j] y;   rms(y) = y / sqrt(mean(y^2) + eps).

Mixers: `latent_attention` (queries through a latent, keys and values of all heads from one normed latent and one rotated
key part per token, a sigmoid gate per element), `lightning` (linear attention with a fixed decay per head between SiLUs,
one norm over all heads), `parallel` (attention whose values are its unrotated keys, over chunks, with one added to the
softmax's denominator, beside a gated linear recurrence per channel behind a short convolution).
"""
from __future__ import annotations

import math

import torch

from .qwen3_plain import read_model_folder  # noqa: F401  (re-exported: the folder reader of the oracles)

F64 = torch.float64


def _same(t):
    return t


def to_bfloat16_and_back(t: torch.Tensor) -> torch.Tensor:
    """What a tensor loses when it is stored in bfloat16: the `rnd` of the functions below, to see how far rounding
    of activations alone moves a result (the tolerance of a comparison in bfloat16 is taken from that)."""
    return t.to(torch.bfloat16).to(t.dtype)


def rms(y, w, eps):
    return y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ---- embedding ------------------------------------------------------------------------------------------------
def embed(config, w, tokens):
    e = config["embedding"]
    pair = e["bigram"]
    rows = []
    for i, t in enumerate(tokens):
        r = pair["buckets"] if i == 0 else (tokens[i - 1] * pair["mul_prev"] + t * pair["mul_cur"]) % pair["buckets"]
        rows.append(w["embed"][t] * float(e["scale"]) + w["bigram"][r])
    return torch.stack(rows)


# ---- residual streams -----------------------------------------------------------------------------------------
def read_streams(X, weights):
    """sum_i weights[i] X[i]; X: [s, n, d]."""
    return sum(weights[i] * X[i] for i in range(X.shape[0]))


def hyper(X, mix, out, y):
    """All streams at once from the old ones; mix: [from, to], out: [to]."""
    return torch.stack([sum(mix[i, j] * X[i] for i in range(X.shape[0])) + out[j] * y for j in range(X.shape[0])])


# ---- rotation -------------------------------------------------------------------------------------------------
def frequencies(dims: int, base: float, scaling=None):
    """(frequency of every pair, the factor on cosine and sine).  scaling {factor, original, fast, slow}: pairs that turn
    often within `original` positions keep their frequency, those that turn seldom are slowed down by `factor`, with a
    ramp over the pairs' indices between the two."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns):
        return dims * math.log(original / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index_of(scaling["fast"])), 0), min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(t, positions, dims: int, base: float, pairs: bool, scaling=None):
    """t: [n, heads, e]; pair i of a head's first `dims` elements (pairs: 2i and 2i + 1, else i and i + dims/2) turns by
    position * f_i; the elements from `dims` on pass."""
    out = t.clone()
    freq, gain = frequencies(dims, base, scaling)
    for i, f in enumerate(freq):
        a = torch.tensor([float(p) * f for p in positions], dtype=F64)
        c, s = (torch.cos(a) * gain)[:, None], (torch.sin(a) * gain)[:, None]
        iu, iv = (2 * i, 2 * i + 1) if pairs else (i, i + dims // 2)
        u, v = t[:, :, iu], t[:, :, iv]
        out[:, :, iu] = u * c - v * s
        out[:, :, iv] = v * c + u * s
    return out


# ---- attention ------------------------------------------------------------------------------------------------
def attend(q, k, v, scale: float, chunk: int = 0, one_added: bool = False):
    """q: [n, H, e], k: [n, G, e], v: [n, G, ev]; query head h reads key/value head h // (H / G), query i sees the keys
    j <= i (of its own chunk of `chunk` positions, where given); one_added: the softmax's denominator is 1 + the sum."""
    n, H, _ = q.shape
    group = H // k.shape[1]
    pos = torch.arange(n)
    hidden = pos[None, :] > pos[:, None]
    if chunk:
        hidden = hidden | (pos[None, :] // chunk != pos[:, None] // chunk)
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T) * scale
        s[hidden] = -math.inf
        m = s.amax(dim=1)
        if one_added:
            m = torch.clamp(m, min=0.0)
        e = torch.exp(s - m[:, None])
        den = e.sum(dim=1) + (torch.exp(-m) if one_added else 0.0)
        out[:, h] = (e @ v[:, h // group]) / den[:, None]
    return out


def latent_attention(h, w, p, mx, eps, rnd=_same):
    n = h.shape[0]
    H, e, r, ev, kr = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    base = float(mx["rot"]["base"])
    cq = rnd(rms(h @ w[p + "dq"].T, w[p + "dq.norm"], eps))
    q = rnd(cq @ w[p + "uq"].T).view(n, H, e + r)
    down = h @ w[p + "dkv"].T
    c = rnd(rms(down[:, :kr], w[p + "dkv.norm"], eps))
    k_rot = rnd(rotate(down[:, None, kr:], range(n), r, base, True))
    q_rot = rnd(rotate(q[:, :, e:], range(n), r, base, True))
    k = torch.cat([(c @ w[p + "uk"].T).view(n, H, e), k_rot.expand(n, H, r)], dim=2)
    v = (c @ w[p + "uv"].T).view(n, H, ev)
    o = attend(torch.cat([q[:, :, :e], q_rot], dim=2), k, v, float(mx["scale"]))
    return rnd(o.reshape(n, H * ev) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def key_value_attention(h, w, p, mx, rnd=_same):
    """Attention whose values are its keys before their rotation."""
    n = h.shape[0]
    H, G, e = mx["heads"], mx["kv_heads"], mx["dim"]
    rot = mx["rot"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, e)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, e)
    turn = lambda t: rnd(rotate(t, range(n), rot["dims"], float(rot["base"]), False, rot.get("scaling")))  # noqa: E731
    o = attend(turn(q), turn(k), rnd(k), float(mx["scale"]), mx["mask"]["size"], one_added=True)
    o = rnd(rnd(o).reshape(n, H * e) * torch.sigmoid(h @ w[p + "g"].T))
    return o @ w[p + "o"].T + w[p + "o.b"]


# ---- recurrences ----------------------------------------------------------------------------------------------
def decay_walk(q, k, v, decay, state=None):
    """q, k: [n, H, e], v: [n, H, ev], decay: [H]; state: None (a sequence from its start) or H matrices [e, ev] that are
    updated in place."""
    n, H, e = q.shape
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for h in range(H):
        S = torch.zeros(e, v.shape[2], dtype=F64) if state is None else state[h]
        for t in range(n):
            S = float(decay[h]) * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
        if state is not None:
            state[h] = S
    return out


def lightning(h, w, p, mx, eps, rnd=_same):
    n = h.shape[0]
    H, e, ev = mx["heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(h @ w[p + s].T) for s in "qkv")
    o = decay_walk(q.view(n, H, e), k.view(n, H, e), v.view(n, H, ev), mx["decay"]).reshape(n, H * ev)
    return rnd(rms(o, w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_conv(x, w, b, before=None):
    """out[t, c] = b[c] + sum_j w[c, j] x[t - (taps - 1 - j), c]; before: the taps - 1 rows before the first (None: zeros)."""
    taps = w.shape[1]
    pad = torch.zeros(taps - 1, x.shape[1], dtype=F64) if before is None else before
    xx = torch.cat([pad, x], dim=0)
    return b + sum(xx[j:j + x.shape[0]] * w[:, j] for j in range(taps))


def block_gate(u, w, b):
    """sigmoid(W_b u_b + bias_b) for each of the equal consecutive parts u_b of u; w: [blocks, m, m] ([out, in])."""
    n, blocks = u.shape[0], w.shape[0]
    parts = u.view(n, blocks, -1)
    return torch.sigmoid(torch.stack([parts[:, i] @ w[i].T + b[i] for i in range(blocks)], dim=1)).reshape(n, -1)


def gated_unit_walk(u, r, i, lam, state=None):
    """Per channel log a = -8 r softplus(lam), S = a S + sqrt(1 - a^2) i u.  Returns (every S, the last)."""
    S = torch.zeros(u.shape[1], dtype=F64) if state is None else state
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out, S


def gated_unit(h, w, p, rnd=_same):
    y = gelu_tanh(rnd(h @ w[p + "y"].T) + w[p + "y.b"])
    u = rnd(causal_conv(rnd(h @ w[p + "x"].T) + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"]))
    r, i = block_gate(u, w[p + "ra"], w[p + "ra.b"]), block_gate(u, w[p + "ri"], w[p + "ri.b"])
    S, _ = gated_unit_walk(u, r, i, w[p + "lam"])
    return rnd(S * y) @ w[p + "o"].T


def parallel(h, w, p, mx, eps, rnd=_same):
    left = key_value_attention(h, w, p + "left.", mx["left"], rnd)
    right = gated_unit(h, w, p + "right.", rnd)
    return 0.5 * (rms(left, w[p + "left.out"], eps) + rms(right, w[p + "right.out"], eps))


# ---- the rest -------------------------------------------------------------------------------------------------
def relu2_mlp(h, up, down, rnd=_same):
    return rnd(torch.relu(h @ up.T) ** 2) @ down.T


def schedule(config):
    """The layers in the order in which they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(config: dict, weights: dict, tokens, return_layers: bool = False, rnd=_same):
    """Logits [n, vocab] of a whole sequence (and the sum of the streams after every layer run).  rnd: applied to what a
    16-bit engine would store in 16 bits (what a matrix product reads, cached rows); the identity by default."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    tokens = [int(t) for t in tokens]
    X = torch.stack([embed(config, w, tokens)] * config["streams"])
    after = []
    mixers = {"latent_attention": latent_attention, "lightning": lightning, "parallel": parallel}
    for i in schedule(config):
        layer, p = config["layers"][i], f"l{i}."
        h = rnd(rms(read_streams(X, w[p + "hc1.in"]), 1.0 + w[p + "norm1"], eps))
        X = hyper(X, w[p + "hc1.mix"], w[p + "hc1.out"], mixers[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, rnd))
        if layer.get("mlp") is not None:
            h = rnd(rms(read_streams(X, w[p + "hc2.in"]), 1.0 + w[p + "norm2"], eps))
            X = hyper(X, w[p + "hc2.mix"], w[p + "hc2.out"], relu2_mlp(h, w[p + "mlp.up"], w[p + "mlp.down"], rnd))
        after.append(X.sum(dim=0))
    logits = rnd(rms(X.sum(dim=0), 1.0 + w["final.norm"], eps)) @ w["head"].T
    return (logits, torch.stack(after)) if return_layers else logits
