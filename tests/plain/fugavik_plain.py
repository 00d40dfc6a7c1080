"""Plain, slow implementation of the Fugavik decoder: the oracle of its tests.

Whole sequences, no cache, one function per mechanism, float64 on the CPU.  It shares no code with the product
package (only the oracles' reader of a model folder, which is test code too).

In this file's notation (n tokens, width d, x the residual stream):

    x = E[token]
    for every entry of `layers`:
        x += s1 * ln(mixer(x), w1, b1);   x += s2 * ln(ffn(x), w2, b2)        (the second line if it has an ffn)
    logits = H ln(x, w_final, b_final)

ln(y, w, b) = (y - mean(y)) / sqrt(mean((y - mean(y))^2) + eps) * w + b;   rms(y, w) = y / sqrt(mean(y^2) + eps) * w.

Mixers: `attention` (grouped heads, q and k normed per head and rotated in halves with slowed-down frequencies, a sink
logit per head, values mixed with those of the first such layer), `latent_attention` (keys and values of all heads from
one normed latent per token, no positions, a sink, a sigmoid gate per head), `delta` (the gated delta rule over a matrix
state per head, behind a short causal convolution of q, k and v).  Feed-forwards: down relu(up x)^2, or experts chosen by
the largest sigmoid scores, each fed its input times its score.
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
    out = y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps)
    return out if w is None else out * w


def ln(y, w, b, eps):
    c = y - y.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def rotate(t, positions, dims: int, base: float, slowdown: float = 1.0):
    """t: [n, heads, e]; of every head, element i < dims/2 and element i + dims/2 turn by position * f_i,
    f_i = base^(-2i/dims) / slowdown; the elements from `dims` on pass."""
    out = t.clone()
    half = dims // 2
    for i in range(half):
        f = base ** (-2.0 * i / dims) / slowdown
        a = torch.tensor([float(p) * f for p in positions], dtype=F64)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = t[:, :, i], t[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def sink_attention(q, k, v, scale: float, sink):
    """q: [n, H, e], k: [n, G, e], v: [n, G, ev], sink: [H]; query head h reads key/value head h // (H / G), query i sees
    the keys j <= i, and exp(sink_h) joins the softmax's denominator.  Returns [n, H, ev]."""
    n, H, _ = q.shape
    group = H // k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    hidden = torch.ones(n, n, dtype=torch.bool).triu(1)
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T) * scale
        s[hidden] = -math.inf
        m = torch.maximum(s.amax(dim=1), sink[h])
        e = torch.exp(s - m[:, None])
        out[:, h] = (e @ v[:, h // group]) / (e.sum(dim=1) + torch.exp(sink[h] - m))[:, None]
    return out


def attention(x, w, p, mx, eps, first_values=None, positions=None, rnd=_same):
    """(update, values): values [n, G, ev] are what this layer attends over.  first_values: the values of the first layer
    that mixes values (None: this is that layer, or it does not mix)."""
    n = x.shape[0]
    H, G, e, ev = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    positions = list(range(n)) if positions is None else positions
    q = rms((x @ w[p + "q"].T).view(n, H, e), w[p + "q.norm"], eps)
    k = rms((x @ w[p + "k"].T).view(n, G, e), w[p + "k.norm"], eps)
    v = (x @ w[p + "v"].T).view(n, G, ev)
    rot = mx.get("rot")
    if rot is not None and rot.get("dims", 0) > 0:
        slow = float((rot.get("scaling") or {}).get("factor", 1.0))
        q = rotate(q, positions, rot["dims"], float(rot["base"]), slow)
        k = rotate(k, positions, rot["dims"], float(rot["base"]), slow)
    if mx.get("v_mix") and first_values is not None:
        lam = w[p + "vmix"].reshape(())
        v = (1.0 - lam) * v + lam * first_values
    v = rnd(v)
    o = sink_attention(rnd(q), rnd(k), v, float(mx["scale"]), w[p + "sink"])
    return rnd(o.reshape(n, H * ev)) @ w[p + "o"].T, v


def latent_attention(x, w, p, mx, eps, rnd=_same):
    n = x.shape[0]
    H, e, ev = mx["heads"], mx["dim"], mx["vdim"]
    q = rnd(x @ w[p + "q"].T).view(n, H, e)
    c = rnd(rms(x @ w[p + "dkv"].T, w[p + "dkv.norm"], eps))
    k = (c @ w[p + "uk"].T).view(n, H, e)
    v = (c @ w[p + "uv"].T).view(n, H, ev)
    o = sink_attention(q, k, v, float(mx["scale"]), w[p + "sink"])
    gate = torch.sigmoid(x @ w[p + "g"].T)                       # [n, H]
    return rnd((o * gate[:, :, None]).reshape(n, H * ev)) @ w[p + "o"].T


def causal_conv(x, w, before=None):
    """out[t, c] = sum_j w[c, j] x[t - (taps - 1 - j), c]; before: the taps - 1 rows before the first (None: zeros)."""
    taps = w.shape[1]
    pad = torch.zeros(taps - 1, x.shape[1], dtype=F64) if before is None else before
    xx = torch.cat([pad, x], dim=0)
    return sum(xx[j:j + x.shape[0]] * w[:, j] for j in range(taps))


def unit(y):
    return y / torch.sqrt((y * y).sum(dim=-1, keepdim=True) + 1e-6)


def delta_walk(q, k, v, beta, decay, state=None):
    """q, k: [n, H, e], v: [n, H, ev], beta, decay: [n, H]; state: None (a sequence from its start) or H matrices [e, ev]
    that are updated in place.  Per head and token: forget, write what the state gets wrong about k, read with q."""
    n, H, e = q.shape
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for h in range(H):
        S = torch.zeros(e, v.shape[2], dtype=F64) if state is None else state[h]
        for t in range(n):
            S = decay[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + torch.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
        if state is not None:
            state[h] = S
    return out


def delta(x, w, p, mx, eps, rnd=_same):
    n = x.shape[0]
    H, G, e, ev = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(x @ w[p + s].T, w[p + s + ".conv"])) for s in ("q", "k", "v"))
    spread = lambda t: t.view(n, G, e).repeat_interleave(H // G, dim=1)  # noqa: E731   (head h uses head h // (H / G))
    q, k, v = unit(spread(q)) * float(e) ** -0.5, unit(spread(k)), v.view(n, H, ev)
    beta = torch.sigmoid(x @ w[p + "b"].T)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(x @ w[p + "a"].T + w[p + "dt_bias"]))
    o = rms(delta_walk(q, k, v, beta, decay), w[p + "norm"], eps)
    return rnd(o.reshape(n, H * ev) * silu(x @ w[p + "g"].T)) @ w[p + "o"].T


def relu2_mlp(x, up, down, rnd=_same):
    return rnd(torch.relu(x @ up.T) ** 2) @ down.T


def route(x, w_router, router: dict, swapped=()):
    """Per token the chosen (expert, weight) pairs, best first.  swapped: tokens for which the last choice and the best
    expert that is not chosen change places (a close call taken the other way)."""
    s, top, out = torch.sigmoid(x @ w_router.T), router["top"], []
    for t, row in enumerate(s):
        order = sorted(range(router["experts"]), key=lambda e: (-float(row[e]), e))
        if t in swapped:
            order[top - 1], order[top] = order[top], order[top - 1]
        out.append([(e, float(row[e])) for e in order[:top]])
    return out


def route_gaps(x, w_router, router: dict):
    """Per token how far the last choice's logit lies above the best one that is not chosen (None: all are chosen)."""
    if router["top"] == router["experts"]:
        return None
    z = torch.sort(x @ w_router.T, dim=1, descending=True).values
    return z[:, router["top"] - 1] - z[:, router["top"]]


def expert_mlp(x, w, p, mlp, rnd=_same, swapped=()):
    out = torch.zeros_like(x)
    for t, picks in enumerate(route(x, w[p + "router"], mlp["router"], swapped)):
        for e, wt in picks:
            h = rnd(wt * x[t])
            a = silu(w[f"{p}e{e}.gate"] @ h) * (w[f"{p}e{e}.up"] @ h)
            out[t] += w[f"{p}e{e}.down"] @ rnd(a)
    return out


def forward(config: dict, weights: dict, tokens, return_layers: bool = False, rnd=_same, swapped=(), gaps=None):
    """Logits [n, vocab] of a whole sequence (and the residual stream after every layer).  rnd: applied to what a
    16-bit engine would store in 16 bits (what a matrix product reads, cached rows); the identity by default.  swapped:
    (layer, token) pairs whose router takes its closest call the other way; gaps: a dict that takes the routers' gaps by layer."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    streams, first_values = [], None
    for i, layer in enumerate(config["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        h = rnd(x)
        if layer["type"] == "attention":
            upd, values = attention(h, w, p + "mix.", mx, eps, first_values, rnd=rnd)
            if mx.get("v_mix") and first_values is None:
                first_values = values
        elif layer["type"] == "latent_attention":
            upd = latent_attention(h, w, p + "mix.", mx, eps, rnd=rnd)
        elif layer["type"] == "delta":
            upd = delta(h, w, p + "mix.", mx, eps, rnd=rnd)
        else:
            raise ValueError(f"layer {i}: unknown type {layer['type']!r}")
        x = x + w[p + "ls1"] * ln(upd, w[p + "norm1"], w[p + "norm1.b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rnd(x)
            if mlp["kind"] == "moe" and gaps is not None:
                gaps[i] = route_gaps(h, w[p + "mlp.router"], mlp["router"])
            upd = (expert_mlp(h, w, p + "mlp.", mlp, rnd, [t for n, t in swapped if n == i]) if mlp["kind"] == "moe"
                   else relu2_mlp(h, w[p + "mlp.up"], w[p + "mlp.down"], rnd))
            x = x + w[p + "ls2"] * ln(upd, w[p + "norm2"], w[p + "norm2.b"], eps)
        streams.append(x.clone())
    logits = rnd(ln(x, w["final.norm"], w["final.norm.b"], eps)) @ w["head"].T
    return (logits, torch.stack(streams)) if return_layers else logits
