"""Norms, fused with the residual add that precedes them: RMSNorm (of one residual stream or of several), layer norm, and
none (the add alone)."""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Biased, Combined, Norm, Normed, ParamSpec, Several, Streamed, register_part


def terms_of(update) -> list:
    """The `ops.Term`s whose sum an update is."""
    if isinstance(update, Combined):
        return list(update)
    if isinstance(update, Several):
        return [ops.Term(u) for u in update if u is not None]
    if isinstance(update, Biased) and torch.is_tensor(update.update):
        return [ops.Term(update.update, bias=update.bias)]
    if torch.is_tensor(update):
        return [ops.Term(update)]
    raise TypeError(f"an update of type {type(update).__name__} cannot be summed term by term")


def add_terms(rt, x, delta, out, rows=None, weight=None, eps: float = 0.0, bias=None, center: bool = False) -> None:
    """x += `delta` (None, a tensor, `Several`, `Combined`, or one of them as `Normed`), then out = norm(x), or x converted
    without a weight (out None: the add alone); one kernel."""
    own = delta if isinstance(delta, Normed) else None
    update = own.update if own is not None else delta
    terms = [] if update is None else terms_of(update)
    ops.combine_add(x, terms, own.weight if own is not None else None, own.eps if own is not None else 0.0, weight, eps, out,
                    rows, post_bias=own.bias if own is not None else None, post_center=own is not None and own.center,
                    next_bias=bias, next_center=center)


@register_part("norm", "rmsnorm")
class RMSNorm(Norm):
    """o = w * (x / sqrt(mean(x^2) + eps)), in 32-bit (infer/ops.odin:7-19).

    groups > 1: the row is cut into that many equal consecutive parts and each part is divided
    by its own root mean square; the weight still spans the whole row.
    one_plus: the stored weight lies around zero and the factor is 1 + w (the sum is formed once at load,
    in 32-bit, and kept so)."""

    graph_safe = True
    takes_bias = True
    takes_several = True
    takes_scale = True
    takes_terms = True

    def __init__(self, width: int, eps: float, weight: str, groups: int = 1, one_plus: bool = False):
        if groups < 1 or width % groups:
            raise ValueError(f"a norm over {width} elements cannot be cut into {groups} equal groups")
        self.width, self.eps, self.weight_name, self.groups = width, float(eps), weight, int(groups)
        self.one_plus = bool(one_plus)
        self.weight: torch.Tensor | None = None

    def params(self):
        return [ParamSpec(self.weight_name, (self.width,), init="near_zero" if self.one_plus else "norm")]

    def bind(self, tensors, rt):
        self.weight = tensors[self.weight_name]
        if self.one_plus:
            self.weight = (self.weight.to(torch.float32) + 1.0).contiguous()

    def kernel_groups(self):
        return {"elementwise", "rowwise"}

    def as_update_norm(self, update):
        return Normed(update, self.weight, self.eps)

    @property
    def can_norm_updates(self) -> bool:
        return self.groups == 1

    def pairs_with(self, other) -> bool:
        """Whether `other` norms the same row by the same root mean square (another weight only), so that one kernel
        can write both outputs."""
        return (type(other) is type(self) and other.width == self.width and other.eps == self.eps
                and other.groups == self.groups)

    def forward(self, rt, x, delta, rows=None, bias=None, scale: float = 1.0, second=None):
        """second: a norm that `pairs_with` this one; both outputs of the one updated row come back, (out, out2)."""
        n = x.shape[0] if rows is None else rows.numel()
        out = rt.empty(n, self.width)
        if isinstance(delta, (Normed, Combined)):
            # a sum of terms, a norm of the update's own, the add and this norm: one kernel
            if self.groups != 1 or bias is not None or scale != 1.0 or second is not None:
                raise TypeError("an update of several terms or with a norm of its own meets a plain RMSNorm only")
            add_terms(rt, x, delta, out, rows, self.weight, self.eps)
            return out
        if isinstance(delta, (list, tuple)) and len(delta) == 1:
            delta = delta[0]
        if delta is None and bias is None:
            scale = 1.0
        if second is not None:
            out2 = rt.empty(n, self.width)
            ops.row_update(x, delta, bias, self.weight, self.eps, self.groups, out, rows, scale=scale,
                           weight2=second.weight, out2=out2)
            return out, out2
        if self.groups == 1 and bias is None and scale == 1.0 and not isinstance(delta, (list, tuple)):
            ops.add_rmsnorm(x, delta, self.weight, self.eps, out, rows)
        else:
            ops.row_update(x, delta, bias, self.weight, self.eps, self.groups, out, rows, scale=scale)
        return out

    def in_place(self, rt, x) -> None:
        """x (32-bit) <- its own norm."""
        ops.row_update(x, None, None, self.weight, self.eps, self.groups, x)


@register_part("norm", "streams_rmsnorm")
class StreamsRMSNorm(Norm):
    """Reads a residual of several streams: o = w * u / sqrt(mean(u^2) + eps) of u = sum_i read[i] X[i], in 32-bit.

    x is [streams, n, width]; a pending `Streamed` update is applied to the streams first, and the sum, the norm and that
    update are one kernel.  read: name of a vector [streams] (None: the plain sum of the streams).  one_plus: as RMSNorm."""

    graph_safe = True
    takes_streams = True

    def __init__(self, width: int, eps: float, weight: str, streams: int, read: str | None = None, one_plus: bool = False):
        if not 1 <= streams <= ops.MAX_STREAMS:
            raise ValueError(f"a residual has 1 to {ops.MAX_STREAMS} streams, got {streams}")
        self.width, self.eps, self.weight_name, self.streams = width, float(eps), weight, int(streams)
        self.read_name, self.one_plus = read, bool(one_plus)
        self.weight = self.read = None

    def params(self):
        out = [ParamSpec(self.weight_name, (self.width,), init="near_zero" if self.one_plus else "norm")]
        if self.read_name is not None:
            out.append(ParamSpec(self.read_name, (self.streams,), init="unit"))
        return out

    def bind(self, tensors, rt):
        self.weight = tensors[self.weight_name]
        if self.one_plus:
            self.weight = (self.weight.to(torch.float32) + 1.0).contiguous()
        if self.read_name is not None:
            self.read = tensors[self.read_name].to(torch.float32).contiguous()
        else:
            self.read = torch.ones(self.streams, dtype=torch.float32, device=rt.device)

    def kernel_groups(self):
        return {"streams"}

    def forward(self, rt, x, delta, rows=None):
        if delta is not None and not isinstance(delta, Streamed):
            raise TypeError(f"a residual of several streams takes updates through a connection, not {type(delta).__name__}")
        n = x.shape[1] if rows is None else rows.numel()
        out = rt.empty(n, self.width)
        terms, mix, add = ([], None, None) if delta is None else (terms_of(delta.update), delta.mix, delta.out)
        ops.mix_streams(x, terms, mix, add, self.read, self.weight, self.eps, out, rows)
        return out


@register_part("norm", "layernorm")
class LayerNorm(Norm):
    """o = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w + b, in 32-bit.

    scale: name of a vector that multiplies the result element by element (a learned scale on a sublayer's output); it is
    multiplied into w and b once, at load, in 32-bit."""

    graph_safe = True
    takes_several = True
    takes_terms = True
    can_norm_updates = True

    def __init__(self, width: int, eps: float, weight: str, bias: str, scale: str | None = None):
        self.width, self.eps, self.weight_name, self.bias_name, self.scale_name = width, float(eps), weight, bias, scale
        self.weight = self.bias = None

    def params(self):
        out = [ParamSpec(self.weight_name, (self.width,), init="norm"), ParamSpec(self.bias_name, (self.width,), init="near_zero")]
        if self.scale_name is not None:
            out.append(ParamSpec(self.scale_name, (self.width,), init="unit"))
        return out

    def bind(self, tensors, rt):
        w, b = (tensors[n].to(torch.float32) for n in (self.weight_name, self.bias_name))
        if self.scale_name is not None:
            s = tensors[self.scale_name].to(torch.float32)
            w, b = w * s, b * s
        self.weight, self.bias = w.contiguous(), b.contiguous()

    def kernel_groups(self):
        return {"rowwise"}

    def as_update_norm(self, update):
        return Normed(update, self.weight, self.eps, self.bias, True)

    def forward(self, rt, x, delta, rows=None):
        n = x.shape[0] if rows is None else rows.numel()
        out = rt.empty(n, self.width)
        add_terms(rt, x, Several(delta) if isinstance(delta, list) and not isinstance(delta, (Several, Combined)) else delta,
                  out, rows, self.weight, self.eps, self.bias, True)
        return out


@register_part("norm", "none")
class NoNorm(Norm):
    """Adds what is pending to the residual stream and hands the stream on as it is, in the element type of activations (the
    stream itself in the 32-bit engine): for sublayers that read the stream without a norm."""

    graph_safe = True
    takes_bias = True
    takes_several = True
    takes_terms = True

    def __init__(self, width: int):
        self.width = width

    def kernel_groups(self):
        return {"rowwise"}

    def forward(self, rt, x, delta, rows=None, bias=None):
        if rows is not None:
            raise TypeError("this part hands on whole streams, no gathered rows")
        if isinstance(delta, (Normed, Combined)):
            out = None if rt.dtype == torch.float32 else rt.empty(x.shape[0], self.width)
            add_terms(rt, x, delta, out)
            return x if out is None else out
        return rt.settle(x, delta, bias)
