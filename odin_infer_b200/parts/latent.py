"""Attention whose keys and values come from one small latent per token."""
from __future__ import annotations

import torch

from ..cache import KVRequest
from ..csrc import ops
from .base import Mixer, ParamSpec, register_part


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    """Queries through a latent: c_q = RMSNorm(W_dq h) * w, q = W_uq c_q, or straight from the input, q = W_q h
    (q_rank 0); per head [head_dim unrotated | rot_dim rotated].  Keys and values through ONE latent per token: W_dkv h = [c' | k_r], c = RMSNorm(c') * w (kv_rank wide),
    k_r (rot_dim wide, not normed) rotated by the position and shared by all heads; per head k = [W_uk c | k_r],
    v = W_uv c.  score = (q . k) * scale over the visible keys (window > 0: the last `window`), softmax, W_o on the
    heads side by side.

    The cache keeps one row [c | rotated k_r] per token (`KVRequest.shared_kv`), never a key or a value per head.
    Every head's unrotated query is carried over to the latent instead, q' = W_uk^T q (q . (W_uk c) = q' . c), so that
    attention is one kv head of kv_rank + rot_dim elements under all query heads with the cached rows as keys AND as
    values; the kernels' output over the row's first kv_rank elements goes through W_uv head by head.  Prompts,
    portions of prompts and decoding run the same way, through whichever attention kernel takes the row's size.

    sink: name of a tensor [n_heads], a learned logit per head whose exponential joins the softmax's denominator (no key, no
    value, not scaled).  gate: name of a matrix G [n_heads, width]; head h's output is multiplied by sigmoid(G h)_h as it
    leaves W_uv; with gate_per_head=False G is [n_heads * v_head_dim, width] and every element has a factor of its own.

    names: "dq", "dq_norm", "uq" (q_rank 0: "q" instead), "dkv", "dkv_norm", "uk", "uv", "o".  All products that read the
    input (W_dq or W_q, W_dkv, G) are fused into one.
    The rotation's layout is the position encoding's (`pairs` or `halves`)."""

    graph_safe = True
    rope_layouts = ("halves", "pairs")

    def __init__(self, width: int, n_heads: int, head_dim: int, rot_dim: int, v_head_dim: int, q_rank: int, kv_rank: int,
                 names: dict, position_encoding: str | None, eps: float, scale: float, window: int = 0,
                 sink: str | None = None, gate: str | None = None, gate_per_head: bool = True):
        if min(width, n_heads, head_dim, v_head_dim, kv_rank) <= 0 or q_rank < 0 or rot_dim < 0 or rot_dim % 2:
            raise ValueError("latent attention needs positive sizes and an even rot_dim")
        if kv_rank + rot_dim > 1024:
            raise ValueError(f"latent attention: a cached row of kv_rank + rot_dim = {kv_rank + rot_dim} elements is more than "
                             "the attention kernels take (1024)")
        if rot_dim and position_encoding is None:
            raise ValueError("latent attention with a rotated part needs a position encoding")
        self.width, self.H, self.e, self.r, self.ev = width, n_heads, head_dim, rot_dim, v_head_dim
        self.q_rank, self.kv_rank, self.L = q_rank, kv_rank, kv_rank + rot_dim
        self.names, self.pe_name, self.eps = dict(names), position_encoding, float(eps)
        self.scale, self.window = float(scale), int(window)
        self.sink_name, self.gate_name, self.gate_per_head = sink, gate, bool(gate_per_head)
        self.n_first = q_rank or n_heads * (head_dim + rot_dim)   # columns of the fused product before the kv latent's
        self.pe = None
        self.sink = self.q_norm = self.w_uq = self._dummy = None

    def params(self):
        n, H = self.names, self.H
        if self.q_rank:
            out = [ParamSpec(n["dq"], (self.q_rank, self.width)), ParamSpec(n["dq_norm"], (self.q_rank,), init="norm"),
                   ParamSpec(n["uq"], (H * (self.e + self.r), self.q_rank))]
        else:
            out = [ParamSpec(n["q"], (H * (self.e + self.r), self.width))]
        out += [ParamSpec(n["dkv"], (self.L, self.width)), ParamSpec(n["dkv_norm"], (self.kv_rank,), init="norm"),
                ParamSpec(n["uk"], (H * self.e, self.kv_rank)), ParamSpec(n["uv"], (H * self.ev, self.kv_rank)),
                ParamSpec(n["o"], (self.width, H * self.ev))]
        if self.sink_name is not None:
            out.append(ParamSpec(self.sink_name, (H,), init="logit"))
        if self.gate_name is not None:
            out.append(ParamSpec(self.gate_name, (H if self.gate_per_head else H * self.ev, self.width)))
        return out

    def bind(self, tensors, rt):
        n, H = self.names, self.H
        mats = [tensors.pop(n["dq" if self.q_rank else "q"]), tensors.pop(n["dkv"])]
        if self.gate_name is not None:
            mats.append(tensors.pop(self.gate_name))
        if len({t.dtype for t in mats}) > 1:
            mats = [t.float() for t in mats]
        self.w_down = torch.cat(mats, dim=0).contiguous()
        self.c_norm, self.w_o = tensors[n["dkv_norm"]], tensors[n["o"]]
        if self.q_rank:
            self.q_norm, self.w_uq = tensors[n["dq_norm"]], tensors[n["uq"]]
            if self.q_norm.dtype != self.c_norm.dtype:
                self.q_norm, self.c_norm = self.q_norm.float(), self.c_norm.float()
        if self.sink_name is not None:
            self.sink = tensors[self.sink_name].to(torch.float32).contiguous()
        # per head, (input channel before output channel, output before input): W_uk of a head is stored the first way, W_uv
        # the second
        uk, uv = tensors.pop(n["uk"]).view(H, self.e, self.kv_rank), tensors.pop(n["uv"]).view(H, self.ev, self.kv_rank)
        self.w_uk = (uk.contiguous(), uk.transpose(1, 2).contiguous())
        self.w_uv = (uv.transpose(1, 2).contiguous(), uv.contiguous())
        self._dummy = torch.zeros(1, 1, dtype=torch.float32, device=rt.device)

    def cache_request(self):
        return KVRequest(1, self.L, self.window, 0, 0, shared_kv=True)

    def kernel_groups(self):
        return {"latent", "moe_tc", "attention_plain", "gemm_plain"}

    def notes(self, rt):
        if rt.dtype != torch.bfloat16:
            return []
        out = []
        if not ops.attention_prefill_supported(self.L):
            out.append(f"latent attention: a cached row of {self.L} elements (kv_rank + rot_dim) is not 64 or 128: prompts "
                       "run the CUDA-core attention kernel (one warp per token and head)")
        if self.L not in (64, 128) or self.H > 16:
            out.append(f"latent attention: {self.H} heads over rows of {self.L}: decoding runs a CUDA-core attention kernel "
                       "(the tensor-core one takes rows of 64 or 128 and up to 16 heads)")
        return out

    def forward(self, rt, step, h, entry):
        T, H, e, r, L = h.shape[0], self.H, self.e, self.r, self.L
        # a rotated part of q straight from this product cannot come as partial sums
        down = rt.linear(h, self.w_down, may_split=bool(self.q_rank or not r), beside_attention=True)
        line, _, block_table = step.kv(entry)
        rot = self.pe.rotation() if (self.pe is not None and r) else None
        cos, sin = (rot[0], rot[1]) if rot is not None else (self._dummy, self._dummy)
        pairs = rot is not None and self.pe.layout == "pairs"
        n0, n1 = self.n_first, self.n_first + L
        cq = rt.empty(T, self.q_rank) if self.q_rank else None
        ops.latent_prep(down[..., (0 if self.q_rank else n0):n1], self.q_rank, self.kv_rank, r, pairs, self.q_norm,
                        self.c_norm, self.eps, cq, cos, sin, step.tok_pos, step.tok_seq, block_table, line,
                        write_cache=step.writes_cache(entry))
        q = rt.linear(cq, self.w_uq) if self.q_rank else down[..., :n0]
        qf = rt.empty(T, H * L)
        rt.heads_linear(q, e + r, self.w_uk, qf, L)
        if r:
            ops.rope_heads(q[:, e:], e + r, qf[:, self.kv_rank:], L, H, r, r, pairs, cos, sin, step.tok_pos)
        o = rt.empty(T, H * L)
        rt.attention(step, qf, o, H, 1, L, line, line, block_table, self.window, scale=self.scale, sink=self.sink)
        ov = rt.empty(T, H * self.ev)
        rt.heads_linear(o, L, self.w_uv, ov, self.ev, gate=down[..., n1:] if self.gate_name is not None else None)
        return rt.linear(ov, self.w_o, out_dtype=torch.float32, may_split=True, beside_attention=True)
