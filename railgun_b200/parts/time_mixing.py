"""Mixing a token with the token before it: the token shift in front of a
mixer, and RWKV-style time mixing.

"token_shift": a wrapper.  The inner mixer reads h + (h' - h) shift instead of
h, element by element, h' being the request's previous token's h (zeros
before the first).

"rwkv": linear attention with a decay per token and key channel.  With h' as
above, each of r, k, v, g and w reads a mix h + (h' - h) mu_s of its own:
  r, k, v = W_r ., W_k ., W_v .  [heads, d];   gate = silu(W_g .)
  w = exp(-exp(W_w2 tanh(W_w1 .) + w0))        per head and key channel
  o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t;   S_t = diag(w_t) S_(t-1) + k_t v_t^T
  out = W_o (unit_rms(o_t) per head * norm * gate)
The four wide products are one batched library product into 32-bit rows.  The
recurrence runs token by token, or in chunks of 64 tokens side by side once a
portion is long.  The
decay is 32-bit from its mix on: in bfloat16 mode the mix enters its product
as two bfloat16 numbers (hi + lo to 2^-17) against the matrix stacked twice,
accumulated in 32-bit.

Between steps a request keeps, in its state slot and in 32-bit: the last
token's h (of each of the two), and S of every head (transposed, [d, d]).
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache.manager import StateNeed
from ..weights.loader import AnySize, TensorSpec
from .base import CacheView, Mixer
from .registry import MIXERS, register_mixer


class TokenShift(Mixer):
    """params: ``hidden_size``, ``name`` (the shares' tensor after the prefix, [hidden_size]), ``inner`` (the PartSpec
    of the mixer that reads the shifted rows)."""

    takes_stream = True

    @classmethod
    def tensor_specs(cls, p, prefix):
        inner = p["inner"]
        out = dict(MIXERS.get(inner.kind).tensor_specs(inner.params, prefix))
        out[prefix + p["name"]] = TensorSpec((p["hidden_size"],))
        return out

    @classmethod
    def _inner_needs(cls, p):
        inner = p["inner"]
        need = MIXERS.get(inner.kind).cache_need(inner.params)
        return (tuple(need), True) if isinstance(need, (tuple, list)) else ((need,), False)

    @classmethod
    def cache_need(cls, p):
        return (StateNeed((1, int(p["hidden_size"])), "float32"),) + cls._inner_needs(p)[0]

    def __init__(self, p, prefix, env, tensors):
        super().__init__(p, prefix, env, tensors)
        inner = p["inner"]
        self.inner = MIXERS.get(inner.kind)(inner.params, prefix, env, tensors)
        self.inner_composite = self._inner_needs(p)[1]
        self.share = tensors.get(prefix + p["name"], torch.float32).contiguous()
        self.graph_safe = getattr(self.inner, "graph_safe", True)

    def _inner_view(self, cache):
        return CacheView(cache.cache_id, parts=cache.parts[1:]) if self.inner_composite else cache.parts[1]

    def forward(self, x, batch, cache, writes=True):
        # rows that come from a norm: the shift is a convolution of two taps
        taps = torch.stack([self.share, 1.0 - self.share])
        h = ops.causal_conv(x, 0, taps, cache.parts[0].state, batch, self.env.dtype)
        if writes:
            ops.conv_state_update(x, 0, cache.parts[0].state, batch)
        return self.inner.forward(h, batch, self._inner_view(cache), writes)

    def forward_stream(self, stream, batch, cache, writes=True):
        """The same behind the stream itself: what is pending is added to it in the same kernel."""
        pending = stream.pending
        if isinstance(pending, (ops.PendingLinear, ops.PendingSum)):
            pending = pending.materialize()
        stream.resid, h = ops.postnorm_shift(stream.resid, pending, self.share, cache.parts[0].state, batch,
                                             self.env.dtype)
        stream.pending = None
        return self.inner.forward(h, batch, self._inner_view(cache), writes)


class RwkvTimeMixing(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``head_dim`` (of keys and values alike), ``eps`` (of the heads' norm),
    ``base`` (what the tensor names start with after the prefix, default "mix."; the tensors are mu.r, mu.k, mu.v,
    mu.g, mu.w, r, k, v, g, w1 [rank, hidden_size], w2 [heads * head_dim, rank], w0, u [heads, head_dim], norm, o).
    The rank is whatever the files have."""

    DEFAULT_RANK = 64

    @classmethod
    def _base(cls, p, prefix):
        return prefix + (p.get("base") if p.get("base") is not None else "mix.")

    @classmethod
    def tensor_specs(cls, p, prefix):
        W, H, d = p["hidden_size"], p["num_heads"], p["head_dim"]
        b, n, rank = cls._base(p, prefix), p["num_heads"] * p["head_dim"], AnySize(cls.DEFAULT_RANK)
        out = {b + "mu." + s: TensorSpec((W,)) for s in "rkvgw"}
        out.update({b + s: TensorSpec((n, W)) for s in "rkvg"})
        out.update({b + "w1": TensorSpec((rank, W)), b + "w2": TensorSpec((n, rank)), b + "w0": TensorSpec((n,)),
                    b + "u": TensorSpec((H, d)), b + "norm": TensorSpec((n,), init="norm"), b + "o": TensorSpec((W, n))})
        return out

    @classmethod
    def cache_need(cls, p):
        H, d = int(p["num_heads"]), int(p["head_dim"])
        return (StateNeed((H, d, d), "float32"), StateNeed((1, int(p["hidden_size"])), "float32"))

    def __init__(self, p, prefix, env, tensors):
        super().__init__(p, prefix, env, tensors)
        self.H, self.d, self.eps = int(p["num_heads"]), int(p["head_dim"]), float(p.get("eps") or 0.0)
        if self.d > 256:
            raise ValueError(f"head size {self.d} is above the scan's limit of 256")
        b = self._base(p, prefix)
        f32 = lambda n: tensors.get(b + n, torch.float32).contiguous()
        self.mu = torch.stack([f32("mu." + s) for s in "rkvgw"]).contiguous()
        self.w_rkvg = torch.stack([tensors.get(b + s, env.dtype) for s in "rkvg"]).contiguous()     # [4, H d, W]
        tensors.drop(*(b + s for s in "rkvg"))
        w1 = tensors.get(b + "w1", env.dtype)
        self.w2 = tensors.get(b + "w2", env.dtype).contiguous()
        if self.w2.shape[1] != w1.shape[0]:
            raise ValueError(f"{b}w1 has {w1.shape[0]} rows, {b}w2 {self.w2.shape[1]} columns")
        # for bfloat16 the mix comes as hi | lo: the matrix stands twice side by side
        self.w1 = (torch.cat([w1, w1], dim=1) if env.dtype == torch.bfloat16 else w1).contiguous()
        self.w0, self.u, self.norm = f32("w0"), f32("u"), f32("norm")
        self.w_o = tensors.get(b + "o", env.dtype)
        self.out_features = self.H * self.d

    w_in = None                     # as a branch of "parallel": its products read mixes of x

    def mix(self, x, batch, cache, writes=True, out=None, out_scale: float = 1.0, proj=None):
        """The gated heads [T, heads * head_dim] times ``out_scale`` (into ``out`` if given), before the output
        product.  The state advances by the step's tokens."""
        H, d = self.H, self.d
        mixes, last = ops.shift_mixes(x, self.mu, cache.parts[1].state, batch)
        wide = self.w_rkvg.transpose(1, 2)
        if mixes.dtype == torch.float32:
            r, k, v, g = torch.bmm(mixes, wide)
        else:
            r, k, v, g = torch.bmm(mixes, wide, out_dtype=torch.float32)
        w = ops.lowrank_decay(ops.linear(last, self.w1, out_dtype=torch.float32), self.w2, self.w0)
        if batch.max_query_len >= ops.SCAN_CHUNKED_MIN_TOKENS:
            o = ops.channel_chunk_scan(r, k, v, w, self.u, cache.parts[0].state, batch, H, d, d)
        else:
            o = ops.state_scan(r, k, v, cache.parts[0].state, batch, H, d, d, rule="channel", w=w, bonus=self.u)
        return ops.head_norm_gate(o, g, self.norm, self.eps, self.env.dtype, out=out, out_scale=out_scale)

    def forward(self, x, batch, cache, writes=True):
        return ops.linear(self.mix(x, batch, cache, writes), self.w_o)


register_mixer("token_shift", TokenShift)
register_mixer("rwkv", RwkvTimeMixing)
