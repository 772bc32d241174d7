"""The matrix memory of xLSTM (Beck et al., "xLSTM: Extended Long Short-Term
Memory"): a matrix per head with an exponential input gate, divided by what a
normalizer remembers of the keys.

Per head, with the raw numbers of the two gates cut off softly at +-cap (c(z) = cap tanh(z / cap)):

  a = c(z_in),  b = log sigmoid(c(z_forget))         logarithms of what a token brings and of what is kept
  m' = max(m + b, a)                                 m = 0 where a sequence begins
  [S | n] <- e^(m + b - m') [S | n] + e^(a - m') k [v | 1]^T
  [y | y_n] = q^T [S | n],  out = y / (max(|y_n|, e^(-m')) + 1e-6)

so that S and n hold their sums over all tokens divided by e^m and stay in range.  The heads' outputs, each divided by its
root mean square, are multiplied with a weight of all heads' size and the sigmoid of a gate before the output product.

All first products are one, with 32-bit rows: everything from there to the
rounding before the output product is 32-bit, and q's factor is applied where
the division is.  Steps of single tokens run gates and recurrence as one
kernel; portions run the gates first (m is a scan of maxima) and then the
recurrence token by token, or in chunks of 64 tokens side by side once a
portion is long.  Between steps a request keeps, in its state slot and in
32-bit, S of every head transposed with n behind it, [dv + 1, d], and m.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache.manager import StateNeed
from ..weights.loader import TensorSpec
from .base import Mixer
from .registry import register_mixer


class MLSTM(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``head_dim``, ``v_dim``, ``gate_cap``, ``eps`` (of the heads' norm),
    ``q_scale`` (None: head_dim^-1/2), ``base`` (what the tensor names start with after the prefix, default "mix."; the
    tensors are q, k, v, g, i, i.b, f, f.b, norm [heads * v_dim], o)."""

    @classmethod
    def _base(cls, p, prefix):
        return prefix + (p.get("base") if p.get("base") is not None else "mix.")

    @classmethod
    def tensor_specs(cls, p, prefix):
        W, H, d, dv = p["hidden_size"], p["num_heads"], p["head_dim"], p["v_dim"]
        b = cls._base(p, prefix)
        return {b + "q": TensorSpec((H * d, W)), b + "k": TensorSpec((H * d, W)), b + "v": TensorSpec((H * dv, W)),
                b + "g": TensorSpec((H * dv, W)), b + "i": TensorSpec((H, W)), b + "i.b": TensorSpec((H,)),
                b + "f": TensorSpec((H, W)), b + "f.b": TensorSpec((H,)), b + "norm": TensorSpec((H * dv,), init="norm"),
                b + "o": TensorSpec((W, H * dv))}

    @classmethod
    def cache_need(cls, p):
        H, d, dv = int(p["num_heads"]), int(p["head_dim"]), int(p["v_dim"])
        return (StateNeed((H, dv + 1, d), "float32"), StateNeed((H,), "float32"))          # S transposed and n; m

    def __init__(self, p, prefix, env, tensors):
        super().__init__(p, prefix, env, tensors)
        self.H, self.d, self.dv = int(p["num_heads"]), int(p["head_dim"]), int(p["v_dim"])
        self.cap, self.eps = float(p["gate_cap"]), float(p.get("eps") or 0.0)
        if not self.cap > 0.0:
            raise ValueError(f"gate_cap {self.cap} must be positive")
        self.q_scale = float(p["q_scale"]) if p.get("q_scale") is not None else float(self.d) ** -0.5
        b = self._base(p, prefix)
        names = [b + n for n in ("q", "k", "v", "g", "i", "f")]
        self.w_in = ops.pad_rows(torch.cat([tensors.get(n, env.dtype) for n in names], dim=0))
        tensors.drop(*names)
        f32 = lambda n: tensors.get(b + n, torch.float32).contiguous()
        self.ib, self.fb, self.norm = f32("i.b"), f32("f.b"), f32("norm")
        self.w_o = tensors.get(b + "o", env.dtype)

    def forward(self, x, batch, cache, writes=True):
        H, d, dv = self.H, self.d, self.dv
        state, m = cache.parts[0].state, cache.parts[1].state
        proj = ops.linear(x, self.w_in, out_dtype=torch.float32)             # [T, q | k | v | gate | i | f | padding]
        if batch.decode_only:
            o, m_rows = ops.mlstm_step(proj, self.ib, self.fb, self.cap, state, m, batch, H, d, dv), None
        else:
            o, m_rows = ops.mlstm_scan(proj, self.ib, self.fb, self.cap, state, m, batch, H, d, dv)
        z = ops.mlstm_out(o, proj, self.norm, self.eps, self.q_scale, m_rows, self.ib, self.fb, self.cap, m, batch, H, d, dv,
                          self.env.dtype)
        return ops.linear(z, self.w_o)


register_mixer("mlstm", MLSTM)
