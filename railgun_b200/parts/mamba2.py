"""The mixer of Mamba-2 (Dao and Gu, "Transformers are SSMs: Generalized Models
and Efficient Algorithms Through Structured State Space Duality").

One product gives z, x [heads, dv], B and C [groups, N] and a raw step size
per head.  x, B and C pass a short causal convolution per channel (with a
bias) and silu; with dt = softplus(raw + bias) and head h reading group
h / (heads / groups):
  S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D_h x_t
  out = W_o (group_norm(y * silu(z)) * weight)
where group_norm divides each of ``norm_groups`` equal parts by its own root
mean square.

Steps of single tokens run the convolution, the step sizes and the
recurrence as one kernel from 32-bit rows; portions run the convolution, the
step sizes and the recurrence one after the other (token by token, or in
chunks of 64 tokens side by side once a portion is long), the wide part of
the product in the model's type and the step sizes' columns in 32-bit.  Between steps a request keeps, in its state slot and in 32-bit, S of
every head (transposed, [dv, N]) and the convolution's last taps - 1 inputs.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache.manager import StateNeed
from ..weights.loader import TensorSpec
from .base import Mixer
from .registry import register_mixer


class Mamba2(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``v_dim``, ``state`` (N), ``groups`` (of B and C), ``taps``,
    ``norm_groups``, ``eps`` (of the norm), ``base`` (what the tensor names start with after the prefix, default
    "mix."; the tensors are in, conv, conv.b, dt_bias, A_log, D, norm, o)."""

    # up to this many rows the whole first product comes out in 32-bit (its columns are few bytes beside its matrix)
    ROWS32 = 64

    @classmethod
    def _base(cls, p, prefix):
        return prefix + (p.get("base") if p.get("base") is not None else "mix.")

    @classmethod
    def tensor_specs(cls, p, prefix):
        W, H, dv, N, G, K = (p["hidden_size"], p["num_heads"], p["v_dim"], p["state"], p["groups"], p["taps"])
        inner, b = H * dv, cls._base(p, prefix)
        C = inner + 2 * G * N
        return {b + "in": TensorSpec((inner + C + H, W)), b + "conv": TensorSpec((C, K)), b + "conv.b": TensorSpec((C,)),
                b + "dt_bias": TensorSpec((H,)), b + "A_log": TensorSpec((H,)), b + "D": TensorSpec((H,), init="norm"),
                b + "norm": TensorSpec((inner,), init="norm"), b + "o": TensorSpec((W, inner))}

    @classmethod
    def cache_need(cls, p):
        H, dv, N, G, K = int(p["num_heads"]), int(p["v_dim"]), int(p["state"]), int(p["groups"]), int(p["taps"])
        need = [StateNeed((H, dv, N), "float32")]                                # S transposed
        if K > 1:
            need.append(StateNeed((K - 1, H * dv + 2 * G * N), "float32"))
        return tuple(need)

    def __init__(self, p, prefix, env, tensors):
        super().__init__(p, prefix, env, tensors)
        self.H, self.dv, self.N, self.G, self.K = (int(p["num_heads"]), int(p["v_dim"]), int(p["state"]),
                                                   int(p["groups"]), int(p["taps"]))
        self.norm_groups, self.eps = int(p.get("norm_groups") or 1), float(p.get("eps") or 0.0)
        self.inner = self.H * self.dv
        self.C = self.inner + 2 * self.G * self.N
        if self.H % self.G or self.inner % self.norm_groups:
            raise ValueError(f"{self.H} heads cannot share {self.G} groups, or {self.inner} numbers do not split into "
                             f"{self.norm_groups} equal parts")
        if self.N > 256:
            raise ValueError(f"a state of {self.N} rows is above the scan's limit of 256")
        b = self._base(p, prefix)
        f32 = lambda n: tensors.get(b + n, torch.float32).contiguous()
        self.w_in = tensors.get(b + "in", env.dtype).contiguous()
        self.taps = tensors.get(b + "conv", torch.float32).t().contiguous()      # [taps, channels]
        self.conv_bias, self.dt_bias, self.A_log = f32("conv.b"), f32("dt_bias"), f32("A_log")
        self.D, self.norm = f32("D"), f32("norm")
        self.w_o = tensors.get(b + "o", env.dtype)

    def forward(self, x, batch, cache, writes=True):
        H, dv, N, G, inner, C = self.H, self.dv, self.N, self.G, self.inner, self.C
        state = cache.parts[0].state
        conv_state = cache.parts[1].state if self.K > 1 else None
        if batch.decode_only or x.shape[0] <= self.ROWS32 or self.env.dtype == torch.float32:
            proj = ops.linear(x, self.w_in, out_dtype=torch.float32)             # [T, z | x | B | C | raw dt]
            raw_dt = proj[:, inner + C:]
        else:
            proj = ops.linear(x, self.w_in[:inner + C])
            raw_dt = ops.linear(x, self.w_in[inner + C:], out_dtype=torch.float32)
        z = proj[:, :inner]
        if batch.decode_only:
            o = ops.ssd_step(proj, inner, inner + C, self.taps, self.conv_bias, conv_state, self.dt_bias, self.A_log,
                             self.D, state, batch, H, G, N, dv)
            conv = (proj[:, inner:inner + C], conv_state) if self.K > 1 else None
            y = ops.gate_group_norm(o, z, self.norm, self.eps, self.norm_groups, self.env.dtype, conv=conv, batch=batch)
            return ops.linear(y, self.w_o)
        xbc = ops.causal_conv(proj, inner, self.taps, conv_state, batch, torch.float32, silu=True, bias=self.conv_bias)
        if writes and conv_state is not None:
            ops.conv_state_update(proj, inner, conv_state, batch)
        dt, g = ops.ssd_prepare(raw_dt, self.dt_bias, self.A_log)
        if batch.max_query_len >= ops.SCAN_CHUNKED_MIN_TOKENS:
            o = ops.ssd_chunk_scan(xbc, dt, self.A_log, self.D, state, batch, H, G, N, dv)
        else:
            o = ops.state_scan(xbc[:, inner + G * N:], xbc[:, inner:inner + G * N], xbc[:, :inner], state, batch, H, N, dv,
                               g=g, beta=dt, rule="scalar", skip=self.D)
        y = ops.gate_group_norm(o, z, self.norm, self.eps, self.norm_groups, self.env.dtype)
        return ops.linear(y, self.w_o)


register_mixer("mamba2", Mamba2)
