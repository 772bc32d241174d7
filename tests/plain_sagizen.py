"""Sagizen, stated plainly: dense numpy in 64-bit, one function per mechanism,
whole sequences at once, token-by-token loops for the recurrences, no cache
and no kernels.  Shares nothing with the package; the tests hold the
package's steps to this.

Notation: T tokens, W width, weights are stored [out, in] and applied as
y = x @ w.T.  ``w`` maps tensor names to float64 arrays; ``cfg`` is the
config.json dictionary.
"""
from __future__ import annotations

import json
import struct

import numpy as np


def read_safetensors(path) -> dict:
    """name -> float64 array (integers stay integers)."""
    raw = open(path, "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    header = json.loads(raw[8:8 + n])
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        buf = raw[8 + n + lo:8 + n + hi]
        if meta["dtype"] == "BF16":
            a = (np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif meta["dtype"] == "F32":
            a = np.frombuffer(buf, dtype="<f4").astype(np.float64)
        elif meta["dtype"] == "I32":
            a = np.frombuffer(buf, dtype="<i4")
        else:
            raise ValueError(f"{name}: dtype {meta['dtype']}")
        out[name] = a.reshape(meta["shape"])
    return out


# ---- small pieces ---------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def previous(x):
    """Row t holds row t - 1; row 0 holds zeros."""
    return np.concatenate([np.zeros((1, x.shape[1])), x[:-1]], axis=0)


def token_shift(x, share):
    """x_t + (x_(t-1) - x_t) share, number by number."""
    return x + (previous(x) - x) * share


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K], last column for the current token: bias + sum_j taps[:, j] x_(t - K + 1 + j)."""
    T, C = x.shape
    K = taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, C)), x], axis=0)
    y = np.tile(np.asarray(bias, dtype=np.float64), (T, 1))
    for j in range(K):
        y += padded[j:j + T] * taps[:, j][None, :]
    return y


def rotate_half(x, pos, dims, base, factor=1.0):
    """x [T, heads, d]: numbers (i, i + dims / 2), i < dims / 2, of every head turn by pos base^(-2i / dims) / factor."""
    out = x.copy()
    n = dims // 2
    f = base ** (-2.0 * np.arange(n) / dims) / factor
    a = np.asarray(pos, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def pooled_window_attention(q, k, v, scale, size, pool):
    """q [T, H, d], k [T, G, d], v [T, G, dv].  Query i sees token j with 0 <= i - j < size, and block b of ``pool``
    tokens (the mean of its keys, the mean of its values) once the block's last token is at least ``size`` back;
    one softmax over both.  Returns [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    nb = T // pool
    kb = k[:nb * pool].reshape(nb, pool, G, k.shape[2]).mean(axis=1)
    vb = v[:nb * pool].reshape(nb, pool, G, v.shape[2]).mean(axis=1)
    i, j, b = np.arange(T)[:, None], np.arange(T)[None, :], np.arange(nb)[None, :]
    sees = np.concatenate([b * pool + pool - 1 <= i - size, (j <= i) & (i - j < size)], axis=1)       # [T, nb + T]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        keys, values = np.concatenate([kb[:, g], k[:, g]]), np.concatenate([vb[:, g], v[:, g]])
        s = np.where(sees, (q[:, h] @ keys.T) * scale, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e @ values) / e.sum(axis=1, keepdims=True)
    return out


def rwkv_scan(r, k, v, w, u, state=None):
    """Per head: o_t = (S + diag(u) k_t v_t^T)^T r_t, then S <- diag(w_t) S + k_t v_t^T.  r, k, w [T, H, d],
    v [T, H, dv], u [H, d].  Returns (o, S)."""
    T, H, d = r.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            kv = np.outer(k[t, h], v[t, h])
            o[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = w[t, h][:, None] * S[h] + kv
    return o, S


def ssd_scan(x, dt, A_log, B, C, state=None):
    """Per head h of group g: S <- exp(-exp(A_log_h) dt) S + dt B_t x_t^T, o_t = S^T C_t.  x [T, H, dv], dt [T, H],
    B, C [T, G, N].  Returns (o, S)."""
    T, H, dv = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, dv)) if state is None else state.copy()
    o = np.zeros((T, H, dv))
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            o[t, h] = S[h].T @ C[t, g]
    return o, S


# ---- mixers -----------------------------------------------------------------------------------------
def pooled_attention(h, w, p, m, pos, eps):
    """The left half of a 'parallel' mixer."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        q = rotate_half(q, pos, rot["dims"], rot["base"], factor)
        k = rotate_half(k, pos, rot["dims"], rot["base"], factor)
    o = pooled_window_attention(unit_rms(q, eps), unit_rms(k, eps), v, m["scale"], m["mask"]["size"], m["mask"]["pool"])
    return o.reshape(T, H * dv) @ w[p + "o"].T


def rwkv_decay(z, w, p):
    """exp(-exp(W2 tanh(W1 z) + w0))."""
    return np.exp(-np.exp(np.tanh(z @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))


def rwkv_mixer(h, w, p, m, eps):
    """The right half of a 'parallel' mixer."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    mixed = {s: token_shift(h, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[p + s].T).reshape(T, H, d) for s in "rkv")
    decay = rwkv_decay(mixed["w"], w, p).reshape(T, H, d)
    o, _ = rwkv_scan(r, k, v, decay, w[p + "u"])
    z = unit_rms(o, eps).reshape(T, H * d) * w[p + "norm"] * silu(mixed["g"] @ w[p + "g"].T)
    return z @ w[p + "o"].T


def parallel_mixer(h, w, p, m, pos, eps):
    return (m["left_scale"] * pooled_attention(h, w, p + "left.", m["left"], pos, eps)
            + m["right_scale"] * rwkv_mixer(h, w, p + "right.", m["right"], eps))


def mamba2_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    o, _ = ssd_scan(x, dt, w[p + "A_log"], B, C)
    y = (o + w[p + "D"][None, :, None] * x).reshape(T, inner) * silu(z)
    parts = unit_rms(y.reshape(T, m["norm_groups"], -1), eps).reshape(T, inner)
    return (parts * w[p + "norm"]) @ w[p + "o"].T


def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---- the model -------------------------------------------------------------------------------------------
def layer_forward(x, w, cfg, i, pos):
    """x <- x + norm1(mixer(shifted x)); x <- x + norm2(ff(x))."""
    L = cfg["layers"][i]
    eps = cfg["norm"]["eps"]
    p = f"l{i}."
    h = token_shift(x, w[p + "shift"])
    if L["type"] == "parallel":
        y = parallel_mixer(h, w, p + "mix.", L["mixer"], pos, eps)
    elif L["type"] == "mamba2":
        y = mamba2_mixer(h, w, p + "mix.", L["mixer"], eps)
    else:
        raise ValueError(L["type"])
    x = x + rms_norm(y, w[p + "norm1"], eps)
    if L.get("mlp") is not None:
        x = x + rms_norm(dense_ff(x, w, p + "mlp."), w[p + "norm2"], eps)
    return x


def forward(tokens, w, cfg, return_layers=False):
    """Logits [T, vocab] of one sequence from position 0 (and the stream after every layer)."""
    tokens = np.asarray(tokens)
    pos = np.arange(len(tokens))
    x = w["embed"][tokens]
    layers = []
    for i in range(len(cfg["layers"])):
        x = layer_forward(x, w, cfg, i, pos)
        layers.append(x)
    logits = rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
    return (logits, np.stack(layers)) if return_layers else logits
