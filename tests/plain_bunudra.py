"""Bunudra, stated plainly: dense numpy in 64-bit, one function per mechanism,
whole sequences at once, a token-by-token loop for the recurrence, no cache
and no kernels.  Shares nothing with the package; the tests hold the
package's steps to this.

Notation: T tokens, W width, weights are stored [out, in] and applied as
y = x @ w.T.  ``w`` maps tensor names to float64 arrays; ``cfg`` is the
config.json dictionary.
"""
from __future__ import annotations

import json
import math
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


def layer_norm(x, weight, bias, eps):
    c = x - np.mean(x, axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * weight + bias


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu(z):
    """z times the normal distribution function of z."""
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def frequencies(rot):
    """(angle per position of every pair, what cos and sin are multiplied by) for a ``rot`` entry."""
    dims, base = rot["dims"], rot["base"]
    i = np.arange(dims // 2)
    f = base ** (-2.0 * i / dims)
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    where = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate_half(x, pos, rot):
    """x [T, heads, d]: numbers (i, i + dims / 2), i < dims / 2, of every head turn by the position's angle."""
    out, n = x.copy(), rot["dims"] // 2
    f, amp = frequencies(rot)
    a = np.asarray(pos, dtype=np.float64)[:, None] * f[None, :]
    c, s = amp * np.cos(a)[:, None, :], amp * np.sin(a)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def rotate_pairs(x, pos, rot):
    """The same with numbers (2 i, 2 i + 1)."""
    out, n = x.copy(), rot["dims"] // 2
    f, amp = frequencies(rot)
    a = np.asarray(pos, dtype=np.float64)[:, None] * f[None, :]
    c, s = amp * np.cos(a)[:, None, :], amp * np.sin(a)[:, None, :]
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out[..., 0:2 * n:2] = u * c - v * s
    out[..., 1:2 * n:2] = v * c + u * s
    return out


def sees_chunk(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def sees_window(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def softmax_rows(s, sees):
    s = np.where(sees, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def masked_attention(q, k, v, scale, sees):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads head h // (H / G).  Returns [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_rows((q[:, h] @ k[:, g].T) * scale, sees) @ v[:, g]
    return out


def mlstm_gates(zi, zf, cap):
    """(log input gate, log forget gate) from the two raw numbers."""
    i = cap * np.tanh(zi / cap)
    f = cap * np.tanh(zf / cap)
    return i, -np.logaddexp(0.0, -f)


def mlstm_scan(q, k, v, i, f, state=None):
    """q, k [T, H, d] (q with its factor), v [T, H, dv], log gates i, f [T, H].  ``state`` (S [H, d, dv], n [H, d],
    m [H]) or None for a sequence's beginning.  Returns (o [T, H, dv], state)."""
    T, H, d = q.shape
    if state is None:
        S, n, m = np.zeros((H, d, v.shape[2])), np.zeros((H, d)), np.zeros(H)
    else:
        S, n, m = (x.copy() for x in state)
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        new = np.maximum(f[t] + m, i[t])
        keep, put = np.exp(f[t] + m - new), np.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = new
        top = np.einsum("hij,hi->hj", S, q[t])
        o[t] = top / (np.maximum(np.abs(np.sum(n * q[t], axis=1)), np.exp(-m)) + 1e-6)[:, None]
    return o, (S, n, m)


def choose_experts(s, top, groups):
    """Indices of the ``top`` largest scores of one token among the experts of the groups with the largest best score."""
    s = s.copy()
    if groups:
        best = s.reshape(groups["count"], -1).max(axis=1)
        kept = np.argsort(-best, kind="stable")[:groups["keep"]]
        size = len(s) // groups["count"]
        for g in range(groups["count"]):
            if g not in kept:
                s[g * size:(g + 1) * size] = -np.inf
    return np.argsort(-s, kind="stable")[:top]


# ---- mixers -----------------------------------------------------------------------------------------
def attention_mixer(h, w, p, m, pos, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T).reshape(T, H, d), eps) * w[p + "q.norm"]
    k = unit_rms((h @ w[p + "k"].T).reshape(T, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    o = masked_attention(rotate_half(q, pos, m["rot"]), rotate_half(k, pos, m["rot"]), v, m["scale"],
                         sees_chunk(T, m["mask"]["size"]))
    return o.reshape(T, H * dv) @ w[p + "o"].T


def latent_mixer(h, w, p, m, pos, eps):
    """Every head's keys and values spelled out."""
    T = h.shape[0]
    H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, d + dr)
    down = h @ w[p + "dkv"].T
    c = unit_rms(down[:, :R], eps) * w[p + "dkv.norm"]
    shared = rotate_pairs(down[:, None, R:], pos, m["rot"])                                  # [T, 1, dr]
    q = np.concatenate([q[:, :, :d], rotate_pairs(q[:, :, d:], pos, m["rot"])], axis=2)
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, d), np.repeat(shared, H, axis=1)], axis=2)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = masked_attention(q, k, v, m["scale"], sees_window(T, m["mask"]["size"])).reshape(T, H * dv)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mlstm_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d) / math.sqrt(d)
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    i, f = mlstm_gates(h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"], m["gate_cap"])
    o, _ = mlstm_scan(q, k, v, i, f)
    z = unit_rms(o, eps).reshape(T, H * dv) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return z @ w[p + "o"].T


MIXERS = {"attention": lambda h, w, p, m, pos, eps: attention_mixer(h, w, p, m, pos, eps),
          "latent_attention": lambda h, w, p, m, pos, eps: latent_mixer(h, w, p, m, pos, eps),
          "mlstm": lambda h, w, p, m, pos, eps: mlstm_mixer(h, w, p, m, eps)}


# ---- the feed-forward -----------------------------------------------------------------------------------
def small_ff(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def routing_margin(z, top, groups):
    """By how much the logits z [N] of one token would have to move for another choice: the smaller of the gaps between
    the last group kept and the best one that is not, and between the last expert chosen and the best one that is not."""
    gap = np.inf
    if groups:
        best = np.sort(z.reshape(groups["count"], -1).max(axis=1))[::-1]
        if groups["keep"] < groups["count"]:
            gap = best[groups["keep"] - 1] - best[groups["keep"]]
    allowed = np.sort(z[choose_experts(z, len(z) if not groups else len(z) // groups["count"] * groups["keep"], groups)])[::-1]
    return min(gap, allowed[top - 1] - allowed[top]) if top < len(allowed) else gap


def experts_ff(h, w, p, m, margins=None):
    r = m["router"]
    z = h @ w[p + "router"].T
    if margins is not None:
        margins.append(np.array([routing_margin(row, r["top"], r.get("groups")) for row in z]))
    e = np.exp(z - z.max(axis=1, keepdims=True))
    s = e / e.sum(axis=1, keepdims=True)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for x in choose_experts(s[t], r["top"], r.get("groups")):
            out[t] += s[t, x] * r.get("scale", 1.0) * small_ff(h[t:t + 1], w, f"{p}e{x}.")[0]
    if m.get("shared"):
        out += small_ff(h, w, p + "shared.") * sigmoid(h @ w[p + "shared.sg"].T)
    return out


# ---- the model -------------------------------------------------------------------------------------------
def layer_forward(x, w, cfg, i, pos, margins=None):
    """The stream after one layer: each part's output is normed and added."""
    L = cfg["layers"][i]
    eps = cfg["norm"]["eps"]
    p = f"l{i}."
    norm = lambda y, name: layer_norm(y, w[p + name], w[p + name + ".b"], eps)
    x = x + norm(MIXERS[L["type"]](x, w, p + "mix.", L["mixer"], pos, eps), "norm1")
    if L.get("mlp") is not None:
        x = x + norm(experts_ff(x, w, p + "mlp.", L["mlp"], margins), "norm2")
    return x


def forward(tokens, w, cfg, return_layers=False, margins=None):
    """Logits [T, vocab] of one sequence from position 0 (and the stream after every layer).  ``margins`` (a list)
    receives one array [T] per layer with experts: the routers' margins."""
    tokens = np.asarray(tokens)
    pos = np.arange(len(tokens))
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    layers = []
    for i in range(len(cfg["layers"])):
        x = layer_forward(x, w, cfg, i, pos, margins)
        layers.append(x)
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]) @ w["head"].T
    return (logits, np.stack(layers)) if return_layers else logits
