"""Small Sagizen configurations for the tests, their model folders and plain logits.

The cases differ from one another in every size.  Together they cover: the
two mixers in different orders, layers with and without a feed-forward;
Mamba-2 with one head and several, heads that share B and C in groups and
heads that do not, the norm in one part and in several, convolutions of 1 to
5 taps; attention halves with one key/value head per head and with several
heads per key/value head, keys larger and smaller than values, rotation of
none, part and all of a head with and without scaled frequencies, windows of
1 to 130 tokens, blocks of 1 to 40 tokens, smaller, equal and larger than the
window; time mixing with one head and several and decay ranks of 3 to 40;
halves scaled on both sides of one; sizes that are no multiple of 8, and a
width that is no multiple of 4.

Weights are random but not all alike: norm weights away from one, biases
that matter, shares of the previous token from below zero to above one,
decays near 1 (so that the states remember).
"""
from __future__ import annotations

import json
import math
import tempfile
from pathlib import Path

import numpy as np


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv,
                                          norm_groups=norm_groups))


def left(heads, kv_heads, dim, vdim, size, pool, dims=0, base=10000.0, factor=None, scale=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or 1.0 / math.sqrt(dim),
             mask=dict(size=size, pool=pool))
    if dims:
        m["rot"] = dict(base=base, dims=dims)
        if factor:
            m["rot"]["scaling"] = dict(factor=factor)
    return m


def parallel(l, heads, dim, left_scale, right_scale):
    return dict(type="parallel", mixer=dict(left=l, right=dict(heads=heads, dim=dim), left_scale=left_scale,
                                            right_scale=right_scale))


def layer(mix, ff):
    return dict(mix, mlp=dict(kind="dense", ff=ff) if ff else None)


# A: a parallel layer first; part of the left heads rotated with scaled frequencies, a window of 12 with blocks of 5;
#    a layer without a feed-forward; blocks larger than the window.
CASE_A = dict(
    architecture="Sagizen", width=64, vocab=200, norm=dict(eps=1e-5),
    layers=[layer(parallel(left(4, 2, 16, 24, 12, 5, dims=8, base=100.0, factor=2.5), 3, 12, 0.7, 1.3), 96),
            layer(mamba(4, 16, 24, 2, 4, 2), None),
            layer(parallel(left(6, 3, 24, 8, 7, 11, dims=24, base=1000.0, scale=0.9), 2, 32, 1.1, 0.4), 40),
            layer(mamba(6, 8, 16, 3, 3, 1), 56)])
# B: one block per token (every key far away is seen by itself), a window of one token; every head its own key/value
#    head; a convolution of one tap; one state head; no rotation.
CASE_B = dict(
    architecture="Sagizen", width=96, vocab=130, norm=dict(eps=1e-6),
    layers=[layer(mamba(1, 48, 32, 1, 1, 3), 64),
            layer(parallel(left(3, 3, 32, 32, 9, 1), 1, 48, 1.0, 1.0), None),
            layer(parallel(left(4, 1, 16, 48, 1, 3, dims=16, base=500.0), 4, 16, 0.5, 2.0), 72)])
# C: sizes that are no multiple of 8; five taps; large epsilon; blocks as large as the window.
CASE_C = dict(
    architecture="Sagizen", width=40, vocab=90, norm=dict(eps=1e-3),
    layers=[layer(mamba(5, 6, 10, 5, 5, 2), 36),
            layer(parallel(left(6, 3, 12, 20, 8, 8, dims=6, base=70.0, factor=8.0), 3, 7, 1.6, 0.9), 28),
            layer(mamba(3, 20, 12, 1, 2, 5), 52)])
# D: sizes in multiples of 16 with prompts of several hundred tokens (the tensor-core kernels' tiles, many blocks beside
#    a window of several tiles, a state of 128 rows).
CASE_D = dict(
    architecture="Sagizen", width=128, vocab=320, norm=dict(eps=1e-6),
    layers=[layer(mamba(8, 32, 64, 2, 4, 4), 192),
            layer(parallel(left(8, 2, 64, 48, 70, 4, dims=32, base=20000.0, factor=4.0), 4, 32, 0.8, 0.6), 160),
            layer(mamba(4, 16, 128, 4, 3, 1), None),
            layer(parallel(left(4, 4, 32, 32, 130, 16, dims=32, base=300.0), 2, 64, 1.2, 0.7), 64),
            layer(parallel(left(2, 1, 128, 64, 33, 40, dims=64, base=5000.0, factor=1.5), 8, 16, 0.9, 1.1), 96)])
# E: a width and a vocabulary that are multiples of neither 8 nor 4 (rows that start off 16-byte boundaries); head
#    sizes of 10, 6 and 3; a mamba layer last.
CASE_E = dict(
    architecture="Sagizen", width=38, vocab=77, norm=dict(eps=1e-5),
    layers=[layer(parallel(left(2, 2, 10, 6, 3, 2, dims=4, base=50.0, factor=3.0), 5, 3, 1.0, 0.5), 30),
            layer(parallel(left(4, 1, 6, 10, 20, 7, dims=6, base=9.0), 1, 10, 0.3, 1.4), None),
            layer(mamba(3, 6, 9, 3, 4, 3), 22)])

CASES = {"A": (CASE_A, 3, 8), "B": (CASE_B, 5, 16), "C": (CASE_C, 7, 32), "D": (CASE_D, 9, 16),
         "E": (CASE_E, 11, 4)}                                                                # config, seed, page
RANKS = {64: 5, 96: 3, 40: 12, 128: 40, 38: 7}                                                # of the decay, by width

_made: dict = {}
_plain: dict = {}


def random_tensors(cfg: dict, seed: int, std: float = 0.12) -> dict:
    """name -> float32 array for every tensor of the model, by name."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    n = lambda *shape, s=std: rng.normal(0.0, s, size=shape)
    near_one = lambda *shape: 1.0 + rng.uniform(-0.3, 0.3, size=shape)
    share = lambda: rng.uniform(-0.2, 1.1, size=W)
    rank = RANKS.get(W, 16)
    t = {"embed": n(cfg["vocab"], W, s=0.5), "final.norm": near_one(W), "head": n(cfg["vocab"], W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        t[p + "norm1"], t[p + "shift"] = near_one(W) * 0.6, share()
        if L["type"] == "mamba2":
            H, dv, N, G, K = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            inner = H * dv
            C = inner + 2 * G * N
            t.update({q + "in": n(inner + C + H, W), q + "conv": n(C, K, s=0.5), q + "conv.b": n(C, s=0.3),
                      q + "dt_bias": rng.uniform(-4.0, 0.0, size=H), q + "A_log": rng.uniform(-2.0, 1.0, size=H),
                      q + "D": near_one(H), q + "norm": near_one(inner), q + "o": n(W, inner)})
        else:
            a, r = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            b = q + "left."
            t.update({b + "q": n(H * d, W), b + "k": n(G * d, W), b + "v": n(G * dv, W), b + "o": n(W, H * dv),
                      b + "q.b": n(H * d, s=0.4), b + "k.b": n(G * d, s=0.4), b + "v.b": n(G * dv, s=0.4)})
            H, d = r["heads"], r["dim"]
            b = q + "right."
            t.update({b + "mu." + s: share() for s in "rkvgw"})
            t.update({b + s: n(H * d, W) for s in "rkvg"})
            t.update({b + "w1": n(rank, W, s=0.3), b + "w2": n(H * d, rank, s=0.5), b + "w0": rng.uniform(-6.0, 0.5, size=H * d),
                      b + "u": n(H, d, s=0.5), b + "norm": near_one(H * d), b + "o": n(W, H * d)})
        if L["mlp"]:
            F = L["mlp"]["ff"]
            t.update({p + "norm2": near_one(W) * 0.6, p + "mlp.gate": n(F, W), p + "mlp.up": n(F, W), p + "mlp.down": n(W, F)})
    return {k: np.asarray(v, dtype=np.float32) for k, v in t.items()}


def write_model(cfg: dict, seed: int, out_dir, change=None) -> Path:
    """config.json and model.safetensors (bfloat16) for ``cfg``; ``change(tensors)`` may edit the arrays first."""
    import torch
    from railgun_b200.weights.safetensors_io import write_safetensors
    out_dir = Path(out_dir)
    out_dir.mkdir(parents=True, exist_ok=True)
    tensors = random_tensors(cfg, seed)
    if change is not None:
        change(tensors)
    (out_dir / "config.json").write_text(json.dumps(cfg))
    write_safetensors(out_dir / "model.safetensors",
                      {k: torch.from_numpy(v).to(torch.bfloat16) for k, v in tensors.items()})
    return out_dir


def model_dir(name: str) -> Path:
    if name not in _made:
        cfg, seed, _ = CASES[name]
        _made[name] = write_model(cfg, seed, tempfile.mkdtemp(prefix=f"rg_sagizen_{name}_"))
    return _made[name]


class Plain:
    """The plain statement over a model folder."""

    def __init__(self, folder):
        import plain_sagizen as P
        self.P = P
        self.cfg = json.loads((Path(folder) / "config.json").read_text())
        self.w = P.read_safetensors(Path(folder) / "model.safetensors")

    def forward(self, ids):
        return self.P.forward(ids, self.w, self.cfg)

    def greedy(self, prompt, n):
        ids = list(prompt)
        for _ in range(n):
            ids.append(int(np.argmax(self.forward(ids)[-1])))
        return ids[len(prompt):]


def plain_model(name: str) -> Plain:
    if name not in _plain:
        _plain[name] = Plain(model_dir(name))
    return _plain[name]


def prompts(vocab: int, lengths, seed: int):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, vocab, size=n).tolist() for n in lengths]
