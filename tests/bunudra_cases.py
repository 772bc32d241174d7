"""Small Bunudra configurations for the tests, their model folders and plain logits.

The cases differ from one another in every size.  Together they cover: the
three mixers in different orders, several of a kind in one model with sizes
of their own, layers with and without a feed-forward; attention with one
key/value head per head and with several heads per key/value head, keys
larger and smaller than values, rotation of none, part and all of a head,
chunks of 1 to 130 tokens; latents larger and smaller than what they expand
to, rotated parts of none, some and many numbers, frequencies scaled and
not, ramps that start below zero and ramps of one step, windows of 1 to
130 tokens; one memory head and several, gate caps
of 1 to 15; experts in groups of which one, some and all are kept, without
groups, one choice and several, weights times one and something else, with
and without a shared expert; sizes that are no multiple of 8, and a width
that is no multiple of 4.

Weights are random but not all alike: norm weights away from one, biases
that matter, forget gates near one (so that the memories remember), routers
with few close calls.
"""
from __future__ import annotations

import json
import math
import tempfile
from pathlib import Path

import numpy as np


def memory(heads, dim, vdim, cap):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap))


def chunked(heads, kv_heads, dim, vdim, size, dims=0, base=10000.0, scale=None):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim,
                                             scale=scale or 1.0 / math.sqrt(dim), mask=dict(size=size),
                                             rot=dict(base=base, dims=dims)))


def latent(heads, dim, rot_dim, vdim, rank, size, base=10000.0, yarn=None, scale=None):
    """``yarn``: (factor, original, fast, slow)."""
    rot = dict(base=base, dims=rot_dim)
    if yarn:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank,
                                                    scale=scale or 1.0 / math.sqrt(dim + rot_dim), mask=dict(size=size), rot=rot))


def experts(n, top, ff, groups=None, scale=1.0, shared=0):
    router = dict(experts=n, scale=scale, top=top)
    if groups:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", expert=dict(ff=ff), router=router, shared=dict(ff=shared) if shared else None)


def layer(mix, mlp):
    return dict(mix, mlp=mlp)


# A: every mixer, two of the memories; a layer without a feed-forward; two of three groups kept; no groups.
CASE_A = dict(
    architecture="Bunudra", width=64, vocab=200, embedding=dict(scale=1.5), norm=dict(eps=1e-5),
    layers=[layer(memory(3, 16, 24, 9.0), experts(6, 2, 24, (3, 2), 1.7, 40)),
            layer(latent(4, 16, 16, 24, 48, 12, 1000.0, (4.0, 64.0, 8.0, 1.0)), None),
            layer(chunked(6, 2, 24, 16, 10, dims=16, base=100.0), experts(5, 1, 40, None, 0.8, 16)),
            layer(memory(1, 24, 8, 4.0), experts(8, 3, 16, (4, 3), 1.0, 24))])
# B: a chunk and a window of one token (a token sees itself only); one memory head; every head its own key/value head;
#    nothing rotated in the chunks; all groups kept; no shared expert.
CASE_B = dict(
    architecture="Bunudra", width=96, vocab=130, embedding=dict(scale=1.0), norm=dict(eps=1e-6),
    layers=[layer(latent(2, 32, 8, 16, 32, 1), experts(4, 2, 32, (2, 2), 1.0, 0)),
            layer(memory(1, 48, 32, 1.0), experts(6, 6, 8, (1, 1), 0.5, 56)),
            layer(chunked(3, 3, 32, 48, 1), None),
            layer(chunked(4, 1, 16, 32, 17, dims=16, base=500.0, scale=0.4), experts(4, 1, 16, (4, 1), 2.0, 8))])
# C: sizes that are no multiple of 8; a large epsilon; a ramp of one step at most (fast and slow alike).
CASE_C = dict(
    architecture="Bunudra", width=40, vocab=90, embedding=dict(scale=0.7), norm=dict(eps=1e-3),
    layers=[layer(chunked(6, 3, 12, 20, 8, dims=6, base=70.0), experts(9, 2, 12, (3, 1), 1.3, 20)),
            layer(memory(5, 6, 10, 15.0), experts(3, 2, 28, None, 1.0, 12)),
            layer(latent(3, 10, 6, 14, 20, 7, 30.0, (8.0, 40.0, 2.0, 2.0)), experts(6, 2, 20, (2, 1), 0.6, 36))])
# D: sizes in multiples of 16 with prompts of several hundred tokens (the tensor-core kernels' tiles; windows and chunks
#    of several tiles; a latent that is expanded for prompts and one that is not; the recurrence in chunks).
CASE_D = dict(
    architecture="Bunudra", width=128, vocab=320, embedding=dict(scale=0.9), norm=dict(eps=1e-6),
    layers=[layer(memory(4, 32, 64, 12.0), experts(8, 2, 64, (4, 2), 1.5, 96)),
            layer(latent(8, 32, 16, 32, 64, 70, 20000.0, (16.0, 128.0, 16.0, 1.0)), experts(4, 1, 64, (2, 1), 1.0, 64)),
            layer(chunked(8, 2, 64, 48, 50, dims=32, base=20000.0), experts(6, 2, 48, (2, 1), 0.7, 32)),
            layer(latent(4, 64, 32, 64, 32, 130, 5000.0), None),
            layer(chunked(4, 4, 32, 32, 130, dims=32, base=300.0), experts(8, 2, 32, (2, 1), 1.2, 64))])
# E: a width and a vocabulary that are multiples of neither 8 nor 4 (rows that start off 16-byte boundaries); head sizes
#    of 10, 6 and 3; a rotated part of nothing; a memory last.
CASE_E = dict(
    architecture="Bunudra", width=38, vocab=77, embedding=dict(scale=2.0), norm=dict(eps=1e-5),
    layers=[layer(latent(5, 6, 4, 3, 14, 20, 50.0, (2.0, 500.0, 4.0, 0.5)), experts(6, 2, 10, (2, 1), 1.1, 6)),
            layer(chunked(4, 2, 10, 6, 3, dims=4, base=9.0), None),
            layer(latent(2, 12, 0, 10, 9, 5), experts(5, 3, 14, (5, 4), 1.4, 22)),
            layer(memory(3, 10, 7, 6.0), experts(4, 2, 18, (2, 2), 0.9, 30))])


def with_all_experts(cfg):
    """The same with every expert chosen: no choice that rounding can turn."""
    cfg = json.loads(json.dumps(cfg))
    for L in cfg["layers"]:
        if L["mlp"]:
            L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
            L["mlp"]["router"].pop("groups", None)
    return cfg


CASES = {"A": (CASE_A, 3, 8), "B": (CASE_B, 5, 16), "C": (CASE_C, 7, 32), "D": (CASE_D, 9, 16),
         "E": (CASE_E, 11, 4)}                                                                # config, seed, page
CASES.update({n + "-all": (with_all_experts(CASES[n][0]), *CASES[n][1:]) for n in "ACD"})

_made: dict = {}
_plain: dict = {}


def random_tensors(cfg: dict, seed: int, std: float = 0.12) -> dict:
    """name -> float32 array for every tensor of the model, by name."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    n = lambda *shape, s=std: rng.normal(0.0, s, size=shape)
    near_one = lambda *shape: 1.0 + rng.uniform(-0.3, 0.3, size=shape)
    t = {"embed": n(cfg["vocab"], W, s=0.5), "final.norm": near_one(W), "final.norm.b": n(W, s=0.2), "head": n(cfg["vocab"], W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        t[p + "norm1"], t[p + "norm1.b"] = near_one(W) * 0.6, n(W, s=0.2)
        if L["type"] == "mlstm":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            t.update({q + "q": n(H * d, W, s=0.25), q + "k": n(H * d, W, s=0.25), q + "v": n(H * dv, W), q + "g": n(H * dv, W),
                      q + "i": n(H, W, s=0.2), q + "i.b": rng.uniform(-2.0, 1.0, size=H), q + "f": n(H, W, s=0.2),
                      q + "f.b": rng.uniform(1.0, 5.0, size=H), q + "norm": near_one(H * dv), q + "o": n(W, H * dv)})
        elif L["type"] == "latent_attention":
            H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            t.update({q + "q": n(H * (d + dr), W), q + "dkv": n(R + dr, W), q + "dkv.norm": near_one(R), q + "uk": n(H * d, R, s=0.2),
                      q + "uv": n(H * dv, R, s=0.2), q + "g": n(H * dv, W), q + "o": n(W, H * dv)})
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            t.update({q + "q": n(H * d, W), q + "k": n(G * d, W), q + "v": n(G * dv, W), q + "q.norm": near_one(d) * 1.5,
                      q + "k.norm": near_one(d), q + "o": n(W, H * dv)})
        if L["mlp"]:
            f = L["mlp"]
            F, N = f["expert"]["ff"], f["router"]["experts"]
            b = p + "mlp."
            t.update({p + "norm2": near_one(W) * 0.6, p + "norm2.b": n(W, s=0.2), b + "router": n(N, W, s=0.4)})
            for e in range(N):
                t.update({f"{b}e{e}.up": n(F, W), f"{b}e{e}.down": n(W, F)})
            if f["shared"]:
                S = f["shared"]["ff"]
                t.update({b + "shared.up": n(S, W), b + "shared.down": n(W, S), b + "shared.sg": n(1, W, s=0.2)})
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
        _made[name] = write_model(cfg, seed, tempfile.mkdtemp(prefix=f"rg_bunudra_{name}_"))
    return _made[name]


class Plain:
    """The plain statement over a model folder."""

    def __init__(self, folder):
        import plain_bunudra as P
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
