"""The plain statement of Bunudra against loop-level formulas, and the package's
configuration, description, tensor list and cache needs for the design (no GPU)."""
import json
import math

import numpy as np
import pytest

import bunudra_cases as C
import plain_bunudra as P


def weights(cfg, seed=1):
    return {k: v.astype(np.float64) for k, v in C.random_tensors(cfg, seed).items()}


def rms(x, eps):
    return math.sqrt(float((np.asarray(x) ** 2).mean()) + eps)


def test_layer_norm_centres_first():
    rng = np.random.default_rng(0)
    x, w, b = rng.normal(size=(4, 7)) + 50.0, rng.normal(size=7), rng.normal(size=7)
    got = P.layer_norm(x, w, b, 1e-2)
    for t in range(4):
        mean = sum(x[t]) / 7
        var = sum((v - mean) ** 2 for v in x[t]) / 7
        assert np.allclose(got[t], [(x[t, i] - mean) / math.sqrt(var + 1e-2) * w[i] + b[i] for i in range(7)], atol=1e-12)
    assert np.allclose(P.layer_norm(x + 3.0, w, b, 1e-2), got, atol=1e-10)


def test_gelu_is_the_exact_one():
    z = np.array([-4.0, -1.0, 0.0, 0.5, 2.0])
    from statistics import NormalDist
    assert np.allclose(P.gelu(z), [v * NormalDist().cdf(v) for v in z], atol=1e-12)
    tanh_form = 0.5 * z * (1 + np.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))
    assert np.abs(tanh_form - P.gelu(z)).max() > 1e-5


def test_rotations_pair_by_pair():
    rng = np.random.default_rng(2)
    x, pos = rng.normal(size=(3, 2, 12)), np.array([0, 5, 900])
    for dims, base, scaling in ((8, 50.0, None), (12, 1000.0, dict(factor=4.0, original=64.0, fast=8.0, slow=1.0))):
        rot = dict(dims=dims, base=base, scaling=scaling)
        f, amp = P.frequencies(rot)
        half, pairs = P.rotate_half(x, pos, rot), P.rotate_pairs(x, pos, rot)
        for t in range(3):
            for i in range(dims // 2):
                a = pos[t] * f[i]
                c, s = amp * math.cos(a), amp * math.sin(a)
                for h in range(2):
                    u, v = x[t, h, i], x[t, h, i + dims // 2]
                    assert abs(half[t, h, i] - (u * c - v * s)) < 1e-12
                    assert abs(half[t, h, i + dims // 2] - (v * c + u * s)) < 1e-12
                    u, v = x[t, h, 2 * i], x[t, h, 2 * i + 1]
                    assert abs(pairs[t, h, 2 * i] - (u * c - v * s)) < 1e-12
                    assert abs(pairs[t, h, 2 * i + 1] - (v * c + u * s)) < 1e-12
        assert np.array_equal(half[..., dims:], x[..., dims:]) and np.array_equal(pairs[..., dims:], x[..., dims:])


YARNS = [(32, 10000.0, 8.0, 2048.0, 32.0, 1.0), (16, 1000.0, 4.0, 64.0, 8.0, 1.0), (8, 30.0, 16.0, 40.0, 2.0, 2.0),
         (64, 500000.0, 40.0, 4096.0, 32.0, 1.0), (6, 7.0, 2.0, 30.0, 90.0, 0.001)]


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", YARNS)
def test_scaled_frequencies(dims, base, factor, original, fast, slow):
    """Pair by pair, by the plain statement and by the package; the ramp's ends kept within the pairs."""
    from railgun_b200.parts.latent_attention import yarn_frequencies
    f, amp = P.frequencies(dict(dims=dims, base=base, scaling=dict(factor=factor, original=original, fast=fast, slow=slow)))
    at = lambda t: dims * math.log(original / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(fast)), 0), min(math.ceil(at(slow)), dims - 1)
    for i in range(dims // 2):
        plain = base ** (-2.0 * i / dims)
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        assert abs(f[i] - (plain / factor * r + plain * (1 - r))) < 1e-15
    assert abs(amp - (0.1 * math.log(factor) + 1.0)) < 1e-15
    g, mult = yarn_frequencies(dims, base, factor, original, fast, slow)
    assert np.allclose(g.numpy(), f, rtol=1e-14) and abs(mult - amp) < 1e-15


@pytest.mark.parametrize("size", [1, 2, 5, 7, 30])
def test_what_a_query_sees(size):
    T = 23
    chunk, window = P.sees_chunk(T, size), P.sees_window(T, size)
    for i in range(T):
        assert [j for j in range(T) if window[i, j]] == [j for j in range(T) if 0 <= i - j <= size - 1]
        first = (i // size) * size
        assert [j for j in range(T) if chunk[i, j]] == list(range(first, i + 1))


def test_attention_against_loops():
    rng = np.random.default_rng(3)
    T, H, G, d, dv = 11, 6, 2, 5, 3
    q, k, v = rng.normal(size=(T, H, d)), rng.normal(size=(T, G, d)), rng.normal(size=(T, G, dv))
    got = P.masked_attention(q, k, v, 0.7, P.sees_chunk(T, 4))
    for i in range(T):
        for h in range(H):
            g = h // 3
            js = range(i // 4 * 4, i + 1)
            e = [math.exp(0.7 * float(q[i, h] @ k[j, g])) for j in js]
            assert np.allclose(got[i, h], sum(a * v[j, g] for a, j in zip(e, js)) / sum(e), atol=1e-12)


def test_memory_is_a_sum_over_the_tokens_before():
    """o without the running maximum: weights exp(i_s + sum of f after s) over max(|their sum with k q|, 1), times the
    same; the maximum only keeps the numbers small (the 1e-6 aside).  The state can be carried on."""
    rng = np.random.default_rng(4)
    T, H, d, dv = 12, 3, 4, 5
    q, k, v = rng.normal(size=(T, H, d)), rng.normal(size=(T, H, d)), rng.normal(size=(T, H, dv))
    i, f = P.mlstm_gates(rng.normal(size=(T, H)) * 3.0, rng.normal(size=(T, H)) + 1.0, 5.0)
    assert (f < 0).all() and (np.abs(i) < 5.0).all()
    o, (S, n, m) = P.mlstm_scan(q, k, v, i, f)
    small = 0
    for t in range(T):
        for h in range(H):
            w = [math.exp(i[s, h] + f[s + 1:t + 1, h].sum()) * float(k[s, h] @ q[t, h]) for s in range(t + 1)]
            den = max(abs(sum(w)), 1.0)
            small += abs(sum(w)) < 1.0
            ref = sum(a * v[s, h] for s, a in enumerate(w)) / den
            assert np.allclose(o[t, h], ref, rtol=1e-3, atol=1e-4)
    assert 0 < small < T * H                                                   # both sides of the maximum
    o1, st = P.mlstm_scan(q[:5], k[:5], v[:5], i[:5], f[:5])
    o2, (S2, n2, m2) = P.mlstm_scan(q[5:], k[5:], v[5:], i[5:], f[5:], st)
    assert np.allclose(np.concatenate([o1, o2]), o, atol=1e-12) and np.allclose(S2, S) and np.allclose(m2, m)
    # the maximum starts at 0: a first token with a small input gate is not brought to full size
    o, (S, n, m) = P.mlstm_scan(q[:1], k[:1], v[:1], np.full((1, H), -3.0), np.full((1, H), -1.0))
    assert np.allclose(m, -1.0) and np.allclose(n, math.exp(-2.0) * k[0])


def test_gates_against_their_formulas():
    zi, zf = np.array([-40.0, 0.3, 90.0]), np.array([-40.0, 0.3, 90.0])
    i, f = P.mlstm_gates(zi, zf, 6.0)
    for a, z in enumerate(zi):
        c = 6.0 * math.tanh(z / 6.0)
        assert abs(i[a] - c) < 1e-12 and abs(f[a] - math.log(1.0 / (1.0 + math.exp(-c)))) < 1e-12


def test_choice_of_experts():
    s = np.array([0.10, 0.30, 0.05, 0.20, 0.25, 0.01, 0.06, 0.03])
    assert list(P.choose_experts(s, 3, None)) == [1, 4, 3]
    assert list(P.choose_experts(s, 2, dict(count=4, keep=1))) == [1, 0]        # the group with the largest best score only
    assert list(P.choose_experts(s, 3, dict(count=4, keep=2))) == [1, 4, 0]     # groups (0, 1) and (4, 5): not 3
    assert list(P.choose_experts(s, 3, dict(count=2, keep=2))) == [1, 4, 3]
    z = np.log(s)
    assert abs(P.routing_margin(z, 3, None) - (z[3] - z[0])) < 1e-12
    assert abs(P.routing_margin(z, 2, dict(count=4, keep=1)) - (z[1] - z[4])) < 1e-12
    assert abs(P.routing_margin(z, 3, dict(count=4, keep=2)) - min(z[4] - z[3], z[0] - z[5])) < 1e-12


def test_experts_against_loops():
    cfg = C.CASE_A
    w = weights(cfg)
    m, p = cfg["layers"][0]["mlp"], "l0.mlp."
    h = np.random.default_rng(6).normal(size=(9, cfg["width"]))
    got = P.experts_ff(h, w, p, m)
    for t in range(9):
        z = w[p + "router"] @ h[t]
        s = np.exp(z) / np.exp(z).sum()
        best = sorted(range(3), key=lambda g: -max(s[2 * g], s[2 * g + 1]))[:2]
        ids = sorted([e for e in range(6) if e // 2 in best], key=lambda e: -s[e])[:2]
        y = sum(1.7 * s[e] * (w[f"{p}e{e}.down"] @ P.gelu(w[f"{p}e{e}.up"] @ h[t])) for e in ids)
        sg = 1.0 / (1.0 + math.exp(-float(w[p + "shared.sg"][0] @ h[t])))
        y = y + sg * (w[p + "shared.down"] @ P.gelu(w[p + "shared.up"] @ h[t]))
        assert np.allclose(got[t], y, atol=1e-10)


def test_mixers_against_loops():
    w, eps = weights(C.CASE_A), 1e-5
    T = 30
    h = np.random.default_rng(5).normal(size=(T, 64))
    pos = np.arange(T)
    # latent attention: scores over the latent itself, the gate on the heads' outputs
    m, p = C.CASE_A["layers"][1]["mixer"], "l1.mix."
    got = P.latent_mixer(h, w, p, m, pos, eps)
    down = h @ w[p + "dkv"].T
    c = np.stack([r[:48] / rms(r[:48], eps) for r in down]) * w[p + "dkv.norm"]
    kr = P.rotate_pairs(down[:, None, 48:], pos, m["rot"])[:, 0]
    for t in (0, 3, 29):
        q = (w[p + "q"] @ h[t]).reshape(4, 32)
        out = []
        for hd in range(4):
            qr = P.rotate_pairs(q[None, hd:hd + 1, 16:], pos[t:t + 1], m["rot"])[0, 0]
            qa = w[p + "uk"][hd * 16:(hd + 1) * 16].T @ q[hd, :16]
            js = range(max(0, t - 11), t + 1)
            e = np.array([math.exp(m["scale"] * (float(qa @ c[j]) + float(qr @ kr[j]))) for j in js])
            out.append(w[p + "uv"][hd * 24:(hd + 1) * 24] @ sum(a * c[j] for a, j in zip(e / e.sum(), js)))
        gate = 1.0 / (1.0 + np.exp(-(w[p + "g"] @ h[t])))
        assert np.allclose(got[t], w[p + "o"] @ (np.concatenate(out) * gate), atol=1e-9)
    # the memory: q's factor, biases of the gates, every head's norm before weight and gate
    m, p = C.CASE_A["layers"][0]["mixer"], "l0.mix."
    got = P.mlstm_mixer(h, w, p, m, eps)
    S, n, mm = np.zeros((3, 16, 24)), np.zeros((3, 16)), np.zeros(3)
    for t in range(T):
        q, k, v = ((w[p + a] @ h[t]).reshape(3, -1) for a in "qkv")
        i = 9.0 * np.tanh((w[p + "i"] @ h[t] + w[p + "i.b"]) / 9.0)
        f = -np.log1p(np.exp(-9.0 * np.tanh((w[p + "f"] @ h[t] + w[p + "f.b"]) / 9.0)))
        out = []
        for hd in range(3):
            new = max(f[hd] + mm[hd], i[hd])
            S[hd] = math.exp(f[hd] + mm[hd] - new) * S[hd] + math.exp(i[hd] - new) * np.outer(k[hd], v[hd])
            n[hd] = math.exp(f[hd] + mm[hd] - new) * n[hd] + math.exp(i[hd] - new) * k[hd]
            mm[hd] = new
            qs = q[hd] / 4.0
            o = S[hd].T @ qs / (max(abs(float(n[hd] @ qs)), math.exp(-new)) + 1e-6)
            out.append(o / rms(o, eps))
        z = np.concatenate(out) * w[p + "norm"] / (1.0 + np.exp(-(w[p + "g"] @ h[t])))
        assert np.allclose(got[t], w[p + "o"] @ z, atol=1e-9)
    # attention: q and k normed per head before the rotation of the first numbers
    m, p = C.CASE_A["layers"][2]["mixer"], "l2.mix."
    got = P.attention_mixer(h, w, p, m, pos, eps)
    t, first = 27, 20
    unit = lambda r, name: r / rms(r, eps) * w[p + name]
    out = []
    for hd in range(6):
        g = hd // 3
        q = unit(w[p + "q"][hd * 24:(hd + 1) * 24] @ h[t], "q.norm")
        e, vs = [], []
        for j in range(first, t + 1):
            k = unit(w[p + "k"][g * 24:(g + 1) * 24] @ h[j], "k.norm")
            turn = lambda a, at: P.rotate_half(a[None, None], np.array([at]), m["rot"])[0, 0]
            e.append(math.exp(m["scale"] * float(turn(q, t) @ turn(k, j))))
            vs.append(w[p + "v"][g * 16:(g + 1) * 16] @ h[j])
        out.append(sum(a * b for a, b in zip(e, vs)) / sum(e))
    assert np.allclose(got[t], w[p + "o"] @ np.concatenate(out), atol=1e-9)


def test_norms_sit_on_the_outputs_and_the_model_is_causal():
    cfg = C.CASE_C
    w, eps = weights(cfg), cfg["norm"]["eps"]
    ids = C.prompts(cfg["vocab"], [14], seed=1)[0]
    logits, layers = P.forward(ids, w, cfg, return_layers=True)
    x = w["embed"][np.asarray(ids)] * 0.7
    ln = lambda y, name: P.layer_norm(y, w[name], w[name + ".b"], eps)
    x = x + ln(P.attention_mixer(x, w, "l0.mix.", cfg["layers"][0]["mixer"], np.arange(14), eps), "l0.norm1")
    x = x + ln(P.experts_ff(x, w, "l0.mlp.", cfg["layers"][0]["mlp"]), "l0.norm2")          # reads x itself
    assert np.allclose(layers[0], x, atol=1e-12)
    assert np.allclose(logits, ln(layers[-1], "final.norm") @ w["head"].T, atol=1e-12)
    other = list(ids)
    other[9] = (ids[9] + 1) % cfg["vocab"]
    moved = P.forward(other, w, cfg)
    assert np.allclose(moved[:9], logits[:9], atol=1e-12) and not np.allclose(moved[9:], logits[9:], atol=1e-6)


# ---- the package's side, without a GPU ------------------------------------------------------------------

@pytest.mark.parametrize("name", sorted(C.CASES))
def test_configuration_round_trip_and_tensor_list(name):
    from railgun_b200.config.bunudra import BunudraConfig
    from railgun_b200.config.registry import architecture_of
    from railgun_b200.parts.model import expected_tensors
    from railgun_b200.weights.loader import load_weights, shapes_match
    cfg = C.CASES[name][0]
    typed = BunudraConfig.from_dict(json.loads(json.dumps(cfg)))
    assert typed.to_dict() == cfg
    arch = architecture_of("Bunudra")
    spec = arch.model_spec(typed)
    expected = expected_tensors(spec)
    made = C.random_tensors(cfg, 0)
    assert set(expected) == set(made)
    assert all(shapes_match(expected[k].shape, made[k].shape) for k in made)
    assert all(L.arrangement == "postnorm" for L in spec.layers)
    assert [len(L.branches()) for L in spec.layers] == [2 if c["mlp"] else 1 for c in cfg["layers"]]
    loaded = load_weights(C.model_dir(name), expected)
    assert set(loaded) == set(made) and all(tuple(loaded[k].shape) == made[k].shape for k in made)


def test_configuration_errors():
    from railgun_b200.config.base import ConfigError
    from railgun_b200.config.bunudra import BunudraConfig
    good = json.loads(json.dumps(C.CASE_A))

    def broken(change):
        c = json.loads(json.dumps(good))
        change(c)
        with pytest.raises(ConfigError):
            BunudraConfig.from_dict(c)

    mixer = lambda c, i: c["layers"][i]["mixer"]
    broken(lambda c: c.pop("width"))
    broken(lambda c: c.pop("norm"))
    broken(lambda c: c.update(layers=[]))
    broken(lambda c: c["layers"][0].update(type="lstm"))
    broken(lambda c: mixer(c, 0).pop("gate_cap"))
    broken(lambda c: mixer(c, 0).update(gate_cap=0.0))
    broken(lambda c: mixer(c, 1).pop("mask"))
    broken(lambda c: mixer(c, 1)["mask"].update(size=0))
    broken(lambda c: mixer(c, 1)["rot"].update(dims=18))
    broken(lambda c: mixer(c, 1)["rot"]["scaling"].pop("slow"))
    broken(lambda c: mixer(c, 1).pop("kv_rank"))
    broken(lambda c: mixer(c, 1).pop("scale"))
    broken(lambda c: mixer(c, 2).update(kv_heads=4))
    broken(lambda c: mixer(c, 2)["rot"].update(dims=15))
    broken(lambda c: mixer(c, 2)["rot"].update(scaling=dict(factor=2.0, original=64.0, fast=8.0, slow=1.0)))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4))
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=5))


def test_cache_needs_of_the_design():
    """A memory is a matrix, a vector and a number per head in 32-bit; a latent's page holds one row a token; pages of a
    complete chunk are given back, those of an open one are not."""
    import torch
    from railgun_b200.cache.manager import CacheError, CacheManager, PageAllocator
    from railgun_b200.parts.attention import NormedAttention
    from railgun_b200.parts.latent_attention import LatentAttention
    from railgun_b200.parts.mlstm import MLSTM
    S, m = MLSTM.cache_need(dict(num_heads=3, head_dim=10, v_dim=7))
    assert (S.shape, S.dtype, m.shape, m.dtype) == ((3, 8, 10), "float32", (3,), "float32")
    lat = LatentAttention.cache_need(dict(kv_rank=20, rot_dim=6, window=9))
    assert lat.window == 9 and lat.shape_of_page(8) == (8, 26)
    att = NormedAttention.cache_need(dict(hidden_size=8, num_heads=2, num_kv_heads=1, head_dim=16, v_dim=16, chunk=10))
    assert att.chunk == 10 and att.window == 0
    cm = CacheManager({0: att, 1: lat}, 4, 64, 2, torch.float32, "cpu")
    g = [i for i, info in enumerate(cm.groups) if info.need.chunk][0]
    cm.alloc.add_request(5)
    held = lambda: [j for j, p in enumerate(cm.alloc.block_table(5, g)) if p >= 0]
    seen = {}
    for n in range(1, 41):
        cm.alloc.reserve(5, n)
        cm.alloc.commit(5, n)
        # positions up to n are still needed from the chunk of the NEXT position on
        first = n // 10 * 10
        seen[n] = held()
        assert seen[n] == list(range(first // 4, -(-n // 4)))
    assert seen[10] == [2] and seen[20] == [] and seen[19] == [2, 3, 4]        # page 2 holds positions 8 to 11
    cm.alloc.release(5)
    cm.alloc.check()
    with pytest.raises(CacheError):
        PageAllocator([4], [8], [6], 2, chunks=[10])                           # a window or chunks, not both


def test_registry_knows_the_design(tmp_path):
    from railgun_b200.config.registry import known_architectures, load_config
    assert "Bunudra" in known_architectures()
    (tmp_path / "config.json").write_text(json.dumps(C.CASE_B))
    arch, cfg = load_config(tmp_path)
    assert arch.name == "Bunudra" and cfg.width == 96 and cfg.layers[0].mixer.size == 1 and cfg.layers[0].mixer.rot.scaling is None
    assert cfg.layers[2].mlp is None and cfg.layers[0].mlp.shared_ff == 0 and cfg.layers[0].mlp.groups == (2, 2)
    assert arch.allow_unexpected(cfg) == ("l2.norm2", "l2.norm2.b")
