"""The plain statement of Sagizen against loop-level formulas, and the package's
configuration, description and tensor list for the design (no GPU)."""
import json
import math

import numpy as np
import pytest

import plain_sagizen as P
import sagizen_cases as C


def weights(cfg, seed=1):
    return {k: v.astype(np.float64) for k, v in C.random_tensors(cfg, seed).items()}


def rms(x, eps):
    return math.sqrt(float((np.asarray(x) ** 2).mean()) + eps)


def test_token_shift_reads_the_token_before_it():
    rng = np.random.default_rng(0)
    x, share = rng.normal(size=(5, 4)), np.array([0.0, 1.0, 0.25, -0.5])
    got = P.token_shift(x, share)
    for t in range(5):
        before = x[t - 1] if t else np.zeros(4)
        assert np.allclose(got[t], (1.0 - share) * x[t] + share * before, atol=1e-14)
    assert np.array_equal(got[:, 0], x[:, 0]) and got[0, 1] == 0.0 and np.allclose(got[1:, 1], x[:-1, 1])


def test_causal_convolution_has_a_bias_and_its_last_column_is_now():
    rng = np.random.default_rng(1)
    x, taps, bias = rng.normal(size=(9, 5)), rng.normal(size=(5, 4)), rng.normal(size=5)
    got = P.causal_conv(x, taps, bias)
    for t in range(9):
        ref = bias.copy()
        for j in range(4):
            s = t - 3 + j
            if s >= 0:
                ref += taps[:, j] * x[s]
        assert np.allclose(got[t], ref, atol=1e-12)
    one = np.zeros((4, 1)); one[0, 0] = 1.0
    assert np.allclose(P.causal_conv(one, np.array([[1.0, 2.0, 3.0]]), [10.0])[:, 0], [13.0, 12.0, 11.0, 10.0])


def test_rotation_pairs_halves_and_scales_the_angle():
    rng = np.random.default_rng(2)
    x = rng.normal(size=(4, 2, 12))
    pos = np.array([0, 1, 300, 4000])
    for dims, factor in ((4, 1.0), (12, 4.0)):
        got = P.rotate_half(x, pos, dims, 50.0, factor)
        n = dims // 2
        for t in range(4):
            for i in range(n):
                a = pos[t] * 50.0 ** (-2.0 * i / dims) / factor
                for h in range(2):
                    u, v = x[t, h, i], x[t, h, i + n]
                    assert abs(got[t, h, i] - (u * math.cos(a) - v * math.sin(a))) < 1e-12
                    assert abs(got[t, h, i + n] - (v * math.cos(a) + u * math.sin(a))) < 1e-12
        assert np.array_equal(got[..., dims:], x[..., dims:])
        # a rotation leaves a head's root mean square alone: normed before or after is the same
        assert np.allclose(P.rotate_half(P.unit_rms(x, 1e-5), pos, dims, 50.0, factor), P.unit_rms(got, 1e-5), atol=1e-12)
    assert np.allclose(P.rotate_half(x, 4 * pos, 8, 50.0, 4.0), P.rotate_half(x, pos, 8, 50.0), atol=1e-9)


@pytest.mark.parametrize("size,pool", [(1, 1), (4, 3), (3, 4), (5, 5), (6, 1), (2, 9)])
def test_pooled_window_against_loops(size, pool):
    """Which tokens and blocks a query sees, one by one."""
    rng = np.random.default_rng(size * 10 + pool)
    T, H, G, d, dv = 23, 4, 2, 5, 3
    q, k, v = rng.normal(size=(T, H, d)), rng.normal(size=(T, G, d)), rng.normal(size=(T, G, dv))
    got = P.pooled_window_attention(q, k, v, 0.7, size, pool)
    unseen_before_window = 0
    for i in range(T):
        keys = [([j], j) for j in range(T) if 0 <= i - j < size]
        blocks, b = [], 0
        while b * pool + pool - 1 <= i - size:
            blocks.append(list(range(b * pool, (b + 1) * pool)))
            b += 1
        seen = set(sum(blocks, [])) | {j for _, j in keys}
        unseen_before_window += len(set(range(i + 1)) - seen)
        assert not set(sum(blocks, [])) & {j for _, j in keys}
        for h in range(H):
            g = h // 2
            e, vs = [], []
            for js in blocks + [a for a, _ in keys]:
                e.append(math.exp(0.7 * float(q[i, h] @ (sum(k[j, g] for j in js) / len(js)))))
                vs.append(sum(v[j, g] for j in js) / len(js))
            ref = sum(a * b for a, b in zip(e, vs)) / sum(e)
            assert np.allclose(got[i, h], ref, atol=1e-12)
    assert (unseen_before_window == 0) == (pool == 1)      # tokens between the last whole block and the window


def test_recurrences_against_their_sums_and_from_a_state():
    rng = np.random.default_rng(4)
    T, H, d, dv = 9, 3, 4, 5
    r, k, v = rng.normal(size=(T, H, d)), rng.normal(size=(T, H, d)), rng.normal(size=(T, H, dv))
    w, u = rng.uniform(0.3, 1.0, size=(T, H, d)), rng.normal(size=(H, d))
    o, S = P.rwkv_scan(r, k, v, w, u)
    for t in range(T):
        for h in range(H):
            ref = float((r[t, h] * u[h]) @ k[t, h]) * v[t, h]
            for s in range(t):
                decay = np.prod(w[s + 1:t, h], axis=0)       # nothing of token s is decayed by its own or by this w
                ref = ref + float((r[t, h] * decay) @ k[s, h]) * v[s, h]
            assert np.allclose(o[t, h], ref, atol=1e-12)
    o1, S1 = P.rwkv_scan(r[:4], k[:4], v[:4], w[:4], u)
    o2, S2 = P.rwkv_scan(r[4:], k[4:], v[4:], w[4:], u, S1)
    assert np.allclose(np.concatenate([o1, o2]), o, atol=1e-12) and np.allclose(S2, S, atol=1e-12)

    G, H, N = 2, 4, 6
    x, dt = rng.normal(size=(T, H, dv)), rng.uniform(0.01, 2.0, size=(T, H))
    A_log, B, Cc = rng.normal(size=H), rng.normal(size=(T, G, N)), rng.normal(size=(T, G, N))
    o, S = P.ssd_scan(x, dt, A_log, B, Cc)
    for t in range(T):
        for h in range(H):
            ref = sum(math.exp(-math.exp(A_log[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * float(Cc[t, h // 2] @ B[s, h // 2])
                      * x[s, h] for s in range(t + 1))
            assert np.allclose(o[t, h], ref, atol=1e-12)
    o1, S1 = P.ssd_scan(x[:4], dt[:4], A_log, B[:4], Cc[:4])
    o2, S2 = P.ssd_scan(x[4:], dt[4:], A_log, B[4:], Cc[4:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o, atol=1e-12) and np.allclose(S2, S, atol=1e-12)


def test_mixers_against_loops():
    cfg = C.CASE_A
    w, eps = weights(cfg), cfg["norm"]["eps"]
    rng = np.random.default_rng(5)
    T = 14
    h = rng.normal(size=(T, cfg["width"]))
    # Mamba-2: the order z | x | B | C | dt, the gate before the norm, D on the convolved x
    m, p = cfg["layers"][1]["mixer"], "l1.mix."
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    got = P.mamba2_mixer(h, w, p, m, eps)
    rows = h @ w[p + "in"].T
    conv = P.silu(P.causal_conv(rows[:, inner:2 * inner + 2 * G * N], w[p + "conv"], w[p + "conv.b"]))
    S = np.zeros((H, N, dv))
    for t in range(T):
        y = np.zeros(inner)
        for hd in range(H):
            g = hd // (H // G)
            x = conv[t, hd * dv:(hd + 1) * dv]
            B, Cc = conv[t, inner + g * N:inner + (g + 1) * N], conv[t, inner + (G + g) * N:inner + (G + g + 1) * N]
            dt = math.log1p(math.exp(rows[t, 2 * inner + 2 * G * N + hd] + w[p + "dt_bias"][hd]))
            S[hd] = math.exp(-math.exp(w[p + "A_log"][hd]) * dt) * S[hd] + dt * np.outer(B, x)
            y[hd * dv:(hd + 1) * dv] = S[hd].T @ Cc + w[p + "D"][hd] * x
        y = y * P.silu(rows[t, :inner])
        n = inner // m["norm_groups"]
        y = np.concatenate([y[i:i + n] / rms(y[i:i + n], eps) for i in range(0, inner, n)])
        assert np.allclose(got[t], w[p + "o"] @ (y * w[p + "norm"]), atol=1e-10)
    # time mixing: five mixes of their own, the norm per head before weight and gate
    m, p = cfg["layers"][0]["mixer"]["right"], "l0.mix.right."
    H, d = m["heads"], m["dim"]
    got = P.rwkv_mixer(h, w, p, m, eps)
    S = np.zeros((H, d, d))
    for t in range(T):
        before = h[t - 1] if t else np.zeros_like(h[t])
        mx = {s: h[t] + (before - h[t]) * w[p + "mu." + s] for s in "rkvgw"}
        r, k, v = (w[p + s] @ mx[s] for s in "rkv")
        wt = np.exp(-np.exp(w[p + "w2"] @ np.tanh(w[p + "w1"] @ mx["w"]) + w[p + "w0"]))
        out = []
        for hd in range(H):
            sl = slice(hd * d, (hd + 1) * d)
            o = np.array([sum(r[sl][i] * (S[hd, i, j] + w[p + "u"][hd, i] * k[sl][i] * v[sl][j]) for i in range(d))
                          for j in range(d)])
            S[hd] = wt[sl][:, None] * S[hd] + np.outer(k[sl], v[sl])
            out.append(o / rms(o, eps))
        gate = P.silu(w[p + "g"] @ mx["g"])
        assert np.allclose(got[t], w[p + "o"] @ (np.concatenate(out) * w[p + "norm"] * gate), atol=1e-10)
    # both halves, each times its constant; biases on q, k and v only, q and k of root mean square one
    m = cfg["layers"][0]["mixer"]
    a = P.pooled_attention(h, w, "l0.mix.left.", m["left"], np.arange(T), eps)
    assert np.allclose(P.parallel_mixer(h, w, "l0.mix.", m, np.arange(T), eps), 0.7 * a + 1.3 * got, atol=1e-12)
    zero = P.pooled_attention(h * 0.0, w, "l0.mix.left.", m["left"], np.arange(T), eps)
    v0 = np.repeat(w["l0.mix.left.v.b"].reshape(2, -1), 2, axis=0).reshape(-1)
    assert np.allclose(zero, w["l0.mix.left.o"] @ v0, atol=1e-12)


def test_norms_sit_on_the_outputs_and_the_model_is_causal():
    cfg = C.CASE_C
    w, eps = weights(cfg), cfg["norm"]["eps"]
    ids = C.prompts(cfg["vocab"], [14], seed=1)[0]
    logits, layers = P.forward(ids, w, cfg, return_layers=True)
    x = w["embed"][np.asarray(ids)]
    h = P.token_shift(x, w["l0.shift"])
    y = P.mamba2_mixer(h, w, "l0.mix.", cfg["layers"][0]["mixer"], eps)
    x = x + np.stack([r / rms(r, eps) for r in y]) * w["l0.norm1"]
    f = (P.silu(x @ w["l0.mlp.gate"].T) * (x @ w["l0.mlp.up"].T)) @ w["l0.mlp.down"].T      # reads x itself, not shifted
    x = x + np.stack([r / rms(r, eps) for r in f]) * w["l0.norm2"]
    assert np.allclose(layers[0], x, atol=1e-12)
    assert np.allclose(logits, P.rms_norm(layers[-1], w["final.norm"], eps) @ w["head"].T, atol=1e-12)
    other = list(ids)
    other[9] = (ids[9] + 1) % cfg["vocab"]
    moved = P.forward(other, w, cfg)
    assert np.allclose(moved[:9], logits[:9], atol=1e-12) and not np.allclose(moved[9:], logits[9:], atol=1e-6)


# ---- the package's side, without a GPU ------------------------------------------------------------------

@pytest.mark.parametrize("name", sorted(C.CASES))
def test_configuration_round_trip_and_tensor_list(name):
    from railgun_b200.config.registry import architecture_of
    from railgun_b200.config.sagizen import SagizenConfig
    from railgun_b200.parts.model import expected_tensors
    from railgun_b200.weights.loader import load_weights, shapes_match
    cfg = C.CASES[name][0]
    typed = SagizenConfig.from_dict(json.loads(json.dumps(cfg)))
    assert typed.to_dict() == cfg
    arch = architecture_of("Sagizen")
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
    from railgun_b200.config.sagizen import SagizenConfig
    good = json.loads(json.dumps(C.CASE_A))

    def broken(change):
        c = json.loads(json.dumps(good))
        change(c)
        with pytest.raises(ConfigError):
            SagizenConfig.from_dict(c)

    broken(lambda c: c.pop("width"))
    broken(lambda c: c.pop("norm"))
    broken(lambda c: c.update(layers=[]))
    broken(lambda c: c["layers"][0].update(type="mamba"))
    broken(lambda c: c["layers"][0]["mixer"].pop("right"))
    broken(lambda c: c["layers"][0]["mixer"].pop("left_scale"))
    broken(lambda c: c["layers"][0]["mixer"]["left"].pop("mask"))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(pool=0))
    broken(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0))
    broken(lambda c: c["layers"][1]["mixer"].update(groups=3))
    broken(lambda c: c["layers"][1]["mixer"].update(norm_groups=3))
    broken(lambda c: c["layers"][1]["mixer"].pop("conv"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))


def test_sizes_that_only_the_files_give(tmp_path):
    """The decay's rank is no key of config.json: any rank loads; other shapes are still held to."""
    from railgun_b200.config.sagizen import SagizenConfig
    from railgun_b200.config.registry import architecture_of
    from railgun_b200.parts.model import expected_tensors
    from railgun_b200.weights.loader import AnySize, WeightError, load_weights, shapes_match
    assert shapes_match((AnySize(64), 4), (3, 4)) and not shapes_match((AnySize(64), 4), (3, 5))
    assert not shapes_match((AnySize(64), 4), (4,)) and not shapes_match((64, 4), (3, 4))
    cfg = C.CASE_B
    expected = expected_tensors(architecture_of("Sagizen").model_spec(SagizenConfig.from_dict(cfg)))

    def wrong(t):
        t["l1.mix.right.w1"] = t["l1.mix.right.w1"][:, :-8]
    folder = C.write_model(cfg, 1, tmp_path / "wrong", change=wrong)
    with pytest.raises(WeightError):
        load_weights(folder, expected)


def test_cache_needs_of_the_design():
    """Window pages are kept until their block is complete; pooled pages cover page_size * pool tokens and there is one
    more of them than the pool's tokens fill for every live request."""
    from railgun_b200.cache.manager import CacheManager, PagedKVNeed
    from railgun_b200.parts.attention import NormedAttention
    base = dict(hidden_size=8, num_heads=2, num_kv_heads=1, head_dim=16, v_dim=16)
    pages, blocks = NormedAttention.cache_need(dict(base, window=4, pool=9))
    assert pages.window == 9 and pages.tokens_per_entry == 1 and blocks.window == 0 and blocks.tokens_per_entry == 9
    assert NormedAttention.cache_need(dict(base, window=40, pool=9))[0].window == 40
    assert isinstance(NormedAttention.cache_need(dict(base, window=4)), PagedKVNeed)
    import torch
    cm = CacheManager({0: (pages, blocks)}, 4, 100, 3, torch.float32, "cpu")
    tok, ent = cm.groups
    assert (tok.page_size, tok.num_pages) == (4, 25) and (ent.page_size, ent.num_pages) == (36, 3 + 3)
    assert tuple(cm.kv[(0, 0)].shape) == (25, 2, 1, 4, 16) and tuple(cm.kv[(0, 1)].shape) == (6, 2, 1, 4, 16)
    # three requests fill the token pool to the brim; the entries' group has room for each one's partly filled page
    for rid, n in ((1, 40), (2, 40), (3, 20)):
        cm.alloc.add_request(rid)
        cm.alloc.reserve(rid, n)
        cm.alloc.commit(rid, n)
    assert [len(cm.alloc.block_table(r, 1)) for r in (1, 2, 3)] == [2, 2, 1]
    assert list(cm.alloc.block_table(1, 0))[:8] == [-1] * 8 and cm.alloc.block_table(1, 0)[8] >= 0   # 40 - 9 + 1 = 32
    for rid in (1, 2, 3):
        cm.alloc.release(rid)
    cm.alloc.check()


def test_registry_knows_the_design(tmp_path):
    from railgun_b200.config.registry import known_architectures, load_config
    assert "Sagizen" in known_architectures()
    (tmp_path / "config.json").write_text(json.dumps(C.CASE_B))
    arch, cfg = load_config(tmp_path)
    assert arch.name == "Sagizen" and cfg.width == 96 and cfg.layers[1].mixer.left.pool == 1
    assert cfg.layers[1].ff == 0 and cfg.layers[1].mixer.left.rot_dims == 0 and cfg.layers[2].mixer.left.rot_factor == 1.0
    assert arch.allow_unexpected(cfg) == ("l1.norm2",)
