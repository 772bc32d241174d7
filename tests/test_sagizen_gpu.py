"""Sagizen on the GPU against the plain statement: each mechanism alone, then
the model through the step function in several cuts and both precisions, then
generation through the engine, its scheduler and the command line."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import helpers
import plain_sagizen as P
import sagizen_cases as C

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = torch.device("cuda:0")
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# bfloat16: the test weights are several times larger than a trained model's, so rounding alone moves logits by some
# 1e-2 of the largest, the same in every cut; a lost key, block, state or tap is caught by the tests of the mechanisms
# alone, where it changes a row by its whole size.
TOL = {"float32": 5e-5, "bfloat16": 6e-2}


def rel(got, ref):
    got = got.double().cpu().numpy() if isinstance(got, torch.Tensor) else np.asarray(got, dtype=np.float64)
    ref = ref.double().cpu().numpy() if isinstance(ref, torch.Tensor) else np.asarray(ref, dtype=np.float64)
    return np.abs(got - ref).max() / np.abs(ref).max()


def dev(x, dtype=None):
    t = torch.as_tensor(x)
    return t.to(DEV, dtype=dtype) if dtype is not None else t.to(DEV)


def step_batch(lengths, starts, slots):
    """What the kernels read of a step: requests packed one after another."""
    cu = np.concatenate([[0], np.cumsum(lengths)]).astype(np.int32)
    return SimpleNamespace(cu_seqlens=dev(cu), num_requests=len(lengths), decode_only=max(lengths) == 1,
                           req_of_token=dev(np.repeat(np.arange(len(lengths)), lengths).astype(np.int32)),
                           start_pos=dev(np.asarray(starts, dtype=np.int32)),
                           state_slots=dev(np.asarray(slots, dtype=np.int32)),
                           positions=dev(np.concatenate([s + np.arange(n) for s, n in zip(starts, lengths)]).astype(np.int32)))


def split(lengths):
    at = np.concatenate([[0], np.cumsum(lengths)])
    return [slice(a, b) for a, b in zip(at[:-1], at[1:])]


# ---- the stream: norm behind a part, addition, token shift -------------------------------------------------

STEPS = [([5], [0], [1]), ([1, 1, 1, 1], [7, 0, 3, 9], [2, 0, 3, -1]), ([40, 1, 9, 2], [0, 33, 12, 0], [2, 0, 3, 1]),
         ([2100, 1, 420], [5, 8, 0], [1, 2, 0])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [24, 41, 256, 2052])
@pytest.mark.parametrize("step", range(len(STEPS)))
def test_postnorm_and_token_shift_alone(step, W, dtype):
    """x + w unit(y), then the row mixed with the request's row before it: inside the step, from the slot, or zeros at
    position 0 whatever the slot holds.  The slot is left with the step's last row, other slots are left alone."""
    from railgun_b200 import ops
    lengths, starts, slots = STEPS[step]
    rng = np.random.default_rng(W + step)
    T = sum(lengths)
    x = torch.tensor(rng.normal(size=(T, W)), dtype=torch.float32)
    y = torch.tensor(rng.normal(size=(T, W)) * rng.choice([0.01, 30.0], size=(T, 1)), dtype=TORCH[dtype])
    w, share = rng.uniform(0.5, 2, size=W), rng.uniform(-0.3, 1.2, size=W)
    state0 = rng.normal(size=(4, 1, W))
    batch = step_batch(lengths, starts, slots)
    for pending in ("normed", "plain", None):
        state = dev(state0, torch.float32)
        p = dict(normed=ops.PendingNormed(dev(y), dev(w, torch.float32), 1e-5), plain=dev(y)).get(pending)
        resid = dev(x)
        new, h = ops.postnorm_shift(resid, p, dev(share, torch.float32), state, batch, TORCH[dtype])
        ref = x.double().numpy()
        if pending:
            ref = ref + (P.rms_norm(y.double().numpy(), w, 1e-5) if pending == "normed" else y.double().numpy())
        assert rel(new, ref) < 2e-6 and torch.equal(resid.cpu(), x)
        want_state = state0.astype(np.float32).astype(np.float64)
        for sl, start, slot in zip(split(lengths), starts, slots):
            first = want_state[slot] if start and slot >= 0 else np.zeros((1, W))
            before = np.concatenate([first, ref[sl][:-1]])
            assert rel(h[sl], ref[sl] + (before - ref[sl]) * share) < (3e-6 if dtype == "float32" else 8e-3)
            if slot >= 0:
                want_state[slot] = ref[sl][-1:]
        assert rel(state, want_state) < 2e-6
        same, out = ops.postnorm_shift(resid, p, None, None, None, TORCH[dtype])              # no shift: in place
        assert same is resid and rel(resid, ref) < 2e-6 and rel(out, ref) < (2e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [24, 41, 1028])
@pytest.mark.parametrize("step", range(len(STEPS)))
def test_five_mixes_alone(step, W, dtype):
    from railgun_b200 import ops
    lengths, starts, slots = STEPS[step]
    rng = np.random.default_rng(W + step)
    T = sum(lengths)
    h = torch.tensor(rng.normal(size=(T, W)), dtype=TORCH[dtype])
    mu, state0 = rng.uniform(-0.3, 1.2, size=(5, W)), rng.normal(size=(4, 1, W))
    state = dev(state0, torch.float32)
    mixes, last = ops.shift_mixes(dev(h), dev(mu, torch.float32), state, step_batch(lengths, starts, slots))
    x, want_state = h.double().numpy(), state0.astype(np.float32).astype(np.float64)
    before = np.zeros_like(x)
    for sl, start, slot in zip(split(lengths), starts, slots):
        before[sl] = np.concatenate([want_state[slot] if start and slot >= 0 else np.zeros((1, W)), x[sl][:-1]])
        if slot >= 0:
            want_state[slot] = x[sl][-1:]
    for s in range(4):
        assert rel(mixes[s], x + (before - x) * mu[s]) < (2e-6 if dtype == "float32" else 5e-3)
    if dtype == "bfloat16":
        assert last.shape == (T, 2 * W)
        last = last[:, :W].double() + last[:, W:].double()                     # the two halves: 32-bit precision
    assert rel(last, x + (before - x) * mu[4]) < 2e-5 and rel(state, want_state) < 1e-7


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,N,rank", [(1, 12, 3), (5, 70, 64), (64, 64, 16), (65, 130, 65), (300, 33, 200)])
def test_lowrank_decay_alone(T, N, rank, dtype):
    """Decays near zero and near one alike, each to its own size."""
    from railgun_b200 import ops
    rng = np.random.default_rng(T + N)
    a = torch.tensor(rng.normal(size=(T, rank)) * 1.5, dtype=torch.float32)
    w = torch.tensor(rng.normal(size=(N, rank)) * 0.5 / rank ** 0.5, dtype=TORCH[dtype])
    w0 = torch.tensor(np.linspace(-9.0, 2.0, N), dtype=torch.float32)
    got = ops.lowrank_decay(dev(a), dev(w), dev(w0)).double().cpu().numpy()
    z = np.tanh(a.double().numpy()) @ w.double().numpy().T + w0.double().numpy()
    assert np.abs(np.log(np.maximum(got, 1e-30)) / -np.exp(z) - 1.0)[np.exp(z) > 1e-2].max() < 1e-4
    assert np.abs(got - np.exp(-np.exp(z))).max() < 2e-6


# ---- the matrix states ---------------------------------------------------------------------------------------

@pytest.mark.parametrize("H,d,dv", [(1, 10, 10), (3, 12, 12), (2, 7, 7), (4, 64, 64), (2, 128, 128), (1, 200, 40), (2, 256, 256)])
@pytest.mark.parametrize("form", ["tokens", "chunks"])
def test_scan_with_a_decay_per_channel(form, H, d, dv):
    """S carried in the slot from an earlier step beside a new request in a dirty slot and a single token; the current
    token counts through the bonus only and is decayed by nobody; a far key made loud is still heard; channels that
    forget at once (a decay of exactly 0) and never (1).  Token by token, and in chunks side by side (whole ones, ends of
    one token and more, requests of less than one)."""
    from railgun_b200 import ops
    rng = np.random.default_rng(H + d)
    lengths, starts, slots = ([40, 75, 1], [0, 33, 9], [2, 0, 3]) if form == "tokens" else (
        [64, 129, 1, 200, 63], [0, 33, 9, 5, 0], [2, 0, 3, 4, -1])
    T, at = sum(lengths), lengths[0]
    r, k, v = (torch.tensor(rng.normal(size=(T, H * n)) * 0.5, dtype=torch.float32) for n in (d, d, dv))
    w = np.exp(-np.exp(rng.uniform(-6.0, 0.0, size=(T, H * d))))
    w[:, 1], w[:, 2], w[7::9, 3] = 0.0, 1.0, 0.0
    w[at:, 4:d] = np.maximum(w[at:, 4:d], 0.99)
    w = torch.tensor(w, dtype=torch.float32)
    far, ask = at + 5, at + lengths[1] - 1
    k[far, :d], r[ask, :d] = 3.0, 3.0                                          # a loud key, and the query that asks for it
    u = rng.normal(size=(H, d))
    state0 = rng.normal(size=(5, H, dv, d)) * 0.3
    state = dev(state0, torch.float32)
    batch = step_batch(lengths, starts, slots)
    if form == "tokens":
        o = ops.state_scan(dev(r), dev(k), dev(v), state, batch, H, d, dv, rule="channel", w=dev(w), bonus=dev(u, torch.float32))
    else:
        o = ops.channel_chunk_scan(dev(r), dev(k), dev(v), dev(w), dev(u, torch.float32), state, batch, H, d, dv)
    f = lambda t, n: t.double().numpy().reshape(T, H, n)
    refs = []
    for sl, start, slot in zip(split(lengths), starts, slots):
        S0 = None if start == 0 or slot < 0 else np.transpose(state0[slot], (0, 2, 1))
        ro, S = P.rwkv_scan(f(r, d)[sl], f(k, d)[sl], f(v, dv)[sl], f(w, d)[sl], u, S0)
        refs.append(ro)
        if slot >= 0:
            assert rel(state[slot], np.transpose(S, (0, 2, 1))) < 3e-5
    ref = np.concatenate(refs)
    assert rel(o, ref) < 3e-5 and rel(state[1], state0[1]) < 1e-7
    assert np.abs(ref[ask, 0]).max() > 3 * np.median(np.abs(ref[:, 0]))


@pytest.mark.parametrize("H,G,N,dv", [(1, 1, 9, 6), (6, 3, 16, 8), (4, 2, 24, 16), (5, 5, 10, 6), (8, 2, 128, 64), (2, 1, 200, 40),
                                      (3, 1, 256, 256)])
@pytest.mark.parametrize("form", ["tokens", "chunks"])
def test_scan_with_step_sizes(form, H, G, N, dv):
    """The state-space duality form: a decay and a step size per token and head, B and C shared by a group's heads,
    D on the token's own x; token by token, and in chunks side by side (whole ones, ends of one token and more, requests
    of less than one, heads that forget within a few tokens)."""
    from railgun_b200 import ops
    rng = np.random.default_rng(H + N)
    lengths, starts, slots = ([40, 75, 1], [0, 33, 9], [2, 0, 3]) if form == "tokens" else (
        [64, 129, 1, 200, 63], [5, 0, 9, 33, 0], [2, 0, 3, 4, -1])
    T = sum(lengths)
    xbc = torch.tensor(rng.normal(size=(T, H * dv + 2 * G * N)) * 0.5, dtype=torch.float32)
    raw = torch.tensor(rng.normal(size=(T, H)) * 2.0, dtype=torch.float32)
    bias, A, D = rng.uniform(-5, 1, size=H), rng.uniform(-3, 1, size=H), rng.normal(size=H)
    A[0] = 2.5
    dt, g = ops.ssd_prepare(dev(raw), dev(bias, torch.float32), dev(A, torch.float32))
    dt_ref = P.softplus(raw.double().numpy() + bias)
    assert rel(dt, dt_ref) < 1e-6 and np.abs(g.double().cpu().numpy() - np.exp(-np.exp(A) * dt_ref)).max() < 1e-6
    state0 = rng.normal(size=(5, H, dv, N)) * 0.3
    state = dev(state0, torch.float32)
    x = dev(xbc)
    inner = H * dv
    batch = step_batch(lengths, starts, slots)
    if form == "tokens":
        o = ops.state_scan(x[:, inner + G * N:], x[:, inner:inner + G * N], x[:, :inner], state, batch, H, N, dv, g=g, beta=dt,
                           rule="scalar", skip=dev(D, torch.float32))
    else:
        o = ops.ssd_chunk_scan(x, dt, dev(A, torch.float32), dev(D, torch.float32), state, batch, H, G, N, dv)
    xr = xbc.double().numpy()
    X, B, Cc = xr[:, :inner].reshape(T, H, dv), xr[:, inner:inner + G * N].reshape(T, G, N), xr[:, inner + G * N:].reshape(T, G, N)
    for sl, start, slot in zip(split(lengths), starts, slots):
        S0 = None if start == 0 or slot < 0 else np.transpose(state0[slot], (0, 2, 1))
        ro, S = P.ssd_scan(X[sl], dt_ref[sl], A, B[sl], Cc[sl], S0)
        ref = ro + D[None, :, None] * X[sl]
        for h in range(H):                                                     # every head to its own size
            assert rel(o[sl][:, h], ref[:, h]) < 3e-5
            if slot >= 0:
                assert rel(state[slot, h], S[h].T) < 3e-5
    assert rel(state[1], state0[1]) < 1e-7


def test_scans_of_the_other_designs_are_unchanged():
    """Retention and the delta rule through the same kernel."""
    from railgun_b200 import ops
    rng = np.random.default_rng(3)
    H, d, dv, T = 2, 24, 16, 30
    q, k, v = (rng.normal(size=(T, H, n)) * 0.4 for n in (d, d, dv))
    decay, g, beta = np.array([0.9, 0.99]), rng.uniform(0.8, 1.0, size=(T, H)), rng.uniform(0.1, 0.9, size=(T, H))
    batch = step_batch([T], [0], [0])
    f = lambda a: dev(a.reshape(T, -1), torch.float32)
    for rule in ("retention", "delta"):
        state = torch.zeros((1, H, dv, d), device=DEV)
        more = dict(decay=dev(decay, torch.float32)) if rule == "retention" else dict(g=f(g), beta=f(beta))
        o = ops.state_scan(f(q), f(k), f(v), state, batch, H, d, dv, **more)
        S, ref = np.zeros((H, d, dv)), np.zeros((T, H, dv))
        for t in range(T):
            for h in range(H):
                S[h] *= decay[h] if rule == "retention" else g[t, h]
                u = v[t, h] if rule == "retention" else beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
                S[h] += np.outer(k[t, h], u)
                ref[t, h] = S[h].T @ q[t, h]
        assert rel(o, ref) < 2e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dv,groups,T", [(4, 16, 1, 5), (6, 8, 3, 40), (3, 20, 5, 7), (2, 6, 2, 300), (32, 64, 2, 3), (8, 2000, 1, 2)])
def test_gate_before_a_norm_in_parts(H, dv, groups, T, dtype):
    """One loud part does not drown the others; the gate changes the root mean square."""
    from railgun_b200 import ops
    rng = np.random.default_rng(T + H)
    n = H * dv
    o = rng.normal(size=(T, n))
    o[:, :n // groups] *= 50.0
    o = torch.tensor(o, dtype=torch.float32)
    wide = torch.tensor(rng.normal(size=(T, n + 8)) * 2.0, dtype=TORCH[dtype])
    w = rng.uniform(0.5, 2, size=n)
    got = ops.gate_group_norm(dev(o).view(T, H, dv), dev(wide)[:, 8:], dev(w, torch.float32), 1e-5, groups, TORCH[dtype])
    y = o.double().numpy() * P.silu(wide[:, 8:].double().numpy())
    ref = P.unit_rms(y.reshape(T, groups, -1), 1e-5).reshape(T, n) * w
    for g in range(groups):
        sl = slice(g * n // groups, (g + 1) * n // groups)
        assert rel(got[:, sl], ref[:, sl]) < (3e-6 if dtype == "float32" else 8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_heads_norm_with_a_weight_per_head_and_a_constant(dtype):
    from railgun_b200 import ops
    rng = np.random.default_rng(0)
    for T, H, dv in ((5, 3, 12), (70, 1, 7), (3, 8, 64)):
        o = torch.tensor(rng.normal(size=(T, H, dv)) * rng.choice([0.1, 20.0], size=(T, H, 1)), dtype=torch.float32)
        gate, w = torch.tensor(rng.normal(size=(T, H * dv)), dtype=torch.float32), rng.uniform(0.5, 2, size=H * dv)
        out = torch.zeros((T, H * dv + 9), dtype=TORCH[dtype], device=DEV)
        ops.head_norm_gate(dev(o), dev(gate), dev(w, torch.float32), 1e-5, TORCH[dtype], out=out[:, 4:4 + H * dv], out_scale=0.3)
        ref = P.unit_rms(o.double().numpy(), 1e-5).reshape(T, -1) * w * P.silu(gate.double().numpy()) * 0.3
        assert rel(out[:, 4:4 + H * dv], ref) < (3e-6 if dtype == "float32" else 8e-3)
        assert float(out[:, :4].abs().max()) == 0.0 and float(out[:, 4 + H * dv:].abs().max()) == 0.0


@pytest.mark.parametrize("H,dv,N,G,K", [(4, 16, 24, 2, 4), (1, 48, 32, 1, 1), (5, 6, 10, 5, 5), (8, 64, 128, 2, 4), (3, 20, 130, 1, 2)])
def test_single_token_step_equals_the_plain_mixer(H, dv, N, G, K):
    """Token by token through the fused step (three live requests, one of them new in a dirty slot, and a padding row):
    convolution tails, step sizes, states, the gate and the norm."""
    from railgun_b200 import ops
    rng = np.random.default_rng(H + N)
    W, steps, inner = 32, 9, H * dv
    Cc = inner + 2 * G * N
    cfg = dict(heads=H, vdim=dv, state=N, groups=G, conv=K, norm_groups=2 if inner % 2 == 0 else 1)
    w = {"in": rng.normal(size=(inner + Cc + H, W)) * 0.2, "conv": rng.normal(size=(Cc, K)) * 0.5, "conv.b": rng.normal(size=Cc) * 0.3,
         "dt_bias": rng.uniform(-4, 0, size=H), "A_log": rng.uniform(-2, 1, size=H), "D": rng.normal(size=H),
         "norm": rng.uniform(0.5, 2, size=inner), "o": np.eye(inner)}
    w = {k: np.asarray(a, dtype=np.float32).astype(np.float64) for k, a in w.items()}
    hs = rng.normal(size=(3, steps, W)).astype(np.float32).astype(np.float64)
    refs = [P.mamba2_mixer(h, w, "", cfg, 1e-5) for h in hs]
    state = dev(rng.normal(size=(5, H, dv, N)), torch.float32)
    tail = dev(rng.normal(size=(5, max(1, K - 1), Cc)), torch.float32)
    untouched = state[1].clone()
    taps = dev(np.ascontiguousarray(w["conv"].T), torch.float32)
    f = lambda n: dev(w[n], torch.float32)
    slots = [4, 0, 2, -1]
    for t in range(steps):
        rows = np.concatenate([hs[:, t] @ w["in"].T, rng.normal(size=(1, inner + Cc + H))])
        proj = dev(rows, torch.float32)
        batch = step_batch([1] * 4, [t, t, t, 0], slots)
        o = ops.ssd_step(proj, inner, inner + Cc, taps, f("conv.b"), tail if K > 1 else None, f("dt_bias"), f("A_log"), f("D"),
                         state, batch, H, G, N, dv)
        y = ops.gate_group_norm(o, proj[:, :inner], f("norm"), 1e-5, cfg["norm_groups"], torch.float32,
                                conv=(proj[:, inner:inner + Cc], tail) if K > 1 else None, batch=batch)
        for b in range(3):
            assert rel(y[b], refs[b][t]) < 3e-5, f"request {b} token {t}"
    assert torch.equal(state[1], untouched)


# ---- pooled blocks ----------------------------------------------------------------------------------------------

def pages_of(x, page, D, dtype, order):
    """x = (k, v), [n, G, *] each, behind a block table."""
    k, v = x
    n, G = k.shape[:2]
    cache = torch.zeros((max(order) + 2, 2, G, page, D), dtype=dtype)
    for j in range(n):
        cache[order[j // page], 0, :, j % page, :k.shape[2]] = k[j].to(dtype)
        cache[order[j // page], 1, :, j % page, :v.shape[2]] = v[j].to(dtype)
    return cache


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("G,D,page,pool", [(2, 16, 8, 5), (1, 48, 16, 1), (3, 32, 4, 4), (2, 128, 16, 40), (1, 16, 64, 7)])
def test_pooled_entries_alone(G, D, page, pool, dtype):
    """Means over blocks that lie across page borders, completed by a portion and by single tokens (inside the per-token
    kernel); a padding row writes nothing; entries of blocks that are not complete stay as they were."""
    from railgun_b200 import ops
    rng = np.random.default_rng(page + pool)
    n = 3 * page * max(1, pool // page) + 3 * pool + 3
    k, v = (torch.tensor(rng.normal(size=(n, G, D)), dtype=TORCH[dtype]) for _ in range(2))
    pages = -(-n // page)
    order = rng.permutation(pages + 2)[:pages].tolist()
    cache, table = dev(pages_of((k, v), page, D, TORCH[dtype], order)), dev(torch.tensor([order], dtype=torch.int32))
    span = page * pool                                                         # tokens of a page of entries
    epages = -(-n // span)
    eorder = rng.permutation(epages + 1)[:epages]
    blank = torch.full((epages + 1, 2, G, page, D), -7.0, dtype=TORCH[dtype])
    eslot = lambda p: int(eorder[p // span]) * span + p % span
    ref = lambda x, b: x.double()[b * pool:(b + 1) * pool].mean(dim=0)
    start = pool + 1                                                           # block 0 was completed earlier
    entries = dev(blank)
    slots = torch.tensor([eslot(p) for p in range(start, n)], dtype=torch.int32)
    ops.pool_blocks(cache, table, step_batch([n - start], [start], [0]), dev(slots), entries, pool)
    done = [b for b in range(n // pool) if (b + 1) * pool - 1 >= start]
    assert len(done) >= 3
    want = blank.double().clone()
    for b in done:
        s = eslot(b * pool) // pool
        want[s // page, 0, :, s % page], want[s // page, 1, :, s % page] = ref(k, b), ref(v, b)
    assert rel(entries, want) < (1e-6 if dtype == "float32" else 5e-3)
    untouched = want == -7.0
    assert torch.equal(entries.cpu().double()[untouched], want[untouched])
    # the same from the per-token kernel, one token at a time (q, k and v without norm and rotation)
    entries, tok = dev(blank), torch.zeros_like(cache)
    freq = torch.zeros(1, dtype=torch.float64, device=DEV)
    for p in range(n):
        row = torch.cat([torch.zeros(1, G * D, dtype=TORCH[dtype]), k[p].reshape(1, -1), v[p].reshape(1, -1)], dim=1)
        rows = torch.cat([row, row])                                           # the second row is padding
        batch = step_batch([1, 1], [p, 0], [0, -1])
        s = dev(torch.tensor([order[p // page] * page + p % page, -1], dtype=torch.int32))
        es = dev(torch.tensor([eslot(p), -1], dtype=torch.int32))
        ops.attention_prepare(dev(rows), tok, None, None, 0.0, freq, 0, False, batch.positions, s, None, G, G, D, D, D,
                              pooled=(entries, es, pool, torch.cat([table, table]), batch))
    for b in range(n // pool):
        s = eslot(b * pool) // pool
        want[s // page, 0, :, s % page], want[s // page, 1, :, s % page] = ref(k, b), ref(v, b)
    assert rel(entries, want) < (1e-6 if dtype == "float32" else 5e-3)
    assert torch.equal(entries.cpu()[want == -7.0], blank[want == -7.0])


def test_bias_in_the_per_token_kernel():
    from railgun_b200 import ops
    from railgun_b200.parts.latent_attention import rotary_frequencies
    rng = np.random.default_rng(4)
    T, H, G, d, dv, D, dims, page = 6, 4, 2, 24, 40, 48, 16, 4
    x, bias = rng.normal(size=(T, (H + G) * d + G * dv)), rng.normal(size=(H + G) * d + G * dv)
    pos = np.array([0, 1, 5, 70000, 9, 2])
    cache = torch.zeros((2, 2, G, page, D), device=DEV)
    ones = torch.ones(d, device=DEV)
    q = ops.attention_prepare(dev(x, torch.float32), cache, ones, ones, 1e-5, (rotary_frequencies(dims, 300.0) / 3.0).to(DEV), dims,
                              False, dev(pos.astype(np.int32)), dev(torch.arange(T, dtype=torch.int32)), None, H, G, d, dv, D,
                              bias=dev(bias, torch.float32))
    y = x + bias
    rot = lambda a, heads: P.unit_rms(P.rotate_half(a.reshape(T, heads, d), pos, dims, 300.0, 3.0), 1e-5)   # rotate, then norm
    assert rel(q[:, :, :d], rot(y[:, :H * d], H)) < 5e-6
    flat = cache.permute(1, 2, 0, 3, 4).reshape(2, G, 2 * page, D)[:, :, :T].permute(0, 2, 1, 3)
    assert rel(flat[0, :, :, :d], rot(y[:, H * d:(H + G) * d], G)) < 5e-6
    assert rel(flat[1, :, :, :dv], y[:, (H + G) * d:].reshape(T, G, dv)) < 1e-6


def pooled_rows(q, k, v, kb, vb, pos, size, pool):
    """One query [H, d] at ``pos`` over tokens k, v [n, G, *] and block means kb, vb; the scale already inside q."""
    H, G = q.shape[0], k.shape[1]
    grp = torch.arange(H) // (H // G)
    lo, nb = max(0, pos - size + 1), max(0, (pos - size + 1) // pool)
    ks, vs = torch.cat([kb[:nb], k[lo:pos + 1]])[:, grp], torch.cat([vb[:nb], v[lo:pos + 1]])[:, grp]
    return torch.einsum("hj,jhd->hd", torch.softmax(torch.einsum("hd,jhd->hj", q, ks), dim=1), vs)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,page,size,pool", [
    (4, 2, 16, 8, 8, 40, 5), (6, 2, 112, 80, 16, 64, 8), (3, 3, 24, 40, 16, 1, 1), (2, 1, 16, 16, 4, 100, 3), (8, 8, 32, 32, 32, 65, 16),
    (5, 1, 12, 20, 6, 63, 64), (16, 2, 128, 128, 16, 128, 2), (12, 1, 64, 32, 16, 7, 90), (2, 1, 256, 64, 16, 30, 4),
    (4, 4, 64, 64, 64, 129, 1)])
def test_pooled_attention_kernels_alone(H, G, d, dv, page, size, pool, dtype):
    """The last query points at one block or key: the first block, the last one it sees, the first one it does not see
    yet (whose weight must be nothing), the oldest key of the window, the one just before it, its own.  It is a single
    token and the end of a portion; in bfloat16 also through the tensor-core kernels (the split kernel in one part and
    in several).  Entries that are not seen hold numbers that would show."""
    from railgun_b200 import ops
    n = 411
    D = -(-max(d, dv) // 16) * 16
    rng = np.random.default_rng(H * d + page)
    nb_all = n // pool
    seen = max(0, (n - 1 - size + 1) // pool)
    lo = n - size
    cases = [("block", 0), ("block", seen - 1), ("block", seen), ("key", lo), ("key", lo - 1), ("key", n - 1), ("key", (lo + n - 1) // 2)]
    dt = TORCH[dtype]
    tol = 2e-5 if dtype == "float32" else 2e-2
    for what, at in cases:
        if what == "block" and not 0 <= at < nb_all:
            continue
        k = torch.tensor(rng.normal(size=(n, G, d)), dtype=dt).double()
        v = torch.tensor(rng.normal(size=(n, G, dv)), dtype=dt).double()
        loud = torch.tensor(rng.normal(size=d) * 1.5)
        rows = range(at * pool, (at + 1) * pool) if what == "block" else [at]
        for j in rows:
            k[j, 0] = loud.to(dt).double()
        kb = torch.stack([k[b * pool:(b + 1) * pool].mean(dim=0) for b in range(nb_all)]).to(dt).double()
        vb = torch.stack([v[b * pool:(b + 1) * pool].mean(dim=0) for b in range(nb_all)]).to(dt).double()
        q = torch.tensor(rng.normal(size=(H, d)) * d ** -0.5, dtype=dt).double()
        q[0] = (loud * 16.0 / float(loud @ loud)).to(dt).double()             # a score of 16 on the loud rows
        order = rng.permutation(-(-n // page) + 3)[:-(-n // page)].tolist()
        eorder = rng.permutation(-(-nb_all // page) + 3)[:-(-nb_all // page)].tolist()
        cache, entries = pages_of((k, v), page, D, dt, order), pages_of((kb, vb), page, D, dt, eorder)
        table, etable = torch.tensor([order], dtype=torch.int32), torch.tensor([eorder], dtype=torch.int32)
        ref = pooled_rows(q, k, v, kb, vb, n - 1, size, pool)
        pooled = (dev(entries), dev(etable), pool)
        for portion in (1, 150):
            qs = torch.zeros((portion, H, D), dtype=dt)
            qs[:, :, :d] = torch.tensor(rng.normal(size=(portion, H, d)) * d ** -0.5, dtype=dt)
            qs[-1, :, :d] = q.to(dt)
            if portion > 1:
                qs[portion // 2] = qs[-1]
            pos = torch.arange(n - portion, n, dtype=torch.int32)
            wide = torch.full((portion, H * D + 24), 3.0, dtype=dt, device=DEV)
            ops.paged_attention_general(dev(qs).view(portion, H * D), H * D, dev(cache), dev(table),
                                        dev(torch.zeros(portion, dtype=torch.int32)), dev(pos), H, G, D, size, 1.0,
                                        pooled=pooled, out=wide[:, 8:8 + H * D], out_scale=0.5)
            outs = [wide]
            if dtype == "bfloat16" and portion == 1:
                for splits in (1, 3, 8):
                    o = torch.full_like(wide, 3.0)
                    ops.decode_attention(dev(qs).view(1, H * D), H * D, o[:, 8:8 + H * D], dev(cache), dev(table), None, 1,
                                         dev(torch.zeros(1, dtype=torch.int32)), dev(pos), H, G, D, size, 1.0, splits,
                                         pooled=pooled, out_scale=0.5)
                    outs.append(o)
            elif dtype == "bfloat16":
                tiles = torch.tensor([[0, 64, 0], [64, 64, 0], [128, portion - 128, 0]], dtype=torch.int32)
                o = torch.full_like(wide, 3.0)
                ops.prefill_attention(dev(qs).view(portion, H * D), H * D, o[:, 8:8 + H * D], dev(cache), dev(table), dev(tiles),
                                      dev(pos), H, G, D, size, 1.0, pooled=pooled, out_scale=0.5)
                outs.append(o)
            for i, o in enumerate(outs):
                got = o[:, 8:8 + H * D].reshape(portion, H, D)
                for e in {0, portion // 2, portion - 1}:
                    r = 0.5 * pooled_rows(qs[e, :, :d].double(), k, v, kb, vb, int(pos[e]), size, pool)
                    assert rel(got[e, :, :dv], r) < tol, f"{what} {at}, row {e} of {portion}, form {i}"
                assert rel(got[-1, :, :dv], 0.5 * ref) < tol
                assert D == dv or float(got[:, :, dv:].abs().max()) == 0.0
                assert float((o[:, :8] - 3.0).abs().max()) == 0.0 and float((o[:, 8 + H * D:] - 3.0).abs().max()) == 0.0


# ---- the model through the step function ---------------------------------------------------------------

LENGTHS = {"A": [1, 2, 12, 13, 40, 77, 150, 64], "B": [1, 3, 17, 64, 100, 33], "C": [1, 7, 8, 33, 90, 65],
           "D": [2, 131, 260, 400, 55, 129, 181], "E": [1, 2, 5, 23, 70, 41]}
PORTIONS = {"D": (130, 2, 64, 7, 128, 3, 65, 2, 33, 129)}
MIXED = {"D": (5, 1, 2, 70, 1, 1, 3, 140, 1, 2, 128, 17)}
TAIL = {"D": 140, "B": 60}
_oracle: dict = {}


def oracle(name):
    if name not in _oracle:
        cfg = C.CASES[name][0]
        reqs = {f"r{i}": p for i, p in enumerate(C.prompts(cfg["vocab"], LENGTHS[name], seed=21))}
        plain = C.plain_model(name)
        _oracle[name] = (reqs, {k: plain.forward(v) for k, v in reqs.items()})
    return _oracle[name]


def make_trace(mode, reqs, name):
    if mode == "whole":
        return helpers.trace_whole(reqs)
    if mode == "tail":
        return helpers.trace_tail_decode(reqs, TAIL.get(name, 32))
    if mode == "every_token":
        return helpers.trace_tail_decode(reqs, 10 ** 6)
    if mode == "portions":
        return helpers.trace_portions(reqs, **({"sizes": PORTIONS[name]} if name in PORTIONS else {}))
    if mode == "twos":
        return helpers.trace_portions(reqs, sizes=(2,))
    if mode == "mixed":
        return helpers.trace_mixed(reqs, max_live=4, seed=5, **({"sizes": MIXED[name]} if name in MIXED else {}))
    raise ValueError(mode)


def replay(folder, cfg, page, dtype, steps, out_dir, **more):
    from railgun_b200.engine.runner import ModelRunner
    from railgun_b200.replay import Replayer
    runner = ModelRunner(folder, dtype=dtype, page_size=page, max_tokens=helpers.peak_tokens(steps, 64),
                         max_requests=4, **more)
    rp = Replayer(runner, out_dir)
    for s in steps:
        rp.feed(s)
    runner.check_device_errors()
    runner.alloc.check()
    assert runner.alloc.num_requests() == 0
    return helpers.collect(steps, out_dir, cfg["vocab"])


def replay_case(name, dtype, steps, out_dir, page=None, **more):
    cfg, _, own_page = C.CASES[name]
    return replay(C.model_dir(name), cfg, page or own_page, dtype, steps, out_dir, **more)


def compare(rows, reqs, logits, tol, what):
    worst = 0.0
    for name, toks in reqs.items():
        ref = logits[name]
        scale = np.abs(ref).max()
        for p in range(len(toks)):
            err = np.abs(rows[(name, p)] - ref[p]).max() / scale
            assert err <= tol, (f"{what}: request {name} (length {len(toks)}) first differs at position {p}: "
                                f"relative error {err:.3e}")
            worst = max(worst, err)
    return worst


@pytest.mark.parametrize("mode", ["whole", "tail", "portions", "mixed"])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_replay_matches_plain(name, dtype, mode, tmp_path):
    """Whole prompts; the last tokens one by one; portions down to two tokens, cut inside pages, windows, blocks and the
    reach of the convolutions; up to four live requests in a pool so small that pages and state slots are used
    again.  Every position of every request is compared, the first tokens included."""
    reqs, logits = oracle(name)
    rows = replay_case(name, dtype, make_trace(mode, reqs, name), tmp_path)
    print(f"{name} {dtype} {mode}: worst relative error "
          f"{compare(rows, reqs, logits, TOL[dtype], f'{name} {dtype} {mode}'):.3e}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "E"])
def test_every_token_decoded_alone_matches_whole_prompts(name, dtype, tmp_path):
    """Token-by-token decoding from the first token on (through the decode graphs and with graphs off), and two tokens
    at a time: states and convolution tails that start from nothing, blocks that single tokens complete."""
    reqs, logits = oracle(name)
    few = dict(list(reqs.items())[1:5])
    steps = make_trace("every_token", few, name)
    compare(replay_case(name, dtype, steps, tmp_path / "g"), few, logits, TOL[dtype], "decoded")
    compare(replay_case(name, dtype, steps, tmp_path / "e", use_graphs=False), few, logits, TOL[dtype], "decoded, no graphs")
    compare(replay_case(name, dtype, make_trace("twos", few, name), tmp_path / "t"), few, logits, TOL[dtype], "in twos")


@pytest.mark.parametrize("page", [2, 64])
def test_other_page_sizes(page, tmp_path):
    reqs, logits = oracle("A")
    for mode in ("portions", "mixed"):
        steps = make_trace(mode, reqs, "A")
        for dtype in DTYPES:
            compare(replay_case("A", dtype, steps, tmp_path / f"{mode}{dtype}", page=page), reqs, logits, TOL[dtype],
                    f"page {page} {dtype}")


def test_repeated_layouts_replay_a_graph(tmp_path, monkeypatch):
    """Large steps whose layout repeats run from a captured graph: same slots and pages used again by other requests."""
    from railgun_b200.engine import runner as R
    monkeypatch.setattr(R, "SHAPE_GRAPH_MIN_TOKENS", 2)
    cfg = C.CASE_A
    reqs = {f"g{i}": p for i, p in enumerate(C.prompts(cfg["vocab"], [48] * 5, seed=31))}
    plain = C.plain_model("A")
    logits = {k: plain.forward(v) for k, v in reqs.items()}
    for dtype in DTYPES:
        compare(replay_case("A", dtype, helpers.trace_portions(reqs, sizes=(24,)), tmp_path / dtype), reqs, logits, TOL[dtype],
                "repeated layouts")


def test_batch_of_unequal_requests_equals_each_alone(tmp_path):
    """One step with four prompts of unequal length beside one another, then single tokens of all four in one
    step: the rows equal those of each request run alone."""
    reqs, logits = oracle("D")
    names = list(reqs)[:4]
    together = [{"step": 0, "entries": [{"id": n, "tokens": reqs[n][:-1], "want": list(range(len(reqs[n]) - 1))}
                                         for n in names], "end": []},
                {"step": 1, "entries": [{"id": n, "tokens": reqs[n][-1:], "want": [0]} for n in names], "end": names}]
    alone, k = [], 0
    for n in names:
        alone.append({"step": k, "entries": [{"id": n, "tokens": reqs[n][:-1], "want": list(range(len(reqs[n]) - 1))}],
                      "end": []})
        alone.append({"step": k + 1, "entries": [{"id": n, "tokens": reqs[n][-1:], "want": [0]}], "end": [n]})
        k += 2
    for dtype in DTYPES:
        a = replay_case("D", dtype, together, tmp_path / f"t{dtype}")
        b = replay_case("D", dtype, alone, tmp_path / f"a{dtype}")
        compare(a, {n: reqs[n] for n in names}, logits, TOL[dtype], "together")
        for key in a:
            assert np.abs(a[key] - b[key]).max() <= (2e-5 if dtype == "float32" else 0.1) * np.abs(b[key]).max(), key


# ---- models in which one mechanism carries everything -----------------------------------------------------

def attention_only(cfg, change_mask=None):
    """The parallel layers of ``cfg`` with the right half silenced."""
    layers = [json.loads(json.dumps(L)) for L in cfg["layers"] if L["type"] == "parallel"]
    for L in layers:
        L["mixer"]["right_scale"] = 0.0
        if change_mask:
            change_mask(L["mixer"]["left"]["mask"])
    return dict(cfg, layers=layers)


def sharpen(cfg):
    """Queries and keys so sharp that single keys and blocks take most of a head's weight."""
    def change(t):
        for i in range(len(cfg["layers"])):
            t[f"l{i}.shift"] *= 0.0
    return change


def test_edges_of_windows_and_blocks_show(tmp_path):
    """Scores ten times larger than usual, no right halves, no shifts: a window one token longer or shorter, blocks one
    token longer or shorter, or blocks left out, move the logits at nearly every position by far more than the
    tolerance.  Prompts, portions, decoding and mixed batches."""
    only = attention_only(C.CASE_D)
    for L in only["layers"]:
        L["mixer"]["left"]["scale"] *= 12.0
    folder = C.write_model(only, 5, tmp_path / "model", change=sharpen(only))
    plain = C.Plain(folder)
    reqs = {f"s{i}": p for i, p in enumerate(C.prompts(only["vocab"], [190, 135, 52, 300], seed=4))}
    logits = {k: plain.forward(v) for k, v in reqs.items()}
    scale = np.abs(logits["s3"]).max()
    for key, by in (("size", 1), ("size", -1), ("pool", 1), ("pool", -1), ("pool", 10 ** 6)):
        other = json.loads(json.dumps(only))
        for L in other["layers"]:
            L["mixer"]["left"]["mask"][key] += by
        moved = np.abs(P.forward(reqs["s3"], plain.w, other) - logits["s3"]).max(axis=1) / scale
        assert np.median(moved[150:]) > 20 * TOL["float32"], (key, by)
    for mode in ("whole", "tail", "portions", "mixed"):
        rows = replay(folder, only, 16, "float32", make_trace(mode, reqs, "D"), tmp_path / mode)
        compare(rows, reqs, logits, 2 * TOL["float32"], f"sharp {mode}")
    rows = replay(folder, only, 16, "bfloat16", make_trace("mixed", reqs, "D"), tmp_path / "b")
    errs = [np.abs(rows[(n, p)] - logits[n][p]).max() / scale for n in reqs for p in range(len(reqs[n]))]
    assert np.median(errs) < TOL["bfloat16"]                  # close calls between sharp scores may fall either way


def test_a_far_block_is_heard(tmp_path):
    """An attention-only model: prompts that differ in one early token only (and so in one pooled block) still differ
    after 380 more, in portions and decoded one by one; the same with the difference in the last block that is seen."""
    only = attention_only(C.CASE_D)
    folder = C.write_model(only, 23, tmp_path / "model", change=sharpen(only))
    plain = C.Plain(folder)
    a = C.prompts(only["vocab"], [400], seed=10)[0]
    reqs = {"a": a}
    for name, at in (("b", 3), ("c", 200)):
        other = list(a)
        other[at] = (a[at] + 7) % only["vocab"]
        reqs[name] = other
    logits = {k: plain.forward(v) for k, v in reqs.items()}
    for name in "bc":
        assert np.abs(logits["a"][-1] - logits[name][-1]).max() > 20 * TOL["float32"] * np.abs(logits["a"]).max()
    for mode in ("tail", "portions"):
        compare(replay(folder, only, 16, "float32", make_trace(mode, reqs, "D"), tmp_path / mode), reqs, logits,
                TOL["float32"], f"far {mode}")


@pytest.mark.parametrize("kind", ["mamba2", "rwkv"])
def test_states_remember_a_far_token(kind, tmp_path):
    """Models in which only the matrix states carry anything further than two tokens, with slow decays: a prompt whose
    second token differs still differs after 300 more tokens, most of them decoded one by one."""
    cfg = json.loads(json.dumps(C.CASE_D))
    cfg["layers"] = [L for L in cfg["layers"] if L["type"] == ("mamba2" if kind == "mamba2" else "parallel")]
    for L in cfg["layers"]:
        if kind == "rwkv":
            L["mixer"]["left_scale"] = 0.0

    def slow(t):
        for name in t:
            if name.endswith("A_log"):
                t[name] = t[name] * 0.0 - 6.0
            if name.endswith("w0"):
                t[name] = t[name] * 0.0 - 8.0
            if name.endswith("right.w2"):
                t[name] *= 0.1

    folder = C.write_model(cfg, 17, tmp_path / "model", change=slow)
    plain = C.Plain(folder)
    a = C.prompts(cfg["vocab"], [310], seed=9)[0]
    b = list(a)
    b[1] = (a[1] + 11) % cfg["vocab"]
    reqs = {"a": a, "b": b}
    logits = {k: plain.forward(v) for k, v in reqs.items()}
    assert np.abs(logits["a"][-1] - logits["b"][-1]).max() > 20 * TOL["float32"] * np.abs(logits["a"]).max()
    steps = helpers.trace_tail_decode(reqs, 250)
    compare(replay(folder, cfg, 16, "float32", steps, tmp_path / "o"), reqs, logits, TOL["float32"], "far")


# ---- generation through the engine and the command line -----------------------------------------------

def greedy_consistent(plain, prompt, out, tol):
    """How many generated tokens are the plain model's choice given the tokens before them (teacher-forced), up
    to ``tol`` of the largest absolute logit."""
    logits = plain.forward(list(prompt) + list(out))
    return sum(int(logits[len(prompt) - 1 + i][t] >= logits[len(prompt) - 1 + i].max() - tol * np.abs(logits).max())
               for i, t in enumerate(out))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_engine(name, dtype):
    """Prompts of one token and more, prefilled in portions by the scheduler beside decoding requests."""
    from railgun_b200.engine.engine import Engine
    from railgun_b200.engine.request import SamplingParams
    cfg, _, page = C.CASES[name]
    prompts = C.prompts(cfg["vocab"], [1, 2, 9, 40, 63, 100], seed=2)
    plain = C.plain_model(name)
    eng = Engine(C.model_dir(name), dtype=dtype, block_size=page, num_gpu_blocks=1024 // page, max_num_seqs=4,
                 max_num_batched_tokens=64, max_prefill_chunk=24, max_model_len=256)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=10))
    good = 0
    for p, o in zip(prompts, outs):
        assert o.finish_reason == "max_tokens" and len(o.token_ids) == 10
        good += greedy_consistent(plain, p, o.token_ids, 1e-4 if dtype == "float32" else 6e-2)
        if dtype == "float32":
            assert o.token_ids == plain.greedy(p, 10)
    assert good == 60
    assert eng.stats()["num_free_blocks"] == 1024 // page and not eng.has_unfinished()


def test_preempted_requests_start_again_from_their_tokens():
    """A pool too small for all requests: the scheduler preempts, and what it recomputes gives the same tokens."""
    from railgun_b200.engine.engine import Engine
    from railgun_b200.engine.request import SamplingParams
    cfg, _, page = C.CASES["A"]
    plain = C.plain_model("A")
    prompts = C.prompts(cfg["vocab"], [30, 41, 25, 37], seed=12)
    eng = Engine(C.model_dir("A"), dtype="float32", block_size=page, num_gpu_blocks=14, max_num_seqs=4,
                 max_num_batched_tokens=64, max_prefill_chunk=24, max_model_len=112)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=40))
    for p, o in zip(prompts, outs):
        assert len(o.token_ids) == 40 and greedy_consistent(plain, p, o.token_ids, 1e-4) == 40


def test_long_decoding_through_the_engine():
    from railgun_b200.engine.engine import Engine
    from railgun_b200.engine.request import SamplingParams
    cfg, _, page = C.CASES["A"]
    plain = C.plain_model("A")
    prompt = C.prompts(cfg["vocab"], [3], seed=8)[0]
    eng = Engine(C.model_dir("A"), dtype="float32", block_size=page, num_gpu_blocks=100, max_num_seqs=2,
                 max_model_len=400)
    out = eng.generate([prompt], SamplingParams(max_new_tokens=300))[0]
    assert len(out.token_ids) == 300
    assert greedy_consistent(plain, prompt, out.token_ids, 1e-4) == 300


def test_command_line_and_trace_runner(tmp_path):
    d = C.model_dir("C")
    plain = C.plain_model("C")
    prompt = [7, 80, 3, 55]
    res = subprocess.run([sys.executable, "-m", "railgun_b200", "generate", "-m", str(d), "--prompt-ids",
                          ",".join(map(str, prompt)), "--max-tokens", "6", "--dtype", "f32", "--block-size", "8"],
                         cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    line = [l for l in res.stdout.splitlines() if l and l[0].isdigit()][0]
    assert [int(t) for t in line.split(",")] == plain.greedy(prompt, 6)
    toks = C.prompts(90, [30], seed=6)[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:19], "want": [0, 18]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[19:21], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[21:], "want": [8]}], "end": ["a"]}]
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out",
                          str(tmp_path), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = plain.forward(toks)
    got0 = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, 90)
    got2 = np.fromfile(tmp_path / "2.f32", dtype="<f4").reshape(1, 90)
    assert not (tmp_path / "1.f32").exists()
    scale = np.abs(ref).max()
    assert np.abs(got0 - ref[[0, 18]]).max() < 1e-4 * scale and np.abs(got2[0] - ref[29]).max() < 1e-4 * scale
