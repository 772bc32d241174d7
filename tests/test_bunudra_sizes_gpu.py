"""Bunudra at the layer sizes the benchmark times (8 memory heads of 64 x 128, 8 heads of 64 + 32 over a latent of 256
and 8 heads of 128 on 2 key/value heads, at width 1,024; fewer experts, a small vocabulary, three layers), against the
plain statement: both precisions, prompts (the recurrence in chunks, the expanded form of the latent, the tensor-core
attention kernels with a window and chunks of several tiles, the grouped tcgen05 product) and single tokens."""
import numpy as np
import pytest

import bunudra_cases as C
import helpers
import plain_bunudra as P

pytestmark = pytest.mark.gpu

CASE_W = dict(
    architecture="Bunudra", width=1024, vocab=512, embedding=dict(scale=1.0), norm=dict(eps=1e-6),
    layers=[C.layer(C.memory(8, 64, 128, 15.0), C.experts(4, 4, 512, None, 1.5, 1024)),
            C.layer(C.latent(8, 64, 32, 64, 256, 150, 10000.0, (8.0, 4096.0, 32.0, 1.0)), C.experts(4, 4, 512, None, 1.0, 512)),
            C.layer(C.chunked(8, 2, 128, 128, 100, dims=64), None)])
LENGTHS = [330, 40, 197, 3]
_state: dict = {}


def setup(tmp_factory):
    if not _state:
        folder = tmp_factory.mktemp("bunudra_W")

        def shrink(t):                              # rows of 1,024 numbers must not saturate the gates
            for k in t:
                if t[k].ndim == 2 and k != "embed":
                    t[k] *= 0.25
        C.write_model(CASE_W, 17, folder, change=shrink)
        plain = C.Plain(folder)
        reqs = {f"r{i}": p for i, p in enumerate(C.prompts(CASE_W["vocab"], LENGTHS, seed=31))}
        _state.update(dir=folder, reqs=reqs, logits={k: P.forward(v, plain.w, plain.cfg) for k, v in reqs.items()})
    return _state


@pytest.mark.parametrize("mode", ["whole", "tail", "mixed"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_benchmark_layer_sizes_match_plain(dtype, mode, tmp_path, tmp_path_factory):
    from railgun_b200.engine.runner import ModelRunner
    from railgun_b200.replay import Replayer
    st = setup(tmp_path_factory)
    reqs = st["reqs"]
    steps = {"whole": lambda: helpers.trace_whole(reqs), "tail": lambda: helpers.trace_tail_decode(reqs, 120),
             "mixed": lambda: helpers.trace_mixed(reqs, max_live=4, seed=3, sizes=(70, 1, 2, 33, 1, 130, 1, 5))}[mode]()
    runner = ModelRunner(st["dir"], dtype=dtype, page_size=16, max_tokens=helpers.peak_tokens(steps, 64), max_requests=4)
    rp = Replayer(runner, tmp_path)
    for s in steps:
        rp.feed(s)
    runner.check_device_errors()
    runner.alloc.check()
    rows = helpers.collect(steps, tmp_path, CASE_W["vocab"])
    tol = 5e-5 if dtype == "float32" else 4e-2
    for name, toks in reqs.items():
        ref = st["logits"][name]
        scale = np.abs(ref).max()
        for p in range(len(toks)):
            err = np.abs(rows[(name, p)] - ref[p]).max() / scale
            assert err <= tol, f"{dtype} {mode}: request {name} position {p}: relative error {err:.3e}"
