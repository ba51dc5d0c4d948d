"""Timopel on the GPU with the engine's kernels, in float32 and bfloat16, against tests/plain_timopel.py: each mechanism
alone, then whole models under every kind of schedule."""

import pytest
import torch

import timopel_cases as tc

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def ops():
    from qwen3_runtime_b200.ops.cuda import CudaOps

    return CudaOps()


DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixers_alone(ops, dtype):
    tc.case_mixers_alone(dtype, ops, DEV)
    tc.case_mixers_alone(dtype, ops, DEV, page_size=4, heads=2, kv_heads=2, dim=16, vdim=16,
                         q_temp=tc.TemperatureConfig(0.8, 1), second=dict(q_temp=None, heads=4))
    big = dict(page_size=16, T=150, cuts=(70, 1, 2, 77), scale=0.1)
    # keys and values of one size (the split-KV kernel makes the newest token's q, k and blended v), of unlike sizes
    tc.case_mixers_alone(dtype, ops, DEV, **big, heads=8, kv_heads=2, dim=64, vdim=64)
    tc.case_mixers_alone(dtype, ops, DEV, **big, heads=4, kv_heads=1, dim=128, vdim=128)
    tc.case_mixers_alone(dtype, ops, DEV, **big, heads=2, kv_heads=1, dim=256, vdim=256)
    tc.case_mixers_alone(dtype, ops, DEV, **big, heads=6, kv_heads=2, dim=128, vdim=64, second=dict(dim=64))
    tc.case_mixers_alone(dtype, ops, DEV, **big, heads=16, kv_heads=1, dim=40, vdim=72, second=dict(heads=20))
    ops.fuse_decode_new_token = False  # the newest token by the q/k kernel, then the plain split-KV kernel
    try:
        tc.case_mixers_alone(dtype, ops, DEV, **big, heads=4, kv_heads=1, dim=128, vdim=128)
    finally:
        ops.fuse_decode_new_token = True
    ops.prefill_attention = "mma"  # the mma.sync prompt kernels at heads of 128
    try:
        tc.case_mixers_alone(dtype, ops, DEV, **big, heads=4, kv_heads=1, dim=128, vdim=128)
    finally:
        ops.prefill_attention = "tcgen05"
    ops.chunk_tc = False  # the general kernel
    try:
        tc.case_mixers_alone(dtype, ops, DEV, **big, heads=6, kv_heads=2, dim=128, vdim=64, second=dict(dim=64))
    finally:
        ops.chunk_tc = True


SIZES = [dict(), dict(page_size=4, heads=1, kv_heads=1, D=20, Dv=8), dict(page_size=16, heads=6, kv_heads=2, D=48, Dv=96, T=330),
         dict(page_size=16, heads=4, kv_heads=1, D=64, Dv=64, T=300), dict(page_size=16, heads=8, kv_heads=1, D=128, Dv=128, T=700),
         dict(page_size=32, heads=4, kv_heads=4, D=128, Dv=128, T=420), dict(page_size=16, heads=4, kv_heads=1, D=256, Dv=256, T=230),
         dict(page_size=16, heads=5, kv_heads=1, D=256, Dv=40, T=230), dict(page_size=8, heads=18, kv_heads=1, D=16, Dv=16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", SIZES, ids=lambda s: "x".join(map(str, s.values())) or "default")
def test_attention_far_keys(ops, dtype, sizes):
    tc.case_attention_far_keys(dtype, ops, DEV, **sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_of_batches(ops, dtype):
    tc.case_attention_batch(dtype, ops, DEV)
    tc.case_attention_batch(dtype, ops, DEV, heads=8, kv_heads=2, D=128, Dv=128)
    tc.case_attention_batch(dtype, ops, DEV, heads=3, kv_heads=3, D=40, Dv=72, page_size=8)
    tc.case_attention_batch(dtype, ops, DEV, heads=8, kv_heads=1, D=128, Dv=64)
    tc.case_attention_batch(dtype, ops, DEV, heads=2, kv_heads=1, D=256, Dv=256)


@pytest.mark.parametrize("dtype", DTYPES)
def test_kernels_alone(ops, dtype):
    tc.case_query_temperature(ops, DEV)
    tc.case_store(dtype, ops, DEV)
    tc.case_routing(dtype, ops, DEV)
    tc.case_output_norm_with_multiplier(dtype, ops, DEV)


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forwards_alone(ops, dtype):
    tc.case_feed_forwards_alone(dtype, ops, DEV)
    tc.case_feed_forwards_alone(dtype, ops, DEV, experts=3, top=3, shared=None, scale=1.0, T=5)
    tc.case_feed_forwards_alone(dtype, ops, DEV, experts=12, top=4, ff=72, shared=(56, 0.6), T=700, width=136)
    tc.case_feed_forwards_alone(dtype, ops, DEV, experts=4, top=1, ff=36, shared=(20, 1.0), T=40, width=60)


@pytest.mark.parametrize("M", [3, 40, 300, 1280])
@pytest.mark.parametrize("activation", ["silu", "gelu"])
def test_gated_products(ops, M, activation):
    """The gated product of a dense layer on every kernel a token count leads to (the streaming kernels, the library
    product and the unit's kernel, tcgen05 on one SM and on pairs)."""
    gen = torch.Generator().manual_seed(3)
    K, I = 512, 2560
    x = torch.randn((M, K), generator=gen).to(torch.bfloat16).cuda()
    w = (torch.randn((2 * I, K), generator=gen) * 0.1).to(torch.bfloat16).cuda()
    g, u = x.double() @ w[:I].double().t(), x.double() @ w[I:].double().t()
    want = (tc.pl.gelu(g) if activation == "gelu" else g * torch.sigmoid(g)) * u
    out = torch.empty((M, I), dtype=torch.bfloat16, device="cuda")
    for large in ("auto", "tcgen05", "library"):
        ops.large_gemm = large
        try:
            ops.gated_linear(x, w, out, activation=activation)
            if M > 128 and large == "tcgen05":
                for pair in (False, True):
                    ops.linear_tcgen05(x, w, out=out, mode=2 + ops.GLU_ACTIVATIONS[activation], pair=pair)
                    assert float((out.double() - want).abs().max()) <= 1e-2 * float(want.abs().max())
        finally:
            ops.large_gemm = "auto"
        assert float((out.double() - want).abs().max()) <= 1e-2 * float(want.abs().max())
    ops.raise_if_kernel_error()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_schedules(tmp_path, ops, name, dtype):
    tc.case_schedules(tmp_path, name, dtype, ops, DEV)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_stream_after_every_layer(tmp_path, ops, name):
    tc.case_stream_after_every_layer(tmp_path, name, ops, DEV)


@pytest.mark.parametrize("name", ["A", "B", "D", "E"])
def test_schedules_through_captured_decode_steps(tmp_path, ops, name):
    tc.case_schedules(tmp_path, name, "bfloat16", ops, DEV, cuda_graph=True)
    tc.case_schedules(tmp_path, name, "float32", ops, DEV, cuda_graph=True, lengths=(40, 5, 33))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode(tmp_path, ops, dtype):
    tc.case_long_decode(tmp_path, "A", dtype, ops, DEV, total=200, cuda_graph=True)
    tc.case_long_decode(tmp_path, "B", dtype, ops, DEV, total=120)
    tc.case_long_decode(tmp_path, "D", dtype, ops, DEV, total=330, cuda_graph=True)
    tc.case_long_decode(tmp_path, "E", dtype, ops, DEV, total=330, cuda_graph=True)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(tmp_path, ops, dtype):
    for name in ("A", "B", "D"):
        tc.case_first_tokens(tmp_path, name, dtype, ops, DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuda_graph", [False, True])
def test_greedy_generation_under_the_scheduler(tmp_path, ops, dtype, cuda_graph):
    tc.case_greedy_generation(tmp_path, "A", dtype, ops, DEV, cuda_graph=cuda_graph)
    tc.case_greedy_generation(tmp_path, "D", dtype, ops, DEV, cuda_graph=cuda_graph)


def test_bfloat16_steps_take_the_specialised_kernels(tmp_path, ops):
    """A bfloat16 model runs prompt portions on the tensor-core kernels (tcgen05 for heads of 128) and decode steps on
    the split-KV kernel that makes the newest token itself, or on the sliced one for unlike sizes; the general attention
    kernel and the FMA expert products are not launched."""
    from helpers import run_trace, trace_tail_decode

    launched, factors = [], []
    call, timed, ops.timing = ops._call, ops._timed, []

    def call_spy(group, name, what, *args):
        launched.append(what)
        factors.extend([what] if what == "query_temperature" else [])
        return call(group, name, what, *args)

    def timed_spy(what):  # launches that may be refused go past _call
        launched.append(what)
        return timed(what)

    ops._call, ops._timed = call_spy, timed_spy
    try:
        rt = tc.runtime(tc.make_dir(tmp_path, "D"), "D", "bfloat16", ops, DEV, pages=16)
        run_trace(rt, trace_tail_decode(tc.requests_for("D", (70,)), tail=5))
    finally:
        del ops._call, ops._timed
        ops.timing = None
    for kernel in ("paged_attention_prefill_tc", "paged_attention_prefill", "paged_attention_decode_fused",
                   "chunk_attention_prefill", "chunk_attention_decode", "qk_norm_store", "query_temperature",
                   "expert_gate_up_tc", "expert_down_tc", "fused_post_norm", "bigram_embed"):
        assert kernel in launched, f"{kernel} was not launched: {sorted(set(launched))}"
    assert "paged_attention" not in launched and "expert_gate_up" not in launched
    # one table of factors per step and set of constants, however many layers use it
    assert len(factors) == 6 * 3


def test_trace_replay_program_on_a_timopel_folder(tmp_path, ops):
    """bin/trace_run as a subprocess: the model class is chosen by config.json."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    folder = tc.make_dir(tmp_path, "C")
    toks = tc.requests_for("C", (40,))["r0"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:31], "want": [0, 30]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[31:], "want": [8]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype",
                           "float32", "--out", str(out), "--max-tokens", "64"],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                          timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    want, tol = tc.expected(folder, {"a": toks}, "float32")
    V = tc.CONFIGS["C"]["config"].vocab
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, V))
    got1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(1, V))
    assert float((got0 - want["a"][[0, 30]]).abs().max()) <= tol
    assert float((got1 - want["a"][[39]]).abs().max()) <= tol


def test_command_line_on_a_timopel_folder(tmp_path):
    """``python -m qwen3_runtime_b200.cli`` generates greedily from a Timopel folder what the plain model does."""
    import os
    import subprocess
    import sys

    folder = tc.make_dir(tmp_path, "A")
    raw, t = tc.read_dir(folder)
    prompt = [5, 6, 7, 8, 9]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cmd = [sys.executable, "-m", "qwen3_runtime_b200.cli", "--model", str(folder), "--max-tokens", "6", "--dtype",
           "float32", "--prompt-tokens", *map(str, prompt), "--num-kv-blocks", "16", "--no-cuda-graph"]
    proc = subprocess.run(cmd, capture_output=True, text=True, cwd=root, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = dict(line.split(" ", 1) for line in proc.stdout.strip().splitlines())
    got = [int(x) for x in lines["runtime"].strip("[]").split(",")]
    assert len(got) == 6
    seq = list(prompt)
    for tok in got:  # every token is the plain model's best (or within float32 rounding of it) given the tokens before
        row = tc.pl.forward(raw, t, seq)[-1].float()
        assert float(row.max() - row[tok]) <= 1e-4 * max(1.0, float(row.abs().max()))
        seq.append(tok)
