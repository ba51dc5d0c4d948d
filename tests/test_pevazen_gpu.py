"""Pevazen on the GPU with the engine's kernels, in float32 and bfloat16, against tests/plain_pevazen.py: each
mechanism alone, then whole models under every kind of schedule."""

import pytest
import torch

import pevazen_cases as pc

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def ops():
    from qwen3_runtime_b200.ops.cuda import CudaOps

    return CudaOps()


DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixers_alone(ops, dtype):
    pc.case_mixer_alone(dtype, ops, DEV, "attention")
    pc.case_mixer_alone(dtype, ops, DEV, "attention", page_size=4, heads=2, kv_heads=2, dim=16, vdim=16, chunk=None,
                        rot=None)
    pc.case_mixer_alone(dtype, ops, DEV, "attention", page_size=16, T=150, cuts=(70, 1, 2, 77), heads=8, kv_heads=2,
                        dim=64, vdim=128, scale=0.125, chunk=48, rot=pc._rot(32, 5e4))
    pc.case_mixer_alone(dtype, ops, DEV, "parallel")
    pc.case_mixer_alone(dtype, ops, DEV, "parallel", left=dict(chunk=None, vdim=10, dim=24),
                        right=dict(conv=1, heads=3, kv_heads=3, dim=16, vdim=16))
    pc.case_mixer_alone(dtype, ops, DEV, "parallel", page_size=16, T=150, cuts=(70, 1, 2, 77),
                        left=dict(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09, chunk=48, rot=pc._rot(128, 1e4, 2.0)),
                        right=dict(heads=4, kv_heads=2, dim=64, vdim=32, decay_rank=16, gate_rank=8))


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_edges(ops, dtype):
    for turned in (False, True):
        pc.case_attention_edges(dtype, ops, DEV, turned=turned)
        pc.case_attention_edges(dtype, ops, DEV, chunk=8, page_size=8, heads=1, kv_heads=1, D=20, Dv=8, turned=turned)
        pc.case_attention_edges(dtype, ops, DEV, chunk=33, page_size=16, heads=6, kv_heads=2, D=48, Dv=96, T=130,
                                turned=turned)
        pc.case_attention_edges(dtype, ops, DEV, chunk=64, page_size=16, heads=4, kv_heads=1, D=64, Dv=64, T=200,
                                turned=turned)
        pc.case_attention_edges(dtype, ops, DEV, chunk=200, page_size=16, heads=4, kv_heads=1, D=128, Dv=128, T=700,
                                turned=turned)
        pc.case_attention_edges(dtype, ops, DEV, chunk=129, page_size=32, heads=2, kv_heads=2, D=128, Dv=32, T=420,
                                turned=turned)
        pc.case_attention_edges(dtype, ops, DEV, chunk=70, page_size=4, heads=5, kv_heads=1, D=96, Dv=96, T=230,
                                turned=turned)
        pc.case_attention_edges(dtype, ops, DEV, chunk=40, page_size=16, heads=2, kv_heads=1, D=256, Dv=192, T=130,
                                turned=turned)


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_of_batches(ops, dtype):
    for turned in (False, True):
        pc.case_attention_batch(dtype, ops, DEV, turned=turned)
        pc.case_attention_batch(dtype, ops, DEV, heads=8, kv_heads=2, D=128, Dv=128, chunk=64, turned=turned)
        pc.case_attention_batch(dtype, ops, DEV, heads=3, kv_heads=3, D=40, Dv=72, chunk=None, page_size=8, turned=turned)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule(ops, dtype):
    pc.case_delta_rule(dtype, ops, DEV)
    pc.case_delta_rule(dtype, ops, DEV, H=3, G=1, D=16, Dv=8, taps=1, ra=3, rg=5, decay=0.5)
    pc.case_delta_rule(dtype, ops, DEV, H=2, G=2, D=64, Dv=64, taps=2, ra=16, rg=8)
    pc.case_delta_rule(dtype, ops, DEV, H=4, G=1, D=128, Dv=128, taps=4, ra=32, rg=16, lens=(130, 3, 33, 16))
    pc.case_delta_rule(dtype, ops, DEV, H=2, G=1, D=128, Dv=40, taps=3, ra=8, rg=8, lens=(300, 17, 1), decay=-5.0)
    # chunks of 16 tokens: portions on both sides of a chunk's edge, very strong and very weak decays, many sequences
    pc.case_delta_rule(dtype, ops, DEV, H=3, G=1, D=72, Dv=24, taps=4, ra=8, rg=8, lens=(15, 16, 17, 33, 64), decay=4.0)
    pc.case_delta_rule(dtype, ops, DEV, H=2, G=1, D=40, Dv=100, taps=2, ra=8, rg=8, lens=(31, 1, 48, 2, 1, 65), decay=-6.0)
    ops.delta_chunks = False  # the same sizes token by token
    try:
        pc.case_delta_rule(dtype, ops, DEV, H=4, G=1, D=128, Dv=128, taps=4, ra=32, rg=16, lens=(130, 3, 33, 16))
        pc.case_delta_rule(dtype, ops, DEV, H=3, G=1, D=72, Dv=24, taps=4, ra=8, rg=8, lens=(15, 16, 17, 33, 64), decay=4.0)
    finally:
        ops.delta_chunks = True
    pc.case_delta_rule(dtype, ops, DEV, H=2, G=2, D=200, Dv=136, taps=5, ra=8, rg=8, lens=(40, 1, 5))
    pc.case_delta_rule(dtype, ops, DEV, H=2, G=2, D=32, Dv=256, taps=4, ra=8, rg=12, lens=(40, 1, 5), decay=3.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_turns_sums_and_norms(ops, dtype):
    pc.case_turn_store(dtype, ops, DEV)
    pc.case_sum_norm(dtype, ops, DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_schedules(tmp_path, ops, name, dtype):
    pc.case_schedules(tmp_path, name, dtype, ops, DEV)


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_stream_after_every_layer(tmp_path, ops, name):
    pc.case_stream_after_every_layer(tmp_path, name, ops, DEV)


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_schedules_through_captured_decode_steps(tmp_path, ops, name):
    pc.case_schedules(tmp_path, name, "bfloat16", ops, DEV, cuda_graph=True)
    pc.case_schedules(tmp_path, name, "float32", ops, DEV, cuda_graph=True, lengths=(40, 5, 33))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode(tmp_path, ops, dtype):
    pc.case_long_decode(tmp_path, "A", dtype, ops, DEV, total=200, cuda_graph=True)
    pc.case_long_decode(tmp_path, "B", dtype, ops, DEV, total=120)
    pc.case_long_decode(tmp_path, "D", dtype, ops, DEV, total=330, cuda_graph=True)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(tmp_path, ops, dtype):
    for name in ("A", "B", "C"):
        pc.case_first_tokens(tmp_path, name, dtype, ops, DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuda_graph", [False, True])
def test_greedy_generation_under_the_scheduler(tmp_path, ops, dtype, cuda_graph):
    pc.case_greedy_generation(tmp_path, "A", dtype, ops, DEV, cuda_graph=cuda_graph)
    pc.case_greedy_generation(tmp_path, "D", dtype, ops, DEV, cuda_graph=cuda_graph)


def test_trace_replay_program_on_a_pevazen_folder(tmp_path, ops):
    """bin/trace_run as a subprocess: the model class is chosen by config.json."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    folder = pc.make_dir(tmp_path, "C")
    toks = pc.requests_for("C", (40,))["r0"]
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
    want, tol = pc.expected(folder, {"a": toks}, "float32")
    V = pc.CONFIGS["C"]["config"].vocab
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, V))
    got1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(1, V))
    assert float((got0 - want["a"][[0, 30]]).abs().max()) <= tol
    assert float((got1 - want["a"][[39]]).abs().max()) <= tol


def test_command_line_on_a_pevazen_folder(tmp_path):
    """``python -m qwen3_runtime_b200.cli`` generates greedily from a Pevazen folder what the plain model does."""
    import os
    import subprocess
    import sys

    import plain_pevazen as pl

    folder = pc.make_dir(tmp_path, "A")
    raw, t = pc.read_dir(folder)
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
        row = pl.forward(raw, t, seq)[-1].float()
        assert float(row.max() - row[tok]) <= 1e-4 * max(1.0, float(row.abs().max()))
        seq.append(tok)


def test_bfloat16_steps_take_the_specialised_kernels(tmp_path, ops):
    """A bfloat16 model runs prompt portions on the tensor-core kernels (tcgen05 for heads of 128) and decode steps on
    the kernel over slices of the visible keys and the kernel that does a whole delta-rule step; the general attention
    kernel is not launched."""
    from helpers import run_trace, trace_tail_decode

    folder = pc.make_dir(tmp_path, "D")
    launched = []
    call, timed, ops.timing = ops._call, ops._timed, []

    def call_spy(group, name, what, *args):
        launched.append(what)
        return call(group, name, what, *args)

    def timed_spy(what):  # launches that may be refused go past _call
        launched.append(what)
        return timed(what)

    ops._call, ops._timed = call_spy, timed_spy
    try:
        rt = pc.runtime(folder, "D", "bfloat16", ops, DEV, pages=16)
        run_trace(rt, trace_tail_decode(pc.requests_for("D", (70,)), tail=5))
    finally:
        del ops._call, ops._timed
        ops.timing = None
    for kernel in ("paged_attention_prefill_tc", "chunk_attention_prefill", "chunk_attention_decode", "delta_step",
                   "delta_prepare", "delta_chunk_scan", "turn_store", "sum_norm", "embed_norm"):
        assert kernel in launched, f"{kernel} was not launched: {sorted(set(launched))}"
    assert "paged_attention" not in launched
