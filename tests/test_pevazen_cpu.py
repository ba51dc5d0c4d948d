"""Pevazen on the CPU: the engine's host logic (configuration, loading, keys and values of another layer, pages kept
for several readers, state slots, batching, scheduling) and the parts' wiring, with the torch statements of the
kernels in place of the kernel table, against tests/plain_pevazen.py."""

import json

import pytest

import pevazen_cases as pc
from emulated_ops import TorchOps

OPS, DEV = TorchOps(), "cpu"


def test_config_round_trip_and_refusals(tmp_path):
    from qwen3_runtime_b200.config import PevazenConfig, load_config, resolve_architecture
    from qwen3_runtime_b200.config.model_config import ConfigError

    cfg = pc.CONFIGS["A"]["config"]
    raw = json.loads(json.dumps(cfg.to_hf_config()))
    assert resolve_architecture(raw).config_class is PevazenConfig
    folder = pc.make_dir(tmp_path, "A")
    _arch, read = load_config(folder)
    _raw, tensors = pc.read_dir(folder)
    assert read != cfg  # the low-rank products' ranks are in the tensors only
    assert read.with_tensor_shapes(lambda n: tensors[n].shape) == cfg
    for key, value, match in ((("layers", 0, "type"), "something_else", "unknown layer type"),
                              (("layers", 1, "mlp", "kind"), "other", "feed-forward"),
                              (("layers", 1, "mixer", "kv_heads"), 3, "multiple of kv_heads"),
                              (("layers", 1, "mixer", "rot", "dims"), 26, "even and at most"),
                              (("layers", 1, "mixer", "mask", "size"), 0, "positive integer"),
                              (("layers", 0, "mixer", "left", "vdim"), 27, "even vdim"),
                              (("layers", 0, "mixer", "left", "rot"), None, "rot.base"),
                              (("layers", 2, "mixer", "kv_from"), 2, "earlier attention layer"),
                              (("layers", 2, "mixer", "kv_from"), 0, "earlier attention layer"),
                              (("layers", 4, "mixer", "kv_from"), 2, "earlier attention layer"),
                              (("layers", 2, "mixer", "vdim"), 8, "vdim differs"),
                              (("norm", "eps"), 0.0, "norm.eps")):
        bad = json.loads(json.dumps(raw))
        at = bad
        for k in key[:-1]:
            at = at[k]
        at[key[-1]] = value
        with pytest.raises(ConfigError, match=match):
            PevazenConfig.from_hf_config(bad)


def test_tensor_names_and_cache_layers(tmp_path):
    from qwen3_runtime_b200.weights.random_init import expected_tensors_for

    specs = expected_tensors_for(pc.CONFIGS["A"]["config"])
    names = set(specs)
    assert {"embed", "embed.norm", "head", "final.norm", "l0.norm1", "l0.mix.left.q", "l0.mix.right.A_log",
            "l0.mix.right.v.conv", "l0.mix.left.out", "l0.mix.right.out", "l1.mix.k.b", "l2.mix.q.b", "l4.dwa",
            "l0.mlp.down"} <= names
    assert not {"l2.mix.k", "l2.mix.v", "l2.mix.k.b", "l2.mlp.gate", "l0.norm2", "l0.mix.left.q.b"} & names
    assert specs["l0.norm1"].shape == () and specs["embed.norm"].shape == () and specs["l4.dwa"].shape == (6,)
    rt = pc.runtime(pc.make_dir(tmp_path, "A"), "A", "float32", OPS, DEV, pages=16)
    kinds = sorted((g.kind, str(g.chunk)) for g in rt.cache.groups)
    # the right side's state and ring differ between layers 0 and 3, layer 1's keys are kept for three readers
    assert kinds == [("chunk", "(7, 20, 33)"), ("chunk", "12"), ("full", "None")] + [("state", "None")] * 4
    own, reader = rt.storage.view(1), rt.storage.view(1, writes=False)
    assert own.k_pages.data_ptr() == reader.k_pages.data_ptr() and own.writes and not reader.writes
    assert own.k_pages.shape[-1] == 20 and own.v_pages.shape[-1] == 12
    assert [r.cache for r in rt.runner.model.spec.order] == [0, 1, 1, 3, 1]


def test_averages_over_the_depth_need_their_weights():
    import dataclasses

    from qwen3_runtime_b200.models.pevazen import pevazen_spec
    from qwen3_runtime_b200.config import PartSpec
    from qwen3_runtime_b200.parts import BuildContext, DecoderModel
    import torch

    spec = pevazen_spec(pc.CONFIGS["C"]["config"])
    ctx = BuildContext(torch.float32, torch.device("cpu"), OPS)
    blocks = list(spec.blocks)
    blocks[1] = PartSpec(blocks[1].kind, dict(blocks[1].params, depth_points=5))
    with pytest.raises(ValueError, match="averages over the depth"):
        DecoderModel(dataclasses.replace(spec, blocks=tuple(blocks)), ctx)


def test_pages_for_readers():
    pc.case_pages_for_readers()


def test_frequencies():
    pc.case_frequencies()


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_schedules(tmp_path, name):
    pc.case_schedules(tmp_path, name, "float32", OPS, DEV, lengths=(50, 9, 2, 41, 1, 30))


def test_schedules_at_tensor_core_sizes(tmp_path):
    pc.case_schedules(tmp_path, "D", "float32", OPS, DEV, lengths=(60, 2, 21))


def test_schedules_with_bfloat16_activations(tmp_path):
    pc.case_schedules(tmp_path, "C", "bfloat16", OPS, DEV, lengths=(40, 2, 21))


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_stream_after_every_layer(tmp_path, name):
    pc.case_stream_after_every_layer(tmp_path, name, OPS, DEV)


def test_long_decode(tmp_path):
    pc.case_long_decode(tmp_path, "A", "float32", OPS, DEV, total=80)


@pytest.mark.parametrize("name", ["A", "B"])
def test_first_tokens(tmp_path, name):
    pc.case_first_tokens(tmp_path, name, "float32", OPS, DEV)


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_under_the_scheduler(tmp_path, name):
    pc.case_greedy_generation(tmp_path, name, "float32", OPS, DEV)


def test_mixers_alone():
    pc.case_mixer_alone("float32", OPS, DEV, "attention")
    pc.case_mixer_alone("float32", OPS, DEV, "attention", page_size=4, heads=2, kv_heads=2, dim=16, vdim=16, chunk=None,
                        rot=None)
    pc.case_mixer_alone("float32", OPS, DEV, "parallel")
    pc.case_mixer_alone("float32", OPS, DEV, "parallel", left=dict(chunk=None, vdim=10, dim=24),
                        right=dict(conv=1, heads=3, kv_heads=3, dim=16, vdim=16))


def test_attention_edges():
    pc.case_attention_edges("float32", OPS, DEV)
    pc.case_attention_edges("float32", OPS, DEV, chunk=8, page_size=8, heads=1, kv_heads=1, D=20, Dv=8, turned=True)
    pc.case_attention_batch("float32", OPS, DEV)


def test_kernels_alone():
    pc.case_turn_store("float32", OPS, DEV)
    pc.case_sum_norm("float32", OPS, DEV)
    pc.case_delta_rule("float32", OPS, DEV)
    pc.case_delta_rule("float32", OPS, DEV, H=3, G=1, D=16, Dv=8, taps=1, ra=3, rg=5, decay=0.5)


def test_model_less_entry():
    """``LLM(model=None, architecture="Pevazen")`` builds the design's tiny configuration."""
    from qwen3_runtime_b200 import LLM

    llm = LLM(None, architecture="Pevazen", dtype="float32", device=DEV, ops=OPS, cuda_graph=False)
    out = llm.generate([[1, 2, 3], [4, 5]], max_tokens=5)
    assert [len(o) for o in out] == [5, 5]
