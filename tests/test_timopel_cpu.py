"""Timopel on the CPU: the engine's host logic (configuration, loading, values shared between layers of a step, batching,
scheduling) and the parts' wiring, with the torch statements of the kernels in place of the kernel table, against
tests/plain_timopel.py."""

import json

import pytest

import timopel_cases as tc
from emulated_ops import TorchOps

OPS, DEV = TorchOps(), "cpu"


def test_config_round_trip_and_refusals(tmp_path):
    from qwen3_runtime_b200.config import TimopelConfig, load_config, resolve_architecture
    from qwen3_runtime_b200.config.model_config import ConfigError

    for name in ("A", "B", "C", "D", "E"):
        cfg = tc.CONFIGS[name]["config"]
        raw = json.loads(json.dumps(cfg.to_hf_config()))
        assert resolve_architecture(raw).config_class is TimopelConfig
        assert TimopelConfig.from_hf_config(raw) == cfg
    assert load_config(tc.make_dir(tmp_path, "A"))[1] == tc.CONFIGS["A"]["config"]
    raw = json.loads(json.dumps(tc.CONFIGS["A"]["config"].to_hf_config()))
    for key, value, match in ((("layers", 0, "type"), "something_else", "unknown mixer type"),
                              (("layers", 0, "mlp", "kind"), "other", "feed-forward"),
                              (("layers", 0, "mixer", "kv_heads"), 4, "multiple of kv_heads"),
                              (("layers", 0, "mixer", "scale"), 0.0, "scale must be positive"),
                              (("layers", 0, "mixer", "q_temp", "every"), 0, "positive integer"),
                              (("layers", 3, "mixer", "vdim"), 24, "mixes 3 value heads of 24 with layer 0"),
                              (("layers", 1, "mlp", "router", "top"), 6, "exceeds experts"),
                              (("layers", 1, "mlp", "shared", "limit"), 0.0, "limit must be positive"),
                              (("norm", "eps"), 0.0, "norm.eps")):
        bad = json.loads(json.dumps(raw))
        at = bad
        for k in key[:-1]:
            at = at[k]
        at[key[-1]] = value
        with pytest.raises(ConfigError, match=match):
            TimopelConfig.from_hf_config(bad)
    # what may be left out
    for path in (("residual_mult",), ("embedding",), ("layers", 0, "mixer", "q_temp"), ("layers", 1, "mlp", "shared"),
                 ("layers", 1, "mlp", "router", "scale"), ("layers", 0, "mixer", "v_mix"), ("layers", 3, "mlp")):
        less = json.loads(json.dumps(raw))
        at = less
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        TimopelConfig.from_hf_config(less)


def test_tensor_names_and_cache_layers(tmp_path):
    from qwen3_runtime_b200.weights.random_init import expected_tensors_for

    specs = expected_tensors_for(tc.CONFIGS["A"]["config"])
    names = set(specs)
    assert {"embed", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2b", "l0.mix.sink", "l0.mix.vmix", "l0.mix.q.norm",
            "l1.mlp.router", "l1.mlp.e4.down", "l1.mlp.shared.up", "l2.mix.vmix", "l3.mix.o"} <= names
    assert not {"head", "l1.mix.vmix", "l2.mlp.shared.up", "l3.norm2", "l3.norm2b", "l3.mlp.gate"} & names
    assert specs["l0.mix.vmix"].shape == () and specs["l0.mix.sink"].shape == (6,) and specs["l1.mix.v"].shape == (12, 72)
    rt = tc.runtime(tc.make_dir(tmp_path, "A"), "A", "float32", OPS, DEV, pages=16)
    assert all(g.kind == "full" for g in rt.cache.groups)
    assert rt.storage.view(0).k_pages.shape[-1] == 24 and rt.storage.view(0).v_pages.shape[-1] == 20
    mixes = [b.mixer.value_mix for b in rt.runner.model.blocks]
    assert mixes == ["source", None, "blend", "blend"]
    assert [b.mixer.value_mix for b in tc.runtime(tc.make_dir(tmp_path, "B"), "B", "float32", OPS, DEV,
                                                 pages=16).runner.model.blocks] == [None, "source", "blend"]


def test_mixer_options_that_do_not_go_together():
    import torch

    from qwen3_runtime_b200.config import PartSpec
    from qwen3_runtime_b200.parts import BuildContext, build_part

    ctx = BuildContext(torch.float32, torch.device("cpu"), OPS)
    base = dict(hidden_size=16, num_heads=2, num_kv_heads=1, dim=8, vdim=8, scale=1.0, qk_norm_eps=1e-5)
    for extra, match in ((dict(qk_norm_eps=None, value_mix="source"), "go with q/k norms"),
                         (dict(qk_norm_eps=None, query_temperature=(0.1, 4)), "go with q/k norms"),
                         (dict(values="keys", value_mix="blend"), "are not mixed"), (dict(value_mix="other"), "value_mix is")):
        with pytest.raises(ValueError, match=match):
            build_part("mixer", PartSpec("sink_window_attention", dict(base, **extra)), ctx)
    with pytest.raises(ValueError, match="silu and gelu"):
        build_part("feed_forward", PartSpec("gated_mlp", dict(hidden_size=8, intermediate_size=8, activation="tanh")), ctx)


@pytest.mark.parametrize("name", ["A", "D", "E"])
def test_every_mechanism_shows(tmp_path, name):
    tc.case_every_mechanism_shows(tmp_path, name)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_schedules(tmp_path, name):
    tc.case_schedules(tmp_path, name, "float32", OPS, DEV, lengths=(50, 9, 2, 41, 1, 30))


@pytest.mark.parametrize("name", ["D", "E"])
def test_schedules_at_tensor_core_sizes(tmp_path, name):
    tc.case_schedules(tmp_path, name, "float32", OPS, DEV, lengths=(60, 2, 21))


def test_schedules_with_bfloat16_activations(tmp_path):
    tc.case_schedules(tmp_path, "C", "bfloat16", OPS, DEV, lengths=(40, 2, 21))


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_stream_after_every_layer(tmp_path, name):
    tc.case_stream_after_every_layer(tmp_path, name, OPS, DEV)


def test_long_decode(tmp_path):
    tc.case_long_decode(tmp_path, "A", "float32", OPS, DEV, total=80)


@pytest.mark.parametrize("name", ["A", "B"])
def test_first_tokens(tmp_path, name):
    tc.case_first_tokens(tmp_path, name, "float32", OPS, DEV)


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_under_the_scheduler(tmp_path, name):
    tc.case_greedy_generation(tmp_path, name, "float32", OPS, DEV)


def test_mixers_alone():
    tc.case_mixers_alone("float32", OPS, DEV)
    tc.case_mixers_alone("float32", OPS, DEV, page_size=4, heads=2, kv_heads=2, dim=16, vdim=16,
                         q_temp=tc.TemperatureConfig(0.8, 1), second=dict(q_temp=None, heads=4))


def test_kernels_alone():
    tc.case_attention_far_keys("float32", OPS, DEV, T=60)
    tc.case_query_temperature(OPS, DEV)
    tc.case_store("float32", OPS, DEV)
    tc.case_routing("float32", OPS, DEV)
    tc.case_feed_forwards_alone("float32", OPS, DEV)
    tc.case_feed_forwards_alone("float32", OPS, DEV, experts=3, top=3, shared=None, scale=1.0)


def test_output_norm_with_multiplier():
    tc.case_output_norm_with_multiplier("float32", OPS, DEV)


def test_model_less_entry():
    """``LLM(model=None, architecture="Timopel")`` builds the design's tiny configuration."""
    from qwen3_runtime_b200 import LLM

    llm = LLM(None, architecture="Timopel", dtype="float32", device=DEV, ops=OPS, cuda_graph=False)
    out = llm.generate([[1, 2, 3], [4, 5]], max_tokens=5)
    assert [len(o) for o in out] == [5, 5]
