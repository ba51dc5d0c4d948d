"""Timopel: engine and parts against the plain statement (tests/plain_timopel.py), written once and run on the CPU with
the torch statements of the kernels and on the GPU with the kernels."""

from __future__ import annotations

import dataclasses
import json
import math

import torch

import plain_timopel as pl
from helpers import (first_mismatch, max_abs_diff, peak_tokens, random_ids, run_trace, trace_mixed, trace_portions,
                     trace_tail_decode, trace_whole)
from puladra_cases import _random_tensors, _step, _tolerance, _views_for
from qwen3_runtime_b200.config import PartSpec, TimopelConfig
from qwen3_runtime_b200.config.logesun_config import ExpertConfig
from qwen3_runtime_b200.config.timopel_config import (DenseConfig, MixedValueAttentionConfig, MoeConfig,
                                                      TemperatureConfig, TimopelLayerConfig)
from qwen3_runtime_b200.engine.factory import build_engine, build_runtime, load_model
from qwen3_runtime_b200.parts import BuildContext, ResidualStream, build_part
from qwen3_runtime_b200.weights import write_random_model

TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _att(**kw):
    base = dict(heads=6, kv_heads=3, dim=24, vdim=20, scale=0.2, q_temp=TemperatureConfig(0.4, 7), v_mix=True)
    base.update(kw)
    return MixedValueAttentionConfig(**base)


def _moe(experts=5, top=2, scale=1.7, ff=24, limit=0.8, shared=(40, 1.3)):
    return MoeConfig(experts=experts, top=top, scale=scale, expert=ExpertConfig(ff, limit),
                     shared=ExpertConfig(*shared) if shared else None)


def _layer(mixer, mlp):
    return TimopelLayerConfig("attention", mixer, mlp)


# Sizes no two of which are equal where the design lets them differ, and the values that turn a mechanism off or into
# a special case: key and value sizes in either order, that are no multiple of 8, of 64 and 128; one key head for all
# query heads, one for each, groups of 18; a query temperature in steps of one token, of thousands, with a coefficient
# of zero and a negative one, different from layer to layer, absent; values mixed in the first layer and later ones, not
# in the first layer, in a single layer, in none; one chosen expert and all, with and without a shared expert, layers
# without a feed-forward; a residual multiplier and an embedding scale of one, below and above.
CONFIGS = {
    "A": dict(page_size=8, seed=61, config=TimopelConfig(
        vocab=150, width=72, norm_eps=1e-5, embed_scale=2.5, residual_mult=0.4,
        layers=(_layer(_att(), DenseConfig(56)),
                _layer(_att(heads=2, kv_heads=1, dim=20, vdim=12, v_mix=False, q_temp=None, scale=0.3), _moe()),
                _layer(_att(heads=3, dim=12, scale=0.35, q_temp=TemperatureConfig(0.25, 1)),
                       _moe(experts=7, top=1, scale=1.0, ff=16, limit=2.0, shared=None)),
                _layer(_att(heads=9, dim=40, scale=0.15), None)))),
    "B": dict(page_size=4, seed=62, config=TimopelConfig(
        vocab=131, width=64, norm_eps=1e-6, embed_scale=1.0, residual_mult=1.0,
        layers=(_layer(_att(heads=18, kv_heads=1, dim=8, vdim=16, v_mix=False, q_temp=TemperatureConfig(0.0, 3)), None),
                _layer(_att(heads=4, kv_heads=4, dim=16, vdim=8, q_temp=TemperatureConfig(0.5, 4000)),
                       _moe(experts=3, top=3, scale=0.5, ff=40, limit=5.0, shared=(8, 0.5))),
                _layer(_att(heads=4, kv_heads=4, dim=32, vdim=8, q_temp=TemperatureConfig(-0.2, 5)), DenseConfig(24))))),
    "C": dict(page_size=16, seed=63, config=TimopelConfig(
        vocab=90, width=48, norm_eps=1e-5, embed_scale=6.0, residual_mult=1.5,
        layers=(_layer(_att(heads=2, kv_heads=2, dim=16, vdim=40, q_temp=TemperatureConfig(0.6, 20)),
                       _moe(experts=4, top=2, scale=3.0, ff=16, limit=1.0, shared=(16, 1.0))),
                _layer(_att(heads=2, kv_heads=1, dim=24, vdim=24, v_mix=False), DenseConfig(40))))),
    # sizes the bfloat16 tensor-core paths take: heads of 64 (split-KV decode with the newest token inside, mma.sync
    # prompts), of 128 (tcgen05 prompts), keys and values of unlike sizes
    "D": dict(page_size=16, seed=64, config=TimopelConfig(
        vocab=210, width=128, norm_eps=1e-5, embed_scale=4.0, residual_mult=0.6,
        layers=(_layer(_att(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.125, q_temp=TemperatureConfig(0.3, 16)),
                       DenseConfig(96)),
                _layer(_att(heads=4, kv_heads=2, dim=128, vdim=64, scale=0.09), _moe(experts=8, top=2, ff=64, limit=1.0,
                                                                                     shared=(64, 2.0))),
                _layer(_att(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09, v_mix=False,
                            q_temp=TemperatureConfig(0.3, 16)), None),
                _layer(_att(heads=2, kv_heads=2, dim=64, vdim=64, scale=0.125, q_temp=TemperatureConfig(0.5, 9)),
                       _moe(experts=6, top=3, scale=2.5, ff=32, limit=0.6, shared=None))))),
    "E": dict(page_size=16, seed=65, config=TimopelConfig(
        vocab=120, width=96, norm_eps=1e-5, embed_scale=3.5, residual_mult=0.5,
        layers=(_layer(_att(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09, q_temp=TemperatureConfig(0.4, 24)), None),
                _layer(_att(heads=8, kv_heads=1, dim=128, vdim=128, scale=0.09), DenseConfig(80)),
                _layer(_att(heads=2, kv_heads=1, dim=256, vdim=128, scale=0.07), DenseConfig(64))))),
}

STD = 0.15  # spread of the random matrices: attention and the feed-forwards have to matter


def _every_expert(cfg: TimopelConfig) -> TimopelConfig:
    """The same model with every expert chosen for every token: whole models in bfloat16 are tested in this form, since
    with many tokens some pair of router logits always lies within bfloat16 rounding and either choice is right.  The
    choice itself is tested in float32 on whole models and in bfloat16 on the feed-forward alone."""
    return dataclasses.replace(cfg, layers=tuple(
        dataclasses.replace(l, mlp=dataclasses.replace(l.mlp, top=l.mlp.experts)) if isinstance(l.mlp, MoeConfig) else l
        for l in cfg.layers))


for _name in ("A", "B", "C", "D"):
    CONFIGS[_name + "all"] = dict(CONFIGS[_name], config=_every_expert(CONFIGS[_name]["config"]))


def model_for(name, dtype):
    return name + "all" if dtype == "bfloat16" and name + "all" in CONFIGS else name


def make_dir(tmp_path, name):
    spec = CONFIGS[name]
    folder = tmp_path / f"timopel_{name}"
    if not (folder / "model.safetensors").exists():
        from safetensors.torch import load_file, save_file

        write_random_model(spec["config"], folder, spec["seed"], std=STD, vector_std=0.1)
        t = load_file(str(folder / "model.safetensors"))
        for k in t:
            x = t[k].float()
            if k.endswith(".sink"):  # sinks that take a visible share of the weight, some negative
                x = (x - 1.0) * 20.0 + 1.0
            elif k.endswith(".vmix"):  # shares between about 0.2 and 0.8
                x = (x - 1.0) * 2.0 + 0.5
            elif k.endswith((".q.norm", ".k.norm")):  # sharper scores
                x = x * 1.6
            elif k.endswith(".router"):
                x = x * 3.0
            elif k == "embed":
                x = x * 2.0
            t[k] = x.to(t[k].dtype)
        save_file(t, str(folder / "model.safetensors"))
    return folder


def read_dir(folder):
    from safetensors.torch import load_file

    return json.loads((folder / "config.json").read_text()), load_file(str(folder / "model.safetensors"))


def expected(folder, requests, dtype):
    """Plain logits per request and the tolerance: float32 a few 1e-5 of the logits' size; bfloat16 three times the
    distance between the plain statement with bfloat16 activations and the exact one."""
    raw, t = read_dir(folder)
    exact = {rid: pl.forward(raw, t, toks).float() for rid, toks in requests.items()}
    scale = max(float(v.abs().max()) for v in exact.values())
    if dtype == "float32":
        return exact, 5e-5 * max(1.0, scale)
    rounded = {rid: pl.forward(raw, t, toks, activations=torch.bfloat16).float() for rid, toks in requests.items()}
    noise = max(float((rounded[r] - exact[r]).abs().max()) for r in exact)
    return exact, 3.0 * noise


def runtime(folder, name, dtype, ops, device, pages, max_live=4, cuda_graph=False):
    model, _cfg, _ = load_model(folder, dtype=dtype, device=device, ops=ops)
    return build_runtime(model, block_size=CONFIGS[name]["page_size"], num_kv_blocks=pages, max_num_seqs=max_live,
                         cuda_graph=cuda_graph)


def requests_for(name, lengths, seed=0):
    vocab = CONFIGS[name]["config"].vocab
    return {f"r{i}": random_ids(vocab, n, 1000 * seed + i) for i, n in enumerate(lengths)}


def check(got, want, tol, what):
    bad = first_mismatch(got, want, tol)
    assert bad is None, f"{what}: request {bad[0]} position {bad[1]} differs by {bad[2]:.3g} (tolerance {tol:.3g})"
    print(f"{what}: worst difference {max_abs_diff(got, want):.3g} (tolerance {tol:.3g})")


def case_schedules(tmp_path, name, dtype, ops, device, lengths=(75, 9, 41, 2, 58, 1, 30), cuda_graph=False):
    """Whole prompts; the tail decoded token by token; portions down to two tokens; unequal requests side by side with
    pages and slots freed and used again (pages poisoned in between)."""
    name = model_for(name, dtype)
    folder = make_dir(tmp_path, name)
    requests = requests_for(name, lengths)
    want, tol = expected(folder, requests, dtype)
    ps = CONFIGS[name]["page_size"]
    results = {}
    for kind, steps in (("whole", trace_whole(requests)), ("tail", trace_tail_decode(requests, tail=30)),
                        ("portions", trace_portions(requests, seed=3)), ("mixed", trace_mixed(requests, seed=5))):
        rt = runtime(folder, name, dtype, ops, device, pages=-(-peak_tokens(steps, 64) // ps), cuda_graph=cuda_graph)
        results[kind] = run_trace(rt, steps, poison=True)
        check(results[kind], want, tol, f"{name} {dtype} {kind}")
        assert rt.cache.num_free_pages == rt.cache.num_pages
        assert rt.cache.slots.num_free == rt.cache.slots.num_slots
        assert sum(len(v) for v in results[kind].values()) == sum(lengths)
    whole = {rid: torch.stack([rows[p] for p in sorted(rows)]) for rid, rows in results["whole"].items()}
    cut_tol = tol if dtype == "bfloat16" else 2e-5 * max(1.0, max(float(v.abs().max()) for v in whole.values()))
    for kind in ("tail", "portions", "mixed"):
        check(results[kind], whole, cut_tol, f"{name} {dtype} {kind} against whole")


def case_stream_after_every_layer(tmp_path, name, ops, device):
    """The stream after every layer against the plain model's."""
    folder = make_dir(tmp_path, name)
    raw, t = read_dir(folder)
    toks = requests_for(name, (23,), seed=4)["r0"]
    _logits, want = pl.forward(raw, t, toks, with_streams=True)
    rt = runtime(folder, name, "float32", ops, device, pages=-(-64 // CONFIGS[name]["page_size"]))
    got: list = []

    def watched(forward):
        def run(stream, step, cache):
            forward(stream, step, cache)
            # what the block left for the next kernel to norm and add (the weight carries the residual multiplier)
            y = stream.pending.double()
            y = y.sum(0) if y.dim() == 3 else y
            weight, eps = stream.pending_norm[0], stream.pending_norm[1]
            got.append((stream.resid.double() + pl.rms_norm(y, weight.double(), eps)).cpu())
        return run

    for block in rt.runner.model.blocks:
        block.forward = watched(block.forward)
    run_trace(rt, trace_whole({"r0": toks}))
    assert len(got) == len(want) == len(CONFIGS[name]["config"].layers)
    for run, (g, w) in enumerate(zip(got, want)):
        diff = float((g - w).abs().max())
        assert diff <= 3e-5 * max(1.0, float(w.abs().max())), f"{name}: stream after layer {run} off by {diff:.3g}"


def case_every_mechanism_shows(tmp_path, name):
    """The test models are made so that what could be left out would be missed: dropping the sinks, the mixed values,
    the query temperature, the residual multiplier, the embedding scale or the router's scale moves the logits by far
    more than the bfloat16 tolerance."""
    folder = make_dir(tmp_path, name)
    raw, t = read_dir(folder)
    requests = requests_for(name, (40,))
    want, tol = expected(folder, requests, "bfloat16")

    def moved(config, tensors):
        return float((pl.forward(config, tensors, requests["r0"]).float() - want["r0"]).abs().max())

    def without(edit):
        cfg = json.loads(json.dumps(raw))
        edit(cfg)
        return cfg

    def each(edit):
        return lambda cfg: [edit(l) for l in cfg["layers"]]

    assert moved(raw, {k: torch.full_like(v, -1e4) if k.endswith(".sink") else v for k, v in t.items()}) > 1.5 * tol
    assert moved(raw, {k: torch.zeros_like(v) if k.endswith(".vmix") else v for k, v in t.items()}) > 1.5 * tol
    assert moved(without(each(lambda l: l["mixer"].pop("q_temp", None))), t) > 1.5 * tol
    assert moved(without(lambda c: c.update(residual_mult=c["residual_mult"] * 1.5)), t) > 1.5 * tol
    assert moved(without(lambda c: c["embedding"].update(scale=c["embedding"]["scale"] * 1.5)), t) > 1.5 * tol


def case_long_decode(tmp_path, name, dtype, ops, device, total=150, cuda_graph=False):
    """A short prompt and then one token at a time, over many pages and steps of the query temperature."""
    name = model_for(name, dtype)
    folder = make_dir(tmp_path, name)
    requests = requests_for(name, (total,), seed=7)
    want, tol = expected(folder, requests, dtype)
    toks = requests["r0"]
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": toks[:3], "want": [0, 1, 2]}], "end": []}]
    steps += [{"step": i - 2, "entries": [{"id": "r0", "tokens": [toks[i]], "want": [0]}],
               "end": ["r0"] if i == total - 1 else []} for i in range(3, total)]
    rt = runtime(folder, name, dtype, ops, device, pages=-(-(total + 63) // CONFIGS[name]["page_size"]),
                 cuda_graph=cuda_graph)
    check(run_trace(rt, steps), want, tol, f"{name} {dtype} long decode")
    assert rt.cache.num_free_pages == rt.cache.num_pages


def case_first_tokens(tmp_path, name, dtype, ops, device):
    """One-, two- and three-token sequences side by side, then sequences fed one token at a time from their first in the
    slots and pages the others left: a sink beside a single key, the first values of the temperature."""
    name = model_for(name, dtype)
    folder = make_dir(tmp_path, name)
    requests = requests_for(name, (1, 2, 3, 1), seed=9)
    want, tol = expected(folder, requests, dtype)
    steps = [{"step": 0, "entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in requests.items()],
              "end": list(requests)}]
    rt = runtime(folder, name, dtype, ops, device, pages=32)
    check(run_trace(rt, steps, poison=True), want, tol, f"{name} {dtype} first tokens")
    again = requests_for(name, (6, 5), seed=10)
    want, tol = expected(folder, again, dtype)
    steps = [{"step": i, "entries": [{"id": r, "tokens": [t[i]], "want": [0]} for r, t in again.items() if i < len(t)],
              "end": [r for r, t in again.items() if i == len(t) - 1]} for i in range(6)]
    check(run_trace(rt, steps), want, tol, f"{name} {dtype} first tokens one by one in used pages")


def case_greedy_generation(tmp_path, name, dtype, ops, device, cuda_graph=False, steps=12):
    """Greedy generation through the engine's own entry point, scheduler and sampler: unequal prompts side by side in a
    small pool, every token checked at its own place against the plain model given the tokens before it."""
    name = model_for(name, dtype)
    folder = make_dir(tmp_path, name)
    raw, t = read_dir(folder)
    prompts = list(requests_for(name, (17, 3, 29, 8), seed=13).values())
    engine = build_engine(folder, dtype=dtype, device=device, ops=ops, block_size=CONFIGS[name]["page_size"],
                          num_kv_blocks=-(-4 * 64 // CONFIGS[name]["page_size"]), max_num_seqs=3,
                          max_num_batched_tokens=24, cuda_graph=cuda_graph)
    outs = engine.generate_batch(prompts, max_tokens=steps)
    for prompt, out in zip(prompts, outs):
        assert len(out) == steps
        seq = list(prompt) + list(out[:-1])
        exact = pl.forward(raw, t, seq).float()[len(prompt) - 1:]
        if dtype == "float32":
            tol = 1e-4 * max(1.0, float(exact.abs().max()))
        else:
            rows = pl.forward(raw, t, seq, activations=torch.bfloat16).float()[len(prompt) - 1:]
            tol = 2 * 3.0 * float((rows - exact).abs().max())
        for i, tok in enumerate(out):
            gap = float(exact[i].max() - exact[i][tok])
            assert gap <= tol, f"token {i} ({tok}) is {gap:.3g} below the plain argmax (allowed {tol:.3g})"
    engine.runtime.cache.check_invariants()
    assert engine.runtime.cache.num_free_pages == engine.runtime.cache.num_pages


# ---- parts and kernels alone ---------------------------------------------------------------------

def case_mixers_alone(dtype, ops, device, *, T=45, page_size=8, cuts=(24, 1, 2, 18), second=None, **sizes):
    """Two mixing layers' mixers on one sequence in portions (one of a single token, one of two) through paged caches
    whose pages are out of order and hold NaN where nothing was written: the first gives its values to the second, which
    reads an input of its own.  Against the plain statement on the whole sequence; what the sinks and the mixed values
    do shows in it."""
    from qwen3_runtime_b200.models.timopel import _mixer_spec

    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(5)
    width, eps = 64, 1e-5
    cfg = TimopelConfig(vocab=8, width=width, norm_eps=eps, layers=(
        _layer(_att(**sizes), None), _layer(_att(**{**sizes, **(second or {})}), None)))
    ctx = BuildContext(dt, torch.device(device), ops)
    pages_needed = -(-T // page_size)
    table = list(reversed(range(1, pages_needed + 1)))  # not in order, page 0 unused
    parts, caches, inputs, want, first = [], [], [], [], None
    for i in range(2):
        part = build_part("mixer", _mixer_spec(cfg, i), ctx)
        tensors = _random_tensors(part, gen, dt, device)
        tensors["sink"] = (tensors["sink"] - 1.0) * 8.0 + 1.0
        tensors["vmix"] = torch.tensor(0.6, dtype=torch.float32, device=device)
        for n in ("q.norm", "k.norm"):
            tensors[n] = tensors[n] * 1.5
        part.load(tensors)
        raw = cfg.layers[i].mixer.to_raw()
        h = torch.randn((T, width), generator=gen).to(torch.bfloat16).float()
        t = {"mix." + k: v.double().cpu() for k, v in tensors.items()}
        y, own = pl.attention(h.double(), t, "mix.", raw, eps, first)
        open_sinks = pl.attention(h.double(), dict(t, **{"mix.sink": t["mix.sink"] - 1e4}), "mix.", raw, eps, first)[0]
        assert float((open_sinks - y).abs().max()) > 0.02 * float(y.abs().max()), "the sinks hardly matter"
        if i:
            unmixed = pl.attention(h.double(), t, "mix.", raw, eps, None)[0]
            assert float((unmixed - y).abs().max()) > 0.1 * float(y.abs().max()), "the mixed values hardly matter"
        first = own
        parts.append(part)
        caches.append(_views_for(part.cache_spec(), device, dt, page_size, pages_needed + 2, slots=3))
        inputs.append(h)
        want.append(y.float())
    assert sum(cuts) == T
    got, lo = [[], []], 0
    for n in cuts:
        step = _step(list(range(lo, lo + n)), [0] * n, [table], device, slots=[2])
        for i in range(2):
            got[i].append(parts[i].forward(inputs[i][lo:lo + n].to(device=device, dtype=dt), step, caches[i]).float().cpu())
        lo += n
    for i in range(2):
        diff = float((torch.cat(got[i]) - want[i]).abs().max())
        tol = _tolerance(dtype, want[i])
        assert diff <= tol, f"mixer {i} ({dtype}, {sizes}): off by {diff:.3g} (allowed {tol:.3g})"


def _paged(x, table, page_size, pages, dt, device):
    """``x`` ``[T, heads, n]`` into NaN-filled pages ``[pages, heads, page_size, n]`` through ``table``."""
    out = torch.full((pages, x.shape[1], page_size, x.shape[2]), float("nan"), dtype=dt, device=device)
    for j in range(x.shape[0]):
        out[table[j // page_size], :, j % page_size] = x[j].to(dt)
    return out


def case_attention_far_keys(dtype, ops, device, *, page_size=8, heads=4, kv_heads=2, D=12, Dv=20, T=200):
    """The attention kernel alone with one key that takes nearly all of a query's weight: the sequence's first key, keys
    on both sides of a page's border hundreds of tokens back, the query's own; with sinks that differ from head to head
    (one that leaves next to nothing, one that is negligible, one of the marked key's own size), in a whole prompt, a
    portion of two and a single decoded token.  A key that lies after the query is never seen.  Pages are out of order,
    unused rows hold NaN."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(19)
    pages_needed = -(-T // page_size)
    table = list(reversed(range(1, pages_needed + 1)))
    strength = 40.0  # the marked key's score
    sink = torch.tensor([(strength + 6.0, -30.0, strength, strength - 2.0)[h % 4] for h in range(heads)])
    for qi, kj in ((T - 1, 0), (T - 1, page_size - 1), (T - 1, page_size), (T - 2, 1), (T - 1, T - 1), (T // 2, T // 2 + 1),
                   (page_size, page_size - 1), (0, 0)):
        q = 0.05 * torch.randn((T, heads, D), generator=gen)
        k = 0.05 * torch.randn((T, kv_heads, D), generator=gen)
        v = torch.randn((T, kv_heads, Dv), generator=gen)
        q[:, :, D - 3] = 0.0
        k[:, :, D - 3] = 0.0
        k[kj, :, D - 3] = strength / 8.0
        q[qi, :, D - 3] = 8.0
        q, k, v = (x.to(torch.bfloat16).float() for x in (q, k, v))
        want = pl.sink_attention_core(q.double(), k.double(), v.double(), 1.0, sink.double()).float()
        if kj <= qi and heads >= 3 and qi > 0:  # the marked key and the sinks decide the query's output
            per = heads // kv_heads
            size = [float((want[qi, h] / v[kj, h // per]).abs().median()) for h in range(3)]
            assert size[0] < 0.02 and abs(size[1] - 1) < 0.05 and abs(size[2] - 0.5) < 0.1, size
        k_pages = _paged(k, table, page_size, pages_needed + 2, dt, device)
        v_pages = _paged(v, table, page_size, pages_needed + 2, dt, device)
        for lo, hi in ((0, T), (qi - 1, qi + 1), (qi, qi + 1)):
            if lo < 0:
                continue
            step = _step(list(range(lo, hi)), [0] * (hi - lo), [table], device)
            out = torch.zeros((hi - lo, heads * Dv), dtype=dt, device=device)
            qd = q[lo:hi].reshape(hi - lo, heads * D).to(device=device, dtype=dt).contiguous()
            ops.paged_attention(qd, qd.stride(0), num_heads=heads, num_kv_heads=kv_heads, head_dim=D, value_dim=Dv,
                                k_pages=k_pages, v_pages=v_pages, block_table=step.block_tables[0],
                                token_seq=step.token_seq, positions=step.positions, out=out, page_size=page_size,
                                scale=1.0, window=None, step=step, sink=sink.to(device))
            diff = float((out.float().cpu().reshape(hi - lo, heads, Dv) - want[lo:hi]).abs().max())
            tol = 3e-5 if dtype == "float32" else 4e-2
            assert diff <= tol, f"query {qi}, key {kj}, tokens {lo}..{hi}: off by {diff:.3g}"


def case_attention_batch(dtype, ops, device, *, heads=4, kv_heads=1, D=64, Dv=64, page_size=16):
    """Sequences of unequal lengths side by side (portions beside single tokens, then single tokens only), each against
    the plain statement of itself alone, with sinks."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(23)
    lens = (5, 70, 1, 333, 41)
    sink = torch.randn(heads, generator=gen) * 2.0
    kv, tables, first = [], [], 1
    for n in lens:
        kv.append(tuple(torch.randn((n, kv_heads, s), generator=gen).to(torch.bfloat16).float() for s in (D, Dv)))
        tables.append(list(range(first, first + -(-n // page_size))))
        first += -(-n // page_size)
    k_pages = torch.full((first + 1, kv_heads, page_size, D), float("nan"), dtype=dt, device=device)
    v_pages = torch.full((first + 1, kv_heads, page_size, Dv), float("nan"), dtype=dt, device=device)
    for (k, v), table, n in zip(kv, tables, lens):
        for j in range(n):
            k_pages[table[j // page_size], :, j % page_size] = k[j].to(dt)
            v_pages[table[j // page_size], :, j % page_size] = v[j].to(dt)
    qs = [torch.randn((n, heads, D), generator=gen).to(torch.bfloat16).float() for n in lens]
    plain = [pl.sink_attention_core(x.double(), k.double(), v.double(), 0.2, sink.double()).float()
             for (k, v), x in zip(kv, qs)]
    for portions in ((5, 64, 1, 331, 1), (1, 1, 1, 1, 1), (2, 1, 1, 3, 41)):
        positions = [p for n, c in zip(lens, portions) for p in range(n - c, n)]
        seqs = [b for b, c in enumerate(portions) for _ in range(c)]
        step = _step(positions, seqs, tables, device)
        step.single_seqs = torch.tensor([b for b, c in enumerate(portions) if c == 1], dtype=torch.int32, device=device)
        step.num_single = step.single_seqs.numel()
        q = torch.cat([x[n - c:] for x, n, c in zip(qs, lens, portions)])
        qd = q.reshape(len(positions), heads * D).to(device=device, dtype=dt).contiguous()
        out = torch.zeros((len(positions), heads * Dv), dtype=dt, device=device)
        ops.paged_attention(qd, qd.stride(0), num_heads=heads, num_kv_heads=kv_heads, head_dim=D, value_dim=Dv,
                            k_pages=k_pages, v_pages=v_pages, block_table=step.block_tables[0], token_seq=step.token_seq,
                            positions=step.positions, out=out, page_size=page_size, scale=0.2, window=None, step=step,
                            sink=sink.to(device))
        got = out.float().cpu().reshape(len(positions), heads, Dv)
        at = 0
        for want, n, c in zip(plain, lens, portions):
            diff = float((got[at:at + c] - want[n - c:]).abs().max())
            assert diff <= (3e-5 if dtype == "float32" else 4e-2), f"portions {portions}, length {n}: off by {diff:.3g}"
            at += c


def case_query_temperature(ops, device):
    """Positions just before, at and after a step of the temperature, far out, and in steps of one token."""
    for coef, every in ((0.45, 48), (0.37, 7), (-0.2, 1), (0.0, 5), (1.5, 8192)):
        positions = sorted({0, 1, every - 2, every - 1, every, 2 * every - 2, 2 * every - 1, 2 * every, 1000, 131071, 16777214}
                           - {-1})
        got = ops.query_temperature(torch.tensor(positions, dtype=torch.int32, device=device), coef, every).double().cpu()
        want = pl.query_temperature(max(2 * every + 1, 1001), coef, every, torch.float64)
        for p, g in zip(positions, got.tolist()):
            exact = float(want[p]) if p < want.numel() else 1.0 + coef * math.log((p + 1) // every + 1)
            assert abs(g - exact) <= 1e-6 * max(1.0, abs(exact)), f"position {p}, every {every}: {g} for {exact}"
    a, b = ops.query_temperature(torch.tensor([46, 47], dtype=torch.int32, device=device), 0.45, 48).tolist()
    assert a == 1.0 and b > 1.3


def case_store(dtype, ops, device):
    """q/k norms, the query factors, the blend of values and the cache write, with sizes that go through 16-byte accesses
    and sizes that do not; the blended rows come from a wider product; q alone."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(31)
    tol = 2e-5 if dtype == "float32" else 4e-2
    eps, page_size = 1e-5, 4
    positions, seqs = [0, 1, 2, 9, 3, 4, 0], [0, 0, 0, 1, 2, 2, 3]
    tables = [[7], [3, 5, 1], [9, 2], [8]]
    for H, G, D, Dv, blend, factors, write in ((4, 2, 24, 16, True, True, True), (4, 1, 128, 128, True, True, True),
                                               (3, 3, 20, 12, True, False, True), (6, 2, 64, 40, False, True, True),
                                               (2, 1, 18, 10, False, True, True), (8, 4, 64, 64, True, True, False),
                                               (2, 2, 256, 64, True, True, True), (33, 3, 16, 8, True, True, True)):
        T = len(positions)
        k0 = -(-H * D // 8) * 8
        v0 = -(-(k0 + G * D) // 8) * 8
        proj = torch.randn((T, v0 + G * Dv), generator=gen).to(dt)
        wide = torch.randn((T, G * Dv + 24), generator=gen).to(dt)
        wq, wk = 1 + 0.3 * torch.randn(D, generator=gen), 1 + 0.3 * torch.randn(D, generator=gen)
        f = 1 + torch.rand(T, generator=gen)
        x = proj.double()
        q = pl.rms_norm(x[:, :H * D].reshape(T, H, D), wq.double(), eps)
        q = q * f.double()[:, None, None] if factors else q
        k = pl.rms_norm(x[:, k0:k0 + G * D].reshape(T, G, D), wk.double(), eps)
        v = x[:, v0:].reshape(T, G, Dv)
        v = pl.mix_values(v, wide[:, 16:16 + G * Dv].double().reshape(T, G, Dv), 0.3) if blend else v
        k_pages = torch.full((11, G, page_size, D), float("nan"), dtype=dt, device=device)
        v_pages = torch.full((11, G, page_size, Dv), float("nan"), dtype=dt, device=device)
        step = _step(positions, seqs, tables, device)
        pd, wd = proj.clone().to(device), wide.to(device)
        ops.qk_norm_store(pd, num_heads=H, num_kv_heads=G, head_dim=D, value_dim=Dv, k_start=k0, v_start=v0,
                          q_weight=wq.to(device), k_weight=wk.to(device), eps=eps, positions=step.positions,
                          token_seq=step.token_seq, block_table=step.block_tables[0], k_pages=k_pages, v_pages=v_pages,
                          page_size=page_size, write_kv=write, q_scale=f.to(device) if factors else None,
                          first_values=wd[:, 16:16 + G * Dv] if blend else None, value_share=0.3 if blend else 0.0)
        what = f"H={H} G={G} D={D} Dv={Dv}"
        assert float((pd[:, :H * D].double().cpu().reshape(T, H, D) - q).abs().max()) <= tol * 2, what
        assert torch.equal(pd[:, k0:].cpu(), proj[:, k0:]), what
        for t, (p, s) in enumerate(zip(positions, seqs)):
            kp = k_pages[tables[s][p // page_size], :, p % page_size].double().cpu()
            vp = v_pages[tables[s][p // page_size], :, p % page_size].double().cpu()
            if not write:
                assert bool(torch.isnan(kp).all()) and bool(torch.isnan(vp).all())
                continue
            assert float((kp - k[t]).abs().max()) <= tol and float((vp - v[t]).abs().max()) <= tol, what


def case_routing(dtype, ops, device):
    """The choice and the weights alone, with factors on the weights, one choice and all of them."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(4)
    T, W = 33, 40
    h = torch.randn((T, W), generator=gen).to(dt).float()
    for E, top, scale in ((8, 2, 2.0), (5, 5, 0.5), (9, 1, 1.0), (40, 6, 3.0), (1, 1, 2.5)):
        router = 0.4 * torch.randn((E, W), generator=gen)
        want = pl.route(h.double() @ router.double().T, top, scale).float()
        chosen, weights = ops.route_top(h.to(device=device, dtype=dt), router.to(device), top, renormalize=True,
                                        score="softmax_all", scale=scale)
        got = torch.zeros(T, E).scatter_(1, chosen.long().cpu(), weights.cpu())
        assert float((got - want).abs().max()) < 1e-5 * max(1.0, scale), f"{top} of {E}"
        assert float((weights.sum(-1).cpu() - scale).abs().max()) < 1e-5 * max(1.0, scale)


def case_feed_forwards_alone(dtype, ops, device, *, experts=6, top=3, scale=1.8, ff=40, limit=0.75, shared=(24, 1.2), T=37,
                             width=48):
    """The routed experts and the dense gelu layer against their plain statements, with inputs large enough for all
    three clamps to bind in the experts and in the shared one."""
    from qwen3_runtime_b200.models.timopel import _feed_forward_spec

    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(8)
    cfg = TimopelConfig(vocab=8, width=width, norm_eps=1e-5, layers=(_layer(_att(), None),))
    ctx = BuildContext(dt, torch.device(device), ops)
    h = torch.randn((T, width), generator=gen).to(torch.bfloat16).float()
    for f in (_moe(experts, top, scale, ff, limit, shared), DenseConfig(ff)):
        part = build_part("feed_forward", _feed_forward_spec(cfg, f), ctx)
        tensors = _random_tensors(part, gen, dt, device, std=0.3)
        part.load(tensors)
        t = {"mlp." + k: v.double().cpu() for k, v in tensors.items()}
        want = pl.feed_forward(h.double(), t, "mlp.", f.to_raw()).float()
        if isinstance(f, MoeConfig):
            for name, lim in (("e0", limit), *((("shared", shared[1]),) if shared else ())):
                g, u = h.double() @ t[f"mlp.{name}.gate"].T, h.double() @ t[f"mlp.{name}.up"].T
                assert (g > lim).any() and (u > lim).any() and (u < -lim).any() and (g < -lim).any()
        got = part.forward(h.to(device=device, dtype=dt), None)
        got = (got.sum(0) if got.dim() == 3 else got).float().cpu()
        diff = float((got - want).abs().max())
        assert diff <= _tolerance(dtype, want), f"{f} ({dtype}): off by {diff:.3g}"


def case_output_norm_with_multiplier(dtype, ops, device):
    """A sublayer's output normed with a multiplier, added to the scaled embedding rows, and the next norm: a finished
    output and partial sums of one."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(6)
    ctx = BuildContext(dt, torch.device(device), ops)
    for W, mult in ((48, 0.3), (520, 1.0), (90, 2.0)):
        embed = torch.randn((11, W), generator=gen).to(torch.bfloat16).float()
        w1, wb = (1 + 0.3 * torch.randn(W, generator=gen) for _ in range(2))
        y = torch.randn((3, 5, W), generator=gen)
        part = build_part("embedding", PartSpec("scaled_bigram", dict(vocab_size=11, hidden_size=W, scale=2.5)), ctx)
        part.load({"embed": embed.to(device=device, dtype=dt)})
        norms = []
        for w, m in ((w1, 1.0), (wb, mult)):
            n = build_part("norm", PartSpec("rmsnorm", dict(size=W, eps=1e-5, weight_name="", weight_scale=m)), ctx)
            n.load({"": w.to(device)})
            norms.append(n)
        ids = [3, 10, 0, 3, 7]
        step = _step(list(range(5)), [0] * 5, [[1]], device, ids=ids)
        for planes in (False, True):
            stream = part.start(step, None, False)
            assert isinstance(stream, ResidualStream)
            pending = y.to(device) if planes else y.sum(0).to(device=device, dtype=dt)
            stream.pending, stream.pending_norm = pending, norms[1].pending_scale()
            exact = pending.double().cpu()
            exact = exact.sum(0) if planes else exact
            x = embed[ids].double() * 2.5 + mult * pl.rms_norm(exact, wb.double(), 1e-5)
            out = norms[0].add_norm(stream)
            tol = 2e-5 if dtype == "float32" else 3e-2
            assert float((stream.resid.double().cpu() - x).abs().max()) <= 2e-5
            assert float((out.double().cpu() - pl.rms_norm(x, w1.double(), 1e-5)).abs().max()) <= tol
