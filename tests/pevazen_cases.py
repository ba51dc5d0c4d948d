"""Pevazen: engine and parts against the plain statement (tests/plain_pevazen.py), written once and run on the CPU
with the torch statements of the kernels and on the GPU with the kernels."""

from __future__ import annotations

import dataclasses
import json

import torch

import plain_pevazen as pl
from helpers import (first_mismatch, max_abs_diff, peak_tokens, random_ids, run_trace, trace_mixed, trace_portions,
                     trace_tail_decode, trace_whole)
from puladra_cases import _random_tensors, _step, _tolerance, _views_for
from qwen3_runtime_b200.config import PartSpec, PevazenConfig
from qwen3_runtime_b200.config.pevazen_config import (ChunkedAttentionConfig, DeltaConfig, PevazenLayerConfig,
                                                      SideBySideConfig)
from qwen3_runtime_b200.config.tabisun_config import RotaryConfig
from qwen3_runtime_b200.engine.factory import build_engine, build_runtime, load_model
from qwen3_runtime_b200.parts import BuildContext, build_part
from qwen3_runtime_b200.weights import write_random_model

TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
L = PevazenLayerConfig


def _rot(dims, base, factor=None):
    return RotaryConfig(dims=dims, base=base, scaling=(("factor", factor),) if factor else ())


def _attn(**kw):
    base = dict(heads=4, kv_heads=2, dim=20, vdim=12, scale=0.3, rot=_rot(12, 1000.0), chunk=20)
    base.update(kw)
    return ChunkedAttentionConfig(**base)


def _left(**kw):
    base = dict(heads=6, kv_heads=3, dim=16, vdim=28, scale=0.25, rot=_rot(16, 300.0, 3.0), chunk=12)
    base.update(kw)
    return ChunkedAttentionConfig(**base)


def _delta(**kw):
    base = dict(heads=4, kv_heads=2, dim=12, vdim=20, conv=4, decay_rank=6, gate_rank=10)
    base.update(kw)
    return DeltaConfig(**base)


def _side(left=None, right=None):
    return SideBySideConfig(left or _left(), right or _delta())


# Sizes no two of which are equal where the design lets them differ: key and value sizes on both sides of each other,
# head counts with and without groups, sizes that are no multiple of 8, chunks that are no multiple of the page, of
# one token, larger than any request and absent, readers of another layer's keys under smaller and larger chunks than
# the owner's (and two readers of one owner), rotation over the whole head and over a part of it, with and without a
# factor, convolutions of 4, 2 and 1 taps, ranks that differ, layers without a feed-forward, either mixer first and last.
CONFIGS = {
    "A": dict(page_size=8, seed=61, config=PevazenConfig(
        vocab=150, width=72, norm_eps=1e-5,
        layers=(L("parallel", _side(), 56), L("attention", _attn(), 40), L("attention", _attn(kv_from=1, chunk=33), None),
                L("parallel", _side(_left(heads=2, kv_heads=2, chunk=None), _delta(conv=2, heads=2)), None),
                L("attention", _attn(kv_from=1, chunk=7, scale=0.4), 48)))),
    "B": dict(page_size=4, seed=62, config=PevazenConfig(
        vocab=131, width=64, norm_eps=1e-6,
        layers=(L("attention", _attn(heads=2, kv_heads=1, dim=16, vdim=24, chunk=1, rot=_rot(16, 50.0, 2.0)), None),
                L("parallel", _side(_left(heads=3, kv_heads=1, dim=8, vdim=16, chunk=9, rot=_rot(4, 100.0)),
                                    _delta(heads=3, kv_heads=1, dim=16, vdim=8, conv=1, decay_rank=3, gate_rank=5)), 48),
                L("attention", _attn(heads=4, kv_heads=4, dim=24, vdim=40, chunk=None, rot=_rot(10, 1e4)), 24)))),
    "C": dict(page_size=16, seed=63, config=PevazenConfig(
        vocab=90, width=48, norm_eps=1e-4,
        layers=(L("attention", _attn(heads=2, kv_heads=1, dim=16, vdim=32, chunk=16, rot=_rot(8, 1e4)), 32),
                L("attention", _attn(heads=2, kv_heads=1, dim=16, vdim=32, chunk=200, rot=_rot(8, 1e4), kv_from=0), 40),
                L("parallel", _side(_left(heads=2, kv_heads=1, dim=24, vdim=8, chunk=30, rot=_rot(24, 1e4, 1.5)),
                                    _delta(heads=6, kv_heads=3, dim=8, vdim=24, conv=3, decay_rank=8, gate_rank=8)), 24)))),
    # sizes the bfloat16 tensor-core paths take
    "D": dict(page_size=16, seed=64, config=PevazenConfig(
        vocab=210, width=128, norm_eps=1e-5,
        layers=(L("parallel", _side(_left(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.125, chunk=48, rot=_rot(64, 1e4, 4.0)),
                                    _delta(heads=4, kv_heads=2, dim=64, vdim=64, decay_rank=16, gate_rank=24)), 96),
                L("attention", _attn(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09, chunk=80, rot=_rot(64, 5e4)), 64),
                L("attention", _attn(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09, chunk=56, rot=_rot(64, 5e4),
                                     kv_from=1), 96),
                L("parallel", _side(_left(heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, chunk=112, rot=_rot(96, 1e4)),
                                    _delta(heads=2, kv_heads=2, dim=128, vdim=128, decay_rank=8, gate_rank=8)), None),
                L("attention", _attn(heads=8, kv_heads=2, dim=96, vdim=48, scale=0.1, chunk=40, rot=_rot(32, 1e4)), None)))),
}

STD = 0.15  # spread of the random matrices: mixers and feed-forwards have to matter


def _shape_vectors(name, x):
    """Random vectors turned into ones that make every mechanism show."""
    leaf = name.split(".")[-1]
    if leaf == "A_log":  # decays from nearly none to strong
        return (x - 1.0) * 15.0 - 2.0
    if leaf == "dt_bias":
        return (x - 1.0) * 10.0
    if leaf == "dwa":  # weights of either sign, the newest point around one
        w = (x - 1.0) * 5.0
        w[-1] += 1.0
        return w
    if name.endswith((".q.b", ".k.b", ".v.b")):
        return (x - 1.0) * 5.0
    return x


def make_dir(tmp_path, name):
    spec = CONFIGS[name]
    folder = tmp_path / f"pevazen_{name}"
    if not (folder / "model.safetensors").exists():
        from safetensors.torch import load_file, save_file

        write_random_model(spec["config"], folder, spec["seed"], std=STD, vector_std=0.1)
        t = load_file(str(folder / "model.safetensors"))
        for k in t:
            x = _shape_vectors(k, t[k].float())
            if k.endswith((".q", ".k")):  # sharper scores
                x = x * 2.0
            elif k.endswith((".conv", ".a2", ".g2", ".b", ".a1", ".g1")) and not k.endswith((".q.b", ".k.b", ".v.b")):
                x = x * 3.0
            t[k] = x.to(t[k].dtype)
        save_file(t, str(folder / "model.safetensors"))
    return folder


def read_dir(folder):
    from safetensors.torch import load_file

    return json.loads((folder / "config.json").read_text()), load_file(str(folder / "model.safetensors"))


def expected(folder, requests, dtype):
    """Plain logits per request and the tolerance: float32 a few 1e-5 of the logits' size; bfloat16 three
    times the distance between the plain statement with bfloat16 activations and the exact one."""
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
    """Whole prompts; the tail decoded token by token; portions down to two tokens; unequal requests side by
    side with pages and slots freed and used again (pages poisoned in between)."""
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
    cut_tol = tol if dtype == "bfloat16" else 4e-5 * max(1.0, max(float(v.abs().max()) for v in whole.values()))
    for kind in ("tail", "portions", "mixed"):
        check(results[kind], whole, cut_tol, f"{name} {dtype} {kind} against whole")


def case_stream_after_every_layer(tmp_path, name, ops, device):
    """The averaged stream after every layer against the plain model's."""
    folder = make_dir(tmp_path, name)
    raw, t = read_dir(folder)
    toks = requests_for(name, (23,), seed=4)["r0"]
    _logits, want = pl.forward(raw, t, toks, with_streams=True)
    rt = runtime(folder, name, "float32", ops, device, pages=-(-64 // CONFIGS[name]["page_size"]))
    got: list = []

    def watched(block, forward):
        def run(stream, step, cache):
            forward(stream, step, cache)
            # what the block left for the next kernel: outputs (some to be normed), then the average over the depth
            v = stream.resid.cpu().double()
            for a in stream.addends:
                x = a.value.float().cpu().double()
                x = x.sum(0) if x.dim() == 3 else x
                v = v + (pl.unit_rms(x, a.norm_eps) * a.norm_weight.cpu().double() if a.norm_weight is not None else x)
            points = [stream.points[j].cpu().double() for j in range(stream.num_points)] + [v]
            got.append(pl.depth_average(points, stream.depth_weights.cpu().double()))
        return run

    for block in rt.runner.model.blocks:
        block.forward = watched(block, block.forward)
    run_trace(rt, trace_whole({"r0": toks}))
    assert len(got) == len(want) == len(CONFIGS[name]["config"].layers)
    for run, (g, w) in enumerate(zip(got, want)):
        diff = float((g - w).abs().max())
        assert diff <= 3e-5 * max(1.0, float(w.abs().max())), f"{name}: stream after layer {run} off by {diff:.3g}"


def case_long_decode(tmp_path, name, dtype, ops, device, total=150, cuda_graph=False):
    """A short prompt and then one token at a time, over many chunks and pages."""
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
    """One-, two- and three-token sequences side by side, then sequences fed one token at a time from their
    first in the slots and pages the others left: convolutions whose taps reach before the start, a state that has to
    be zero again, chunks not yet full."""
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
    """Greedy generation through the engine's own entry point, scheduler and sampler: unequal prompts side by
    side in a small pool, every token checked at its own place against the plain model given the tokens
    before it."""
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

def case_mixer_alone(dtype, ops, device, kind, *, T=45, page_size=8, cuts=(24, 1, 2, 18), left=None, right=None, **sizes):
    """A mixer on one sequence in portions (one of a single token, one of two) through a paged cache whose
    pages are out of order and hold NaN where nothing was written, and state slots that are not the first, against the
    plain statement on the whole sequence.  ``attention`` is run a second time as a reader of the first one's keys
    under another chunk size."""
    from qwen3_runtime_b200.models.pevazen import _mixer_spec

    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(5)
    width, eps = 64, 1e-5
    m = _attn(**sizes) if kind == "attention" else _side(_left(**(left or {})), _delta(**(right or {})))
    cfg = PevazenConfig(vocab=8, width=width, norm_eps=eps, layers=(L(kind, m, None),))
    ctx = BuildContext(dt, torch.device(device), ops)
    mixers = [m]
    if kind == "attention":
        mixers.append(dataclasses.replace(m, chunk=(m.chunk or 0) + 5, scale=m.scale * 1.3, kv_from=0))
    parts, tensors = [], []
    for mm in mixers:
        part = build_part("mixer", _mixer_spec(cfg, mm), ctx)
        t = _random_tensors(part, gen, dt, device)
        for name in t:
            t[name] = _shape_vectors(name, t[name]) if not name.endswith((".q.b", ".k.b", ".v.b")) else t[name] - 1.0
            if name in ("q.b", "k.b", "v.b"):
                t[name] = (t[name] - 1.0) * 3.0
            t[name] = t[name].to(torch.bfloat16).to(t[name].dtype)
        part.load(dict(t))
        parts.append(part)
        tensors.append({"mix." + k: v.double().cpu() for k, v in t.items()})
    h = torch.randn((T, width), generator=gen).to(torch.bfloat16).float()
    if kind == "attention":
        first, kept = pl.biased_attention(h.double(), tensors[0], "mix.", m.to_raw(), None)
        second, _ = pl.biased_attention(h.double(), tensors[1], "mix.", mixers[1].to_raw(), kept)
        want = [first.float(), second.float()]
    else:
        want = [pl.side_by_side(h.double(), tensors[0], "mix.", m.to_raw(), eps).float()]
    pages_needed = -(-T // page_size)
    table = list(reversed(range(1, pages_needed + 1)))  # not in order, page 0 unused
    cache = _views_for(parts[0].cache_spec(), device, dt, page_size, pages_needed + 2, slots=3)
    got, lo = [[] for _ in parts], 0
    assert sum(cuts) == T
    for n in cuts:
        step = _step(list(range(lo, lo + n)), [0] * n, [table], device, slots=[2])
        x = h[lo:lo + n].to(device=device, dtype=dt)
        for i, part in enumerate(parts):
            if i == 1:
                cache = dataclasses.replace(cache, writes=False)
            y = part.forward(x, step, cache)
            if kind == "attention":
                got[i].append((y.sum(0) if y.dim() == 3 else y).float().cpu())
            else:  # two outputs, each with its norm
                total = 0
                for a in y:
                    v = a.value.float().cpu()
                    total = total + pl.unit_rms(v.sum(0) if v.dim() == 3 else v, a.norm_eps) * a.norm_weight.cpu()
                got[i].append(total)
        if kind == "attention":
            cache = dataclasses.replace(cache, writes=True)
        lo += n
    for i, (g, w) in enumerate(zip(got, want)):
        diff = float((torch.cat(g) - w).abs().max())
        tol = _tolerance(dtype, w)
        assert diff <= tol, f"{kind} mixer {i} ({dtype}, {m}): off by {diff:.3g} (allowed {tol:.3g})"


def _paged(x, table, page_size, pages, dt, device):
    """``x`` ``[T, heads, n]`` into NaN-filled pages ``[pages, heads, page_size, n]`` through ``table``."""
    out = torch.full((pages, x.shape[1], page_size, x.shape[2]), float("nan"), dtype=dt, device=device)
    for j in range(x.shape[0]):
        out[table[j // page_size], :, j % page_size] = x[j].to(dt)
    return out


def case_attention_edges(dtype, ops, device, *, chunk=12, page_size=8, heads=4, kv_heads=2, D=12, Dv=20, T=50,
                         turned=False):
    """The attention kernel alone with one key that takes nearly all of a query's weight when it is seen: just inside
    the query's chunk it decides the output, one position before the chunk's start it does not; for queries at a
    chunk's first, second and last position, at page borders, in a whole prompt, a portion of two and a single decoded
    token.  ``turned``: the cached values are turned by their positions and the sum is turned back.  Pages are out of
    order; unused rows hold NaN, and so do the pages that lie wholly before the step's first chunk."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(17)
    pages_needed = -(-T // page_size)
    table = list(reversed(range(1, pages_needed + 1)))
    cases = []
    for qi in (2 * chunk, 2 * chunk + 1, 3 * chunk - 1, T - 1):
        start = qi // chunk * chunk
        cases += [(chunk, qi, start), (chunk, qi, start - 1)]
    cases += [(None, T - 1, 0), (1, T - 1, T - 2), (1, 7, 7), (T + 5, T - 1, 1)]
    base = 80.0
    for ch, qi, kj in cases:
        q = 0.3 * torch.randn((T, heads, D), generator=gen)
        k = 0.3 * torch.randn((T, kv_heads, D), generator=gen)
        v = torch.randn((T, kv_heads, Dv), generator=gen)
        k[kj, :, D - 3] += 8.0
        q[qi, :, D - 3] += 8.0
        q, k, v = (x.to(torch.bfloat16).float() for x in (q, k, v))

        def plain(keys):
            if turned:
                return pl.turned_values_core(q.double(), keys.double(), v.double(), 1.0, ch, base).float()
            return pl.attention_core(q.double(), keys.double(), v.double(), 1.0, ch).float()

        want = plain(k)
        blind = k.clone()
        blind[kj, :, D - 3] -= 8.0
        moved = float((plain(blind)[qi] - want[qi]).abs().max())
        seen = kj <= qi and (ch is None or kj // ch == qi // ch)
        if qi > (qi // ch * ch if ch else 0) + 1:  # (with one or two visible keys the scores hardly matter)
            assert (moved > 0.1) == seen, "the marked key does not stand out as intended"
        pos = torch.arange(T)
        inv = pl.frequencies(Dv, base, torch.float32) if turned else None
        stored = pl.rotate(v.double(), pos, pl.frequencies(Dv, base, torch.float64)).float() if turned else v
        k_pages = _paged(k, table, page_size, pages_needed + 2, dt, device)
        v_pages = _paged(stored, table, page_size, pages_needed + 2, dt, device)
        for lo, hi in ((0, T), (qi - 1, qi + 1), (qi, qi + 1)):  # a whole prompt; a portion of two; one decoded token
            if lo < 0:
                continue
            kp, vp = k_pages.clone(), v_pages.clone()
            gone = list(table)
            if ch:  # pages given back: their entries are -1 and their contents somebody else's
                for idx in range(lo // ch * ch // page_size):
                    kp[table[idx]] = vp[table[idx]] = float("nan")
                    gone[idx] = -1
            step = _step(list(range(lo, hi)), [0] * (hi - lo), [gone], device)
            out = torch.zeros((hi - lo, heads * Dv), dtype=dt, device=device)
            qd = q[lo:hi].reshape(hi - lo, heads * D).to(device=device, dtype=dt).contiguous()
            turns = ops.turn_table(step.positions, inv.to(device)) if turned else None
            ops.paged_attention(qd, qd.stride(0), num_heads=heads, num_kv_heads=kv_heads, head_dim=D, value_dim=Dv,
                                k_pages=kp, v_pages=vp, block_table=step.block_tables[0], token_seq=step.token_seq,
                                positions=step.positions, out=out, page_size=page_size, scale=1.0, window=None,
                                chunk=ch, step=step, value_turns=turns)
            diff = float((out.float().cpu().reshape(hi - lo, heads, Dv) - want[lo:hi]).abs().max())
            # (turned: angles of hundreds of radians carry the rounding of their float32 products)
            tol = (4e-4 if turned else 3e-5) if dtype == "float32" else 4e-2
            assert diff <= tol, f"chunk {ch}, query {qi}, key {kj}, tokens {lo}..{hi}: off by {diff:.3g}"


def case_attention_batch(dtype, ops, device, *, heads=4, kv_heads=1, D=64, Dv=64, chunk=40, page_size=16, turned=True):
    """Sequences of unequal lengths side by side (portions beside single tokens, then single tokens only), each against
    itself alone."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(23)
    lens = (5, 70, 1, 133, 41)
    base = 500.0
    kv, tables, first = [], [], 1
    for n in lens:
        kv.append((torch.randn((n, kv_heads, D), generator=gen), torch.randn((n, kv_heads, Dv), generator=gen)))
        tables.append(list(range(first, first + -(-n // page_size))))
        first += -(-n // page_size)
    k_pages = torch.full((first + 1, kv_heads, page_size, D), float("nan"), dtype=dt, device=device)
    v_pages = torch.full((first + 1, kv_heads, page_size, Dv), float("nan"), dtype=dt, device=device)
    f64, f32 = pl.frequencies(Dv, base, torch.float64), pl.frequencies(Dv, base, torch.float32)
    for (k, v), table, n in zip(kv, tables, lens):
        stored = pl.rotate(v.double(), torch.arange(n), f64).float() if turned else v
        for j in range(n):
            k_pages[table[j // page_size], :, j % page_size] = k[j].to(dt)
            v_pages[table[j // page_size], :, j % page_size] = stored[j].to(dt)
    for portions in ((5, 64, 1, 131, 1), (1, 1, 1, 1, 1), (2, 1, 1, 3, 41)):
        positions = [p for n, c in zip(lens, portions) for p in range(n - c, n)]
        seqs = [b for b, c in enumerate(portions) for _ in range(c)]
        step = _step(positions, seqs, tables, device)
        step.single_seqs = torch.tensor([b for b, c in enumerate(portions) if c == 1], dtype=torch.int32, device=device)
        step.num_single = step.single_seqs.numel()
        qs = [torch.randn((n, heads, D), generator=gen).to(torch.bfloat16).float() for n in lens]
        q = torch.cat([x[n - c:] for x, n, c in zip(qs, lens, portions)])
        qd = q.reshape(len(positions), heads * D).to(device=device, dtype=dt).contiguous()
        out = torch.zeros((len(positions), heads * Dv), dtype=dt, device=device)
        turns = ops.turn_table(step.positions, f32.to(device)) if turned else None
        ops.paged_attention(qd, qd.stride(0), num_heads=heads, num_kv_heads=kv_heads, head_dim=D, value_dim=Dv,
                            k_pages=k_pages, v_pages=v_pages, block_table=step.block_tables[0], token_seq=step.token_seq,
                            positions=step.positions, out=out, page_size=page_size, scale=0.2, window=None, chunk=chunk,
                            step=step, value_turns=turns)
        got = out.float().cpu().reshape(len(positions), heads, Dv)
        at = 0
        for (k, v), x, n, c in zip(kv, qs, lens, portions):
            kk = k.to(dt).double()
            if turned:
                want = pl.turned_values_core(x.double(), kk, v.double(), 0.2, chunk, base)[n - c:].float()
            else:
                want = pl.attention_core(x.double(), kk, v.double(), 0.2, chunk)[n - c:].float()
            diff = float((got[at:at + c] - want).abs().max())
            assert diff <= (3e-5 if dtype == "float32" else 4e-2), f"portions {portions}, length {n}: off by {diff:.3g}"
            at += c


def case_turn_store(dtype, ops, device):
    """Biases, rotation of q, k and values, and the cache write, with sizes that go through 16-byte accesses and sizes
    that do not, rotations over a part of the head, either pairing, positions in the thousands, q alone."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(29)
    tol = 2e-3 if dtype == "float32" else 4e-2  # (positions of thousands: the angle's own rounding)
    T, page_size = 7, 4
    positions = [0, 1, 2, 3, 2050, 2051, 2052]
    table = list(reversed(range(1, 520)))
    step = _step(positions, [0] * T, [table], device)
    pos = torch.tensor(positions)
    for H, G, D, Dv, qn, turned, bias, pairing, write in (
            (4, 2, 24, 16, 8, True, True, "half", True), (4, 2, 16, 32, 8, True, False, "half", True),
            (2, 1, 20, 12, 3, True, True, "half", True), (3, 3, 32, 8, 16, False, True, "half", True),
            (2, 2, 12, 20, 4, True, True, "interleaved", True), (4, 1, 64, 24, 16, False, True, "half", False),
            (2, 1, 16, 16, 0, False, True, "half", True)):
        k0, v0 = H * D, (H + G) * D
        proj = torch.randn((T, v0 + G * Dv), generator=gen).to(dt)
        b = torch.randn(v0 + G * Dv, generator=gen) if bias else None
        x = proj.double() + (b.double() if bias else 0.0)
        fq = torch.tensor([0.8 ** i for i in range(qn)], dtype=torch.float32)
        fv = torch.tensor([0.6 ** i for i in range(Dv // 2)], dtype=torch.float32)

        def turn(y, f):
            if f.numel() == 0:
                return y
            if pairing == "half":
                return pl.rotate(y, pos, f.double())
            n = f.numel()
            idx = torch.cat([torch.arange(0, 2 * n, 2), torch.arange(1, 2 * n, 2), torch.arange(2 * n, y.shape[-1])])
            out = torch.empty_like(y)
            out[..., idx] = pl.rotate(y[..., idx], pos, f.double())
            return out

        q = turn(x[:, :k0].reshape(T, H, D), fq)
        k = turn(x[:, k0:v0].reshape(T, G, D), fq)
        v = x[:, v0:].reshape(T, G, Dv)
        v = turn(v, fv) if turned else v
        k_pages = torch.full((521, G, page_size, D), float("nan"), dtype=dt, device=device)
        v_pages = torch.full((521, G, page_size, Dv), float("nan"), dtype=dt, device=device)
        pd = proj.clone().to(device)
        ops.turn_store(pd, num_heads=H, num_kv_heads=G, head_dim=D, value_dim=Dv, k_start=k0, v_start=v0,
                       bias=b.to(device) if bias else None,
                       qk_turns=ops.turn_table(step.positions, fq.to(device)) if qn else None,
                       value_turns=ops.turn_table(step.positions, fv.to(device)) if turned else None,
                       positions=step.positions, token_seq=step.token_seq, block_table=step.block_tables[0],
                       k_pages=k_pages, v_pages=v_pages, page_size=page_size, write_kv=write, pairing=pairing)
        assert float((pd[:, :k0].float().cpu().reshape(T, H, D) - q.float()).abs().max()) <= tol
        assert torch.equal(pd[:, k0:].cpu(), proj[:, k0:])
        for t, p in enumerate(positions):
            kp, vp = k_pages[table[p // page_size], :, p % page_size].float().cpu(), v_pages[table[p // page_size], :, p % page_size].float().cpu()
            if not write:
                assert bool(torch.isnan(kp).all()) and bool(torch.isnan(vp).all())
                continue
            assert float((kp - k[t].float()).abs().max()) <= tol and float((vp - v[t].float()).abs().max()) <= tol


def _delta_inputs(gen, T, H, G, D, Dv, taps, ra, rg, decay):
    """Raw channels, low-rank rows, steps and weights of one sequence; ``decay``: A_log."""
    C = 2 * G * D + H * Dv
    r = lambda *s: torch.randn(s, generator=gen)  # noqa: E731
    return dict(x=r(T, C), low_a=r(T, ra), low_g=r(T, rg), b=r(T, H), a2=r(H * D, ra) * 0.3, g2=r(H * Dv, rg) * 0.3,
                conv=r(C, taps), a_log=torch.full((H,), decay) + 0.3 * r(H), dt_bias=r(H * D), norm=1 + 0.2 * r(Dv))


def _delta_plain(i, H, G, D, Dv, eps, state=None):
    """(o before the norm, gated output, state) of the plain statement."""
    T, rep = i["x"].shape[0], H // G
    y = pl.silu(pl.short_convolution(i["x"].double(), i["conv"].double()))
    q = (pl.unit_length(y[:, :G * D].reshape(T, G, D)) * D ** -0.5).repeat_interleave(rep, 1)
    k = pl.unit_length(y[:, G * D:2 * G * D].reshape(T, G, D)).repeat_interleave(rep, 1)
    v = y[:, 2 * G * D:].reshape(T, H, Dv)
    g = pl.channel_decay((i["low_a"].double() @ i["a2"].double().T).reshape(T, H, D), i["a_log"].double(),
                         i["dt_bias"].double().reshape(H, D))
    o, S = pl.delta_rule(q, k, v, torch.sigmoid(i["b"].double()), g, state)
    gate = torch.sigmoid(i["low_g"].double() @ i["g2"].double().T).reshape(T, H, Dv)
    return o, pl.unit_rms(o, eps) * i["norm"].double() * gate, S


def case_delta_rule(dtype, ops, device, *, H=4, G=2, D=12, Dv=20, taps=4, ra=6, rg=10, lens=(37, 1, 2, 80), decay=-3.0,
                    page=None):
    """The delta rule's kernels alone: sequences of unequal lengths in one step with slots out of order, then a second
    and a third step that carry on (one of them a single token each, through the kernel that does everything), against
    the plain recurrence over each whole sequence.  With weak decays a token written at the start still shows at the
    end; the state after the last step is compared too."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(41)
    eps = 1e-5
    per_seq = []
    weights = None
    for n in lens:
        i = _delta_inputs(gen, n + 4, H, G, D, Dv, taps, ra, rg, decay)
        for key in ("x", "low_a", "low_g", "b", "a2", "g2"):
            i[key] = i[key].to(torch.bfloat16).float()
        weights = weights or {k: i[k] for k in ("a2", "g2", "conv", "a_log", "dt_bias", "norm")}
        i.update(weights)
        per_seq.append(i)
    C = 2 * G * D + H * Dv
    slots = [len(lens) + 2 - s for s in range(len(lens))]
    state = torch.zeros((len(lens) + 3, H, D, Dv), dtype=torch.float32, device=device)
    ring = torch.full((len(lens) + 3, taps, C), float("nan"), dtype=torch.float32, device=device) if taps > 1 else None
    dev = lambda x, d=None: x.to(device=device, dtype=d or torch.float32).contiguous()  # noqa: E731
    shared = dict(heads=H, kv_heads=G, dim=D, value_dim=Dv, conv_weight=dev(weights["conv"].t()), ring=ring,
                  dt_bias=dev(weights["dt_bias"]), neg_a=dev(-torch.exp(weights["a_log"])), state=state,
                  q_scale=D ** -0.5)
    a2, g2 = dev(weights["a2"], dt), dev(weights["g2"], dt)
    got = [[] for _ in lens]
    done = [0] * len(lens)
    pad = lambda n: -(-n // 8) * 8  # noqa: E731
    starts = [0, pad(C), pad(C) + pad(ra), pad(C) + pad(ra) + pad(rg)]
    gated = [[] for _ in lens]
    for portion in (lens, [1] * len(lens), [3] * len(lens)):
        wide = torch.zeros((sum(portion), starts[3] + pad(H)), dtype=dt, device=device)
        positions, seqs, at = [], [], 0
        for s, n in enumerate(portion):
            i = per_seq[s]
            for key, c0 in (("x", starts[0]), ("low_a", starts[1]), ("low_g", starts[2]), ("b", starts[3])):
                rows = i[key][done[s]:done[s] + n]
                wide[at:at + n, c0:c0 + rows.shape[1]] = rows.to(dt).to(device)
            positions += list(range(done[s], done[s] + n))
            seqs += [s] * n
            at += n
        step = _step(positions, seqs, [[0]] * len(lens), device, slots=slots)
        x, la = wide[:, :C], wide[:, starts[1]:starts[1] + ra]
        lg, b = wide[:, starts[2]:starts[2] + rg], wide[:, starts[3]:starts[3] + H]
        meta = dict(positions=step.positions, cu_seqlens=step.cu_seqlens, state_slots=step.state_slots,
                    num_seqs=len(lens))
        if all(n == 1 for n in portion) and ops.delta_step_ok(D, Dv):
            out = torch.zeros((len(positions), H * Dv), dtype=dt, device=device)
            ops.delta_step(x, la, lg, b, out, a2=a2, g2=g2, norm_weight=dev(weights["norm"]), eps=eps, **shared, **meta)
            res = out.float().cpu().reshape(-1, H, Dv)
            for s in range(len(lens)):
                gated[s].append((done[s], res[s]))
        else:
            z = (la.float() @ a2.float().t()).contiguous()
            res = ops.delta_rule(x, z, b, token_seq=step.token_seq, **shared, **meta).cpu()
            at = 0
            for s, n in enumerate(portion):
                got[s] += [(done[s] + j, res[at + j]) for j in range(n)]
                at += n
        done = [d + n for d, n in zip(done, portion)]
    for s, n in enumerate(lens):
        o, y, S = _delta_plain(per_seq[s], H, G, D, Dv, eps)
        # (bfloat16: v is kept in 16 bits between the kernels)
        tol = (2e-5 if dtype == "float32" else 8e-3) * max(1.0, float(o.abs().max()))
        for p, row in got[s]:
            diff = float((row - o[p].float()).abs().max())
            assert diff <= tol, f"sequence {s} of {n + 4} tokens, position {p}: off by {diff:.3g} (allowed {tol:.3g})"
        for p, row in gated[s]:
            diff = float((row - y[p].float()).abs().max())
            gtol = (1e-4 if dtype == "float32" else 4e-2) * max(1.0, float(y.abs().max()))
            assert diff <= gtol, f"sequence {s}, single token at {p}: off by {diff:.3g} (allowed {gtol:.3g})"
        sdiff = float((state[slots[s]].cpu() - S.float()).abs().max())
        stol = (3e-5 if dtype == "float32" else 8e-3) * max(1.0, float(S.abs().max()))
        assert sdiff <= stol, f"state of sequence {s} off by {sdiff:.3g} (allowed {stol:.3g})"
    if decay <= -3.0 and max(lens) > 30:  # the first token's write shows at the end of a long sequence
        s = max(range(len(lens)), key=lambda j: lens[j])
        other = dict(per_seq[s], x=per_seq[s]["x"].clone())
        other["x"][0] += 3.0
        o, _, _ = _delta_plain(per_seq[s], H, G, D, Dv, eps)
        o2, _, _ = _delta_plain(other, H, G, D, Dv, eps)
        assert float((o2[-1] - o[-1]).abs().max()) > 20 * 2e-5 * max(1.0, float(o.abs().max()))


def case_sum_norm(dtype, ops, device):
    """The kernel that folds several outputs: none, one or three of them, with and without norms, dense rows and
    partial-sum planes, with and without the average over the depth, on all rows and on a few; widths with and without
    16-byte rows."""
    dt = TORCH[dtype]
    gen = torch.Generator().manual_seed(43)
    tol = 3e-5 if dtype == "float32" else 0.08
    for W in (60, 64, 200, 1032):
        T, n = 9, 5
        y = [(torch.randn((T, W), generator=gen) * s).to(dt) for s in (0.2, 3.0, 1.0)]
        planes = torch.randn((3, T, W), generator=gen)
        ws = [1 + 0.2 * torch.randn(W, generator=gen) for _ in range(3)]
        wf = 1 + 0.2 * torch.randn(W, generator=gen)
        points = torch.randn((n + 1, T, W), generator=gen)
        depth = torch.randn(n + 1, generator=gen)
        eps = 1e-5
        for items in ([], [(y[0], None, 0.0)], [(y[0], ws[0], 1e-4), (planes, ws[1], 1e-6), (y[2], None, 0.0)],
                      [(planes, None, 0.0), (y[1], ws[2], 1e-2)]):
            for use_depth in (False, True):
                resid = points[0].clone() if use_depth else torch.randn((T, W), generator=gen) * 2
                v = resid.double()
                for value, w, e in items:
                    x = value.double().sum(0) if value.dim() == 3 else value.double()
                    v = v + (pl.unit_rms(x, e) * w.double() if w is not None else x)
                s = pl.depth_average([points[j].double() for j in range(n)] + [v], depth.double()) if use_depth else v
                dev_items = [(a.to(device), w.to(device) if w is not None else None, e) for a, w, e in items]
                for rows in (None, [7, 0, 3]):
                    pd = points.clone().to(device)
                    rd = pd[0] if use_depth else resid.clone().to(device)
                    target = None if rows else (torch.empty_like(rd) if use_depth else rd)
                    m = T if rows is None else len(rows)
                    out = torch.empty((m, W), dtype=dt, device=device)
                    ops.sum_norm(out, wf.to(device), eps, resid=rd, items=dev_items, resid_out=target,
                                 points=pd if use_depth else None, num_points=n if use_depth else 0,
                                 depth_weights=depth.to(device) if use_depth else None,
                                 rows=torch.tensor(rows, dtype=torch.int32, device=device) if rows else None, num_rows=m)
                    want = pl.unit_rms(s, eps) * wf.double()
                    want = want[rows] if rows else want
                    assert float((out.float().cpu().double() - want).abs().max()) <= tol, (W, len(items), use_depth, rows)
                    if rows:
                        assert torch.equal(pd.cpu(), points)
                        continue
                    assert float((target.cpu().double() - s).abs().max()) <= 3e-5 * max(1.0, float(s.abs().max()))
                    if use_depth:  # the new point is what was folded; the earlier ones are as they were
                        assert float((pd[n].cpu().double() - v).abs().max()) <= 3e-5
                        assert torch.equal(pd[:n].cpu(), points[:n])
    table = torch.randn((40, 72), generator=gen).to(dt)
    ids = torch.tensor([3, 39, 0, 3, 17], dtype=torch.int32)
    for width in (72, 60):
        t = table[:, :width].contiguous()
        w = 1 + 0.3 * torch.randn(width, generator=gen)
        out = torch.empty((5, width), dtype=torch.float32, device=device)
        ops.embed_norm(ids.to(device), t.to(device), w.to(device), 1e-2, out)
        want = pl.unit_rms(t.double()[ids.long()], 1e-2) * w.double()
        assert float((out.cpu().double() - want).abs().max()) <= 3e-5


def case_frequencies():
    """The position part's frequencies: the plain schedule and every frequency divided by a factor."""
    ctx = BuildContext(torch.float32, torch.device("cpu"), None)
    for dims, base, factor in ((24, 1e4, 4.0), (96, 5e4, 2.5), (8, 50.0, None)):
        spec = PartSpec("rotary_scaled", dict(rotary_dim=dims, theta=base, pairing="half",
                                              scaling=dict(factor=factor, kind="linear") if factor else None))
        part = build_part("position", spec, ctx)
        want = pl.frequencies(dims, base, torch.float64, factor or 1.0)
        assert torch.allclose(torch.tensor(part.host_frequencies(), dtype=torch.float64), want, rtol=1e-12)
        assert part.magnitude == 1.0


def case_pages_for_readers():
    """Keys that several layers read under chunks of their own: a page goes back when none of them needs it any more;
    with a reader that sees everything nothing goes back; layouts that differ are refused."""
    import pytest

    from qwen3_runtime_b200.cache.layout import CacheLayout, KVLayerSpec, StateLayerSpec, kept_for_readers
    from qwen3_runtime_b200.cache.manager import FREED, CacheManager

    own = KVLayerSpec(2, 16, value_dim=24, chunk=20)
    spec = kept_for_readers(0, own, [KVLayerSpec(2, 16, value_dim=24, chunk=7), KVLayerSpec(2, 16, value_dim=24, chunk=33)])
    assert spec.chunk == (7, 20, 33) and kept_for_readers(0, own, [own, own]) == own
    assert kept_for_readers(0, own, [KVLayerSpec(2, 16, value_dim=24)]).chunk is None
    w = kept_for_readers(0, KVLayerSpec(2, 16, 8), [KVLayerSpec(2, 16, 12, keep_first=3)])
    assert (w.window, w.keep_first) == (12, 3)
    for bad in (KVLayerSpec(1, 16, value_dim=24, chunk=20), KVLayerSpec(2, 16, value_dim=16, chunk=20), StateLayerSpec((2,))):
        with pytest.raises(ValueError, match="layout differs"):
            kept_for_readers(0, own, [bad])
    layout = CacheLayout({0: spec})
    assert layout.group_specs[0].kind == "chunk" and layout.group_specs[0].reach == 33
    cm = CacheManager(layout.group_specs, 8, 16, 2)
    rc = cm.open("a")
    for n in (19, 1, 1, 12, 7, 26, 1):
        cm.reserve(rc, n)
        cm.commit(rc, n)
        cm.check_invariants()
        first = min(rc.num_computed // c * c for c in (7, 20, 33))
        for idx, page in enumerate(rc.tables[0]):
            assert (page == FREED) == ((idx + 1) * 8 <= first), (rc.num_computed, idx)
    cm.close(rc)
    assert cm.num_free_pages == cm.num_pages
