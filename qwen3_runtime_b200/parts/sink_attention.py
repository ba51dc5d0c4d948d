"""Softmax attention with grouped key/value heads, a window that keeps the sequence's first tokens, a
sink in the softmax and a gate on the heads' outputs.

    q, k, v, g = W_q h, W_k h, W_v h, W_g h              (one product)
    q, k: every head divided by its root mean square, times a weight shared by the heads (optional)
    score(i, j) = (q_i . k_j) * scale;  i sees j <= i with i - j < window or j < keep_first
    p_j = exp(s_j) / (exp(sink) + sum_j' exp(s_j'))      (``sink`` None: a plain softmax)
    out = W_o (heads' outputs * sigmoid(g))              (``gate`` None: no gate)

Keys and values may have unlike sizes per head.  The cache is a paged key/value layer whose group gives
back the pages that lie wholly between the kept first tokens and the window.  Further options:
``position`` (a rotary position part with inverse frequencies: q and k are turned after their norm, inside
the same kernel; without it positions do not enter the scores); ``softcap`` (scores become softcap *
tanh(score / softcap) after the scale); ``values="keys"`` (there is no W_v: the values are the keys as
projected, before norm and rotation); ``chunk`` (position i sees j <= i of its own chunk only, chunks of
that many tokens counted from the sequence's first token); ``qkv_bias`` (biases ``q.b``, ``k.b``, ``v.b`` in the
projections); ``own_kv=False`` (the layer has no key and value projections and reads the keys and values another
layer has stored, under its own mask); ``value_turn`` (a rotary base: the value of position j is turned by j over
all its dimensions before it is stored, pair m by ``j * base^(-2m / vdim)``, and a head's sum at position i is turned
back by i); ``query_temperature`` ``(coef, every)`` (the normed and turned query of position p is multiplied by
1 + coef * ln(floor((p + 1) / every) + 1)); ``value_mix`` (``"source"``: the layer's values as projected are kept for
the later layers of the step; ``"blend"``: the layer's values become (1 - lambda) v + lambda v_source before they are
stored, lambda being the stored number ``vmix``, which a source has too but does not use).  ``sink`` is one score for
all heads (a number) or ``"learned"`` (one stored number per head, ``sink``).

The part is a :class:`BranchMixer`: it runs alone or as a branch of the ``parallel`` mixer.
"""

from __future__ import annotations

import torch

from ..cache.layout import KVLayerSpec
from ..config.spec import PartSpec
from .base import BuildContext, ParamSpec, StepContext, build_part, register_part
from .linear_state import BranchMixer, _pad_rows


class SinkWindowAttention(BranchMixer):
    def __init__(self, spec, ctx: BuildContext):
        super().__init__(spec, ctx)
        self.hidden_size = int(spec["hidden_size"])
        self.num_heads = int(spec["num_heads"])
        self.num_kv_heads = int(spec["num_kv_heads"])
        self.dim = int(spec["dim"])
        self.vdim = int(spec["vdim"])
        self.scale = float(spec["scale"])
        self.window = spec.get("window") or None
        self.keep_first = int(spec.get("keep_first") or 0) if self.window else 0
        sink = spec.get("sink")  # one score for all heads (a number), "learned" (a stored score per head), or None
        self.learned_sink = sink == "learned"
        self.has_sink = sink is not None
        self.sink = None  # float32 [heads]
        if self.has_sink and not self.learned_sink:
            self.sink = torch.full((self.num_heads,), float(sink), dtype=torch.float32, device=ctx.device)
        self.gate = spec.get("gate")  # "sigmoid" or None
        self.qk_norm_eps = spec.get("qk_norm_eps")
        if self.num_heads % self.num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if self.dim > 256 or self.vdim > 256:
            raise ValueError(f"dim={self.dim}, vdim={self.vdim}: the attention kernels take sizes up to 256")
        if self.gate not in (None, "sigmoid"):
            raise ValueError(f"sink_window_attention: gate is 'sigmoid' or absent, not {self.gate!r}")
        self.softcap = float(spec.get("softcap") or 0.0) or None
        self.chunk = int(spec.get("chunk") or 0) or None
        self.values_are_keys = spec.get("values", "own") == "keys"
        if spec.get("values", "own") not in ("own", "keys"):
            raise ValueError(f"sink_window_attention: values are 'own' or 'keys', not {spec.get('values')!r}")
        if self.values_are_keys and self.vdim != self.dim:
            raise ValueError("sink_window_attention: values that are the keys have the keys' size")
        if self.chunk and self.window:
            raise ValueError("sink_window_attention: a window or chunks, not both")
        self.position = build_part("position", spec.get("position") or PartSpec("none"), ctx)
        if self.position.style == "rotary":
            if not hasattr(self.position, "inverse_frequencies") or self.position.rotary_dim > self.dim:
                raise ValueError("sink_window_attention turns q and k by angles worked out from inverse "
                                 "frequencies over at most the head's size; the position part offers otherwise")
        elif self.position.style != "none":
            raise ValueError(f"sink_window_attention has no {self.position.style!r} position encoding")
        self.qkv_bias = bool(spec.get("qkv_bias", False))
        self.own_kv = bool(spec.get("own_kv", True))
        self.value_position = None
        if spec.get("value_turn") is not None:
            if self.vdim % 2 or self.values_are_keys:
                raise ValueError("sink_window_attention: turned values have an even size and a projection of their own")
            self.value_position = build_part("position", PartSpec("rotary_scaled", dict(
                rotary_dim=self.vdim, theta=float(spec["value_turn"]),
                pairing=getattr(self.position, "pairing", "half"))), ctx)
        # q and k without norms: biases, rotations and the cache write are one kernel reading the step's turn tables
        self.turned = self.qk_norm_eps is None and not self.values_are_keys
        if not self.turned and (self.qkv_bias or not self.own_kv or self.value_position is not None):
            raise ValueError("sink_window_attention: biases, shared keys and turned values go without q/k norms and with "
                             "values of their own")
        temperature = spec.get("query_temperature")
        self.temperature = (float(temperature[0]), int(temperature[1])) if temperature else None
        self.value_mix = spec.get("value_mix")
        if self.value_mix not in (None, "source", "blend"):
            raise ValueError(f"sink_window_attention: value_mix is 'source', 'blend' or absent, not {self.value_mix!r}")
        if self.turned and (self.temperature or self.value_mix):
            raise ValueError("sink_window_attention: a query temperature and mixed values go with q/k norms")
        if self.values_are_keys and self.value_mix:
            raise ValueError("sink_window_attention: values that are the keys are not mixed")
        self.value_share = 0.0
        self.in_weight = self.o_weight = self.q_norm = self.k_norm = self.bias = None
        self._tables = None
        self.starts: list[int] = []

    def param_specs(self):
        H, G, D, Dv, W = self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.hidden_size
        specs = {"q": ParamSpec((H * D, W)), "k": ParamSpec((G * D, W)), "v": ParamSpec((G * Dv, W)),
                 "o": ParamSpec((W, H * Dv))}
        if self.values_are_keys:
            del specs["v"]
        if not self.own_kv:
            del specs["k"], specs["v"]
        if self.qkv_bias:
            specs.update({n + ".b": ParamSpec((specs[n].shape[0],), "vector") for n in ("q", "k", "v") if n in specs})
        if self.gate:
            specs["g"] = ParamSpec((H * Dv, W))
        if self.qk_norm_eps is not None:
            specs["q.norm"] = ParamSpec((D,), "vector")
            specs["k.norm"] = ParamSpec((D,), "vector")
        if self.value_mix:
            specs["vmix"] = ParamSpec((), "vector")
        if self.learned_sink:
            specs["sink"] = ParamSpec((H,), "vector")
        return specs

    def load(self, tensors):
        if self.values_are_keys:  # no W_v: the value heads are read where the key heads are
            self.in_weight, starts = _pad_rows([tensors["q"], tensors["k"]] + ([tensors["g"]] if self.gate else []))
            self.starts = [starts[0], starts[1], starts[1], *starts[2:]]
        elif not self.own_kv:
            self.in_weight, starts = _pad_rows([tensors["q"]] + ([tensors["g"]] if self.gate else []))
            self.starts = [0, 0, 0, *starts[1:]]
        else:
            blocks = [tensors["q"], tensors["k"], tensors["v"]] + ([tensors["g"]] if self.gate else [])
            self.in_weight, self.starts = _pad_rows(blocks)
        if self.qkv_bias:
            self.bias = torch.zeros(self.in_weight.shape[0], dtype=torch.float32, device=self.in_weight.device)
            for name, at in zip(("q", "k", "v"), self.starts):
                if name + ".b" in tensors:
                    b = tensors[name + ".b"]
                    self.bias[at:at + b.numel()] = b
        self.o_weight = tensors["o"].contiguous()
        self.q_norm = tensors.get("q.norm")
        self.k_norm = tensors.get("k.norm")
        if self.learned_sink:
            self.sink = tensors["sink"].contiguous()
        if self.value_mix == "blend":
            self.value_share = float(tensors["vmix"])

    def input_weight(self):
        return self.in_weight

    def release_input_weight(self):
        self.in_weight = None

    def context_size(self):
        return self.num_heads * self.vdim

    def output_weight(self):
        return self.o_weight

    def kernel_groups(self):
        groups = ["rope_kv", "attention_generic"]
        groups += ["gemm_f32"] if self.ctx.dtype == torch.float32 else ["gemm_small_m", "gemm_stream"]
        if self.ctx.dtype == torch.bfloat16 and not self.window and not self.gate and not self.softcap:
            if self.turned or not self._specialised() or self.dim == 256:
                groups.append("attention_chunk")
            if self.dim == 128 and self.vdim == 128:
                groups.append("attention_prefill_tc")
        if self._specialised():
            groups += ["attention_decode"] + (["attention_prefill"] if self.dim in (64, 128) else [])
        return groups

    def _specialised(self) -> bool:
        """Keys and values of one size that the split-KV decode kernel (64, 128, 256) and the tensor-core prompt
        kernel (64, 128) take (ops.paged_attention sends a dense output there), with the window's kept first tokens, the
        sink, the gate and capped scores."""
        return (self.ctx.dtype == torch.bfloat16 and self.dim == self.vdim and self.dim in (64, 128, 256)
                and self.num_heads // self.num_kv_heads <= 16 and not self.chunk and self.value_position is None)

    # positions for which the decode kernel that also makes the newest token's q and k keeps rotation tables;
    # steps that reach beyond run the q/k kernel (which needs none) and the plain decode kernel
    FUSED_POSITIONS = 32768

    def _fused_tables(self):
        """cos and sin ``[FUSED_POSITIONS, dim / 2]`` for the decode kernel that norms, turns and stores the newest
        token itself: the part's frequencies followed by zeros (pairs that do not turn), times the magnitude.
        None when this rotation cannot be put that way (halves pairing over a part of the head)."""
        if self._tables is None:
            pos = self.position
            inv = pos.inverse_frequencies()
            if pos.pairing == "half" and 2 * inv.numel() != self.dim:
                self._tables = False
            else:
                padded = torch.zeros(self.dim // 2, dtype=torch.float32, device=inv.device)
                padded[: inv.numel()] = inv
                cos, sin = self.ops.rope_table(padded, self.FUSED_POSITIONS)
                magnitude = float(getattr(pos, "magnitude", 1.0))
                if magnitude != 1.0:
                    cos, sin = cos * magnitude, sin * magnitude
                self._tables = (cos, sin)
        return self._tables or None

    def _slices_key(self):
        reach = self.window + self.keep_first if self.window else None  # the most keys a token sees
        return ("decode_slices", self.num_kv_heads, self.dim, reach)

    def step_choosers(self):
        """Into how many slices the split-KV decode kernel cuts the longest sequence's keys."""
        model = getattr(self.ops, "decode_slices_for", None)
        if model is None or not self._specialised():
            return {}
        key = self._slices_key()
        return {key: lambda kv_lens: model(kv_lens, key[1], key[2], key[3])}

    def cache_spec(self):
        return KVLayerSpec(self.num_kv_heads, self.dim, self.window, value_dim=self.vdim, keep_first=self.keep_first,
                           chunk=self.chunk)

    def position_limit(self):
        return self.position.position_limit()

    def _turns(self, position, step: StepContext):
        """The step's turn table for one set of frequencies, made by the first layer that asks for it."""
        inv = position.inverse_frequencies()
        key = ("turns", inv.data_ptr(), inv.numel())
        if key not in step.extras:
            step.extras[key] = self.ops.turn_table(step.positions, inv)
        return step.extras[key]

    def _query_scale(self, step: StepContext):
        """The factors of the step's queries, made by the first layer that asks for these constants."""
        if self.temperature is None:
            return None
        key = ("query_temperature", *self.temperature)
        if key not in step.extras:
            step.extras[key] = self.ops.query_temperature(step.positions, *self.temperature)
        return step.extras[key]

    def _first_values(self, own, step: StepContext):
        """The values this layer's are blended with (None: they stay as they are).  ``own``: its values as projected."""
        if self.value_mix == "source":
            step.extras["first_values"] = own
        return step.extras["first_values"] if self.value_mix == "blend" else None

    def _turned_context(self, proj, step: StepContext, cache, ctx) -> None:
        ops = self.ops
        H, G, D, Dv = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        s = self.starts
        block_table = step.block_tables[cache.paged_index]
        pairing = getattr(self.position, "pairing", "half")
        qk_turns = self._turns(self.position, step) if self.position.style == "rotary" else None
        v_turns = self._turns(self.value_position, step) if self.value_position is not None else None
        gate = proj[:, s[3]:s[3] + H * Dv] if self.gate else None
        ops.turn_store(proj, num_heads=H, num_kv_heads=G, head_dim=D, value_dim=Dv, k_start=s[1], v_start=s[2],
                       bias=self.bias, qk_turns=qk_turns, value_turns=v_turns, positions=step.positions,
                       token_seq=step.token_seq, block_table=block_table, k_pages=cache.k_pages, v_pages=cache.v_pages,
                       page_size=cache.page_size, write_kv=cache.writes, pairing=pairing)
        ops.paged_attention(proj, proj.stride(0), num_heads=H, num_kv_heads=G, head_dim=D, k_pages=cache.k_pages,
                            v_pages=cache.v_pages, block_table=block_table, token_seq=step.token_seq,
                            positions=step.positions, out=ctx, page_size=cache.page_size, scale=self.scale,
                            window=self.window, step=step, value_dim=Dv, keep_first=self.keep_first, sink=self.sink,
                            gate=gate, decode_slices=step.choices.get(self._slices_key()), chunk=self.chunk,
                            softcap=self.softcap, value_turns=v_turns, pairing=pairing)

    def context(self, proj, step: StepContext, cache, out, out_scale):
        if out_scale != 1.0:
            raise NotImplementedError("sink_window_attention: a branch's scale goes into the norm of its output")
        ops = self.ops
        if self.turned:
            return self._turned_context(proj, step, cache, out)
        H, G, D, Dv = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        s = self.starts
        ctx = out
        block_table = step.block_tables[cache.paged_index]
        gate = proj[:, s[3]:s[3] + H * Dv] if self.gate else None
        fusable = getattr(ops, "decode_new_token_ok", None)
        rotary = self.position.style == "rotary"
        blend = {}
        if self.temperature or self.value_mix:
            blend = dict(q_scale=self._query_scale(step), value_share=self.value_share,
                         first_values=self._first_values(proj[:, s[2]:s[2] + G * Dv], step))
        tables = None
        if (fusable is not None and step.decode_only and cache.writes and self._specialised() and rotary
                and (step.captured_width * cache.page_size or step.max_kv_len) <= self.FUSED_POSITIONS):
            tables = self._fused_tables()
        cos, sin = tables if tables is not None else (None, None)
        if (fusable is not None and step.decode_only and cache.writes and self._specialised()
                and (not rotary or tables is not None)
                # q, k and v heads side by side, as that kernel reads them (v where k is, if the values are the keys)
                and s[1] == H * D and s[2] == (H * D if self.values_are_keys else (H + G) * D)
                and fusable(proj, num_heads=H, num_kv_heads=G, head_dim=D, cos=cos, q_weight=self.q_norm,
                            k_weight=self.k_norm)):
            # one kernel: norm (and rotation) of the newest q and k, cache write, split-KV attention with sink, gate
            # and capped scores
            width = step.captured_width
            ops.paged_attention_decode(
                proj, proj.stride(0), num_heads=H, num_kv_heads=G, head_dim=D, k_pages=cache.k_pages,
                v_pages=cache.v_pages, block_table=block_table, kv_lens=step.kv_lens, cu_seqlens=step.cu_seqlens,
                out=ctx, page_size=cache.page_size, scale=self.scale, window=self.window, num_seqs=step.num_seqs,
                max_kv_len=width * cache.page_size or step.max_kv_len,
                new_token=dict(q_weight=self.q_norm, k_weight=self.k_norm,
                               eps=self.qk_norm_eps if self.qk_norm_eps is not None else 0.0, cos=cos, sin=sin,
                               pairing=getattr(self.position, "pairing", "half"),
                               values_are_keys=self.values_are_keys, **blend),
                num_splits=step.choices.get(self._slices_key()), longest=step.kv_longest, step=step,
                keep_first=self.keep_first, sink=self.sink, gate=gate, softcap=self.softcap)
            return
        ops.qk_norm_store(proj, num_heads=H, num_kv_heads=G, head_dim=D, value_dim=Dv, k_start=s[1], v_start=s[2],
                          q_weight=self.q_norm, k_weight=self.k_norm,
                          eps=self.qk_norm_eps if self.qk_norm_eps is not None else 0.0, positions=step.positions,
                          token_seq=step.token_seq, block_table=block_table, k_pages=cache.k_pages,
                          v_pages=cache.v_pages, page_size=cache.page_size, write_kv=cache.writes,
                          **(dict(inv_freq=self.position.inverse_frequencies(), pairing=self.position.pairing,
                                  magnitude=getattr(self.position, "magnitude", 1.0)) if rotary else {}), **blend)
        ops.paged_attention(proj, proj.stride(0), num_heads=H, num_kv_heads=G, head_dim=D, k_pages=cache.k_pages,
                            v_pages=cache.v_pages, block_table=block_table, token_seq=step.token_seq,
                            positions=step.positions, out=ctx, page_size=cache.page_size, scale=self.scale,
                            window=self.window, step=step, value_dim=Dv, keep_first=self.keep_first, sink=self.sink,
                            gate=gate, decode_slices=step.choices.get(self._slices_key()),
                            **(dict(chunk=self.chunk, softcap=self.softcap) if self.chunk or self.softcap else {}))


register_part("mixer", "sink_window_attention", SinkWindowAttention)
