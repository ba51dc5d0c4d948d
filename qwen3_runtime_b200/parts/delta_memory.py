"""A matrix memory per (request, head) that is written by the delta rule, with a decay per key channel.

    q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))     causal, a few taps, per channel
    q, k: unit vectors per head (1e-6 inside the root); q times dim^(-1/2)
    g_t = exp(-exp(A_log_head) * softplus(W_a2 (W_a1 h) + dt_bias))        per head and key channel
    S <- diag(g_t) S;  u = sigmoid(W_b h) * (v - S^T k);  S <- S + k u^T;  o = S^T q
    out = W_o (o / sqrt(mean(o^2) + eps) * w * sigmoid(W_g2 (W_g1 h)))      norm per head, w shared by the heads

q and k have ``kv_heads`` heads, v and the state ``num_heads``: head h reads q/k head h / (num_heads / kv_heads).
The state and the convolution's past inputs live in two state slots of float32 per request (the inputs as a ring of
``taps`` rows).  Decays, steps, unit vectors, the recurrence and the norm are float32 whatever the compute dtype.
A step in which every request brings one token runs everything between the two projections as one kernel.
The part is a :class:`BranchMixer`: it runs alone or as a branch of the ``parallel`` mixer.
"""

from __future__ import annotations

import torch

from ..cache.layout import StateLayerSpec
from .base import BuildContext, ParamSpec, StepContext, register_part
from .linear_state import BranchMixer, _pad_rows


class GatedDelta(BranchMixer):
    def __init__(self, spec, ctx: BuildContext):
        super().__init__(spec, ctx)
        self.hidden_size = int(spec["hidden_size"])
        self.num_heads = int(spec["num_heads"])
        self.num_kv_heads = int(spec["num_kv_heads"])
        self.dim = int(spec["dim"])
        self.vdim = int(spec["vdim"])
        self.taps = int(spec["taps"])
        self.decay_rank = int(spec["decay_rank"])
        self.gate_rank = int(spec["gate_rank"])
        self.eps = float(spec["eps"])
        if self.num_heads % self.num_kv_heads:
            raise ValueError("gated_delta: num_heads must be a multiple of num_kv_heads")
        if self.dim > 256:
            raise ValueError(f"dim={self.dim} is not supported: the state kernel keeps up to 256 key rows per head")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"taps={self.taps}: the convolution takes 1 to 16")
        if self.decay_rank < 1 or self.gate_rank < 1:
            raise ValueError("gated_delta: the ranks are the row counts of the stored a1 and g1")
        self.channels = 2 * self.num_kv_heads * self.dim + self.num_heads * self.vdim
        self.in_weight = self.o_weight = self.a2 = self.g2 = None
        self.conv_weight = self.dt_bias = self.neg_a = self.norm_weight = None
        self.starts: list[int] = []

    def param_specs(self):
        H, G, D, Dv, W = self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.hidden_size
        specs = {}
        for name, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
            specs[name] = ParamSpec((rows, W))
            specs[name + ".conv"] = ParamSpec((rows, self.taps), "matrix_f32")
        specs.update({"b": ParamSpec((H, W)), "A_log": ParamSpec((H,), "vector"), "norm": ParamSpec((Dv,), "vector"),
                      "a1": ParamSpec((self.decay_rank, W)), "a2": ParamSpec((H * D, self.decay_rank)),
                      "dt_bias": ParamSpec((H * D,), "vector"), "g1": ParamSpec((self.gate_rank, W)),
                      "g2": ParamSpec((H * Dv, self.gate_rank)), "o": ParamSpec((W, H * Dv))})
        return specs

    def load(self, tensors):
        qkv = torch.cat([tensors["q"], tensors["k"], tensors["v"]], dim=0)  # one run of channels for the convolution
        self.in_weight, self.starts = _pad_rows([qkv, tensors["a1"], tensors["g1"], tensors["b"]])
        self.o_weight = tensors["o"].contiguous()
        self.a2, self.g2 = tensors["a2"].contiguous(), tensors["g2"].contiguous()
        # tap-major [taps, channels]: neighbouring channels read neighbouring weights
        self.conv_weight = torch.cat([tensors[n + ".conv"] for n in ("q", "k", "v")], dim=0).t().contiguous()
        self.dt_bias = tensors["dt_bias"].contiguous()
        self.neg_a = -torch.exp(tensors["A_log"].float())
        self.norm_weight = tensors["norm"].contiguous()

    def input_weight(self):
        return self.in_weight

    def release_input_weight(self):
        self.in_weight = None

    def context_size(self):
        return self.num_heads * self.vdim

    def output_weight(self):
        return self.o_weight

    def kernel_groups(self):
        groups = ["delta_state", "linear_state"]
        groups += ["gemm_f32"] if self.ctx.dtype == torch.float32 else ["gemm_small_m", "gemm_stream"]
        return groups

    def cache_spec(self):
        ring = StateLayerSpec((self.taps, self.channels)) if self.taps > 1 else None
        return (StateLayerSpec((self.num_heads, self.dim, self.vdim)), ring)

    def context(self, proj, step: StepContext, cache, out, out_scale):
        ops = self.ops
        memory, ring = cache
        H, G, D, Dv = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        s = self.starts
        x = proj[:, : self.channels]
        low_a, low_g = proj[:, s[1]:s[1] + self.decay_rank], proj[:, s[2]:s[2] + self.gate_rank]
        b = proj[:, s[3]:s[3] + H]
        shared = dict(heads=H, kv_heads=G, dim=D, value_dim=Dv, conv_weight=self.conv_weight,
                      ring=ring.state if ring is not None else None, dt_bias=self.dt_bias, neg_a=self.neg_a,
                      state=memory.state, positions=step.positions, cu_seqlens=step.cu_seqlens,
                      state_slots=step.state_slots, num_seqs=step.num_seqs, q_scale=D ** -0.5)
        if step.decode_only and out_scale == 1.0 and ops.delta_step_ok(D, Dv):
            ops.delta_step(x, low_a, low_g, b, out, a2=self.a2, g2=self.g2, norm_weight=self.norm_weight, eps=self.eps,
                           **shared)
            return
        z = ops.linear(low_a, self.a2, out_dtype=torch.float32)
        gate = ops.linear(low_g, self.g2)
        o = ops.delta_rule(x, z, b, token_seq=step.token_seq, **shared)
        ops.head_norm_gate(o, gate.unflatten(1, (H, Dv)), out.unflatten(1, (H, Dv)), weight=self.norm_weight,
                           eps=self.eps, out_scale=out_scale, gate_act="sigmoid")


register_part("mixer", "gated_delta", GatedDelta)
