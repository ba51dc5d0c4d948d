"""Timopel stated plainly: whole sequences, no cache, one function per mechanism, float64 or float32.

Nothing here is shared with the package.  A model is ``(config, tensors)``: ``config`` the dictionary of a
config.json, ``tensors`` name -> tensor.  Notation: ``x`` is the stream ``[T, W]``, N a root-mean-square norm; a layer
computes ``x += m N_1b(mixer(N_1(x)))`` and ``x += m N_2b(ff(N_2(x)))``.
"""

from __future__ import annotations

import math

import torch

ACTIVATIONS = None  # a dtype: products' results and sublayer inputs are rounded to it (a model of 16-bit activations)


def _r(x):
    return x if ACTIVATIONS is None else x.to(ACTIVATIONS).to(x.dtype)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def query_temperature(T, coef, every, dtype):
    """``[T]``: 1 + coef ln(n + 1), n the number of whole runs of ``every`` tokens up to and including the token."""
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in range(T)], dtype=dtype)


def mix_values(v, first, lam):
    """A share ``lam`` of each token's value comes from the first mixing layer."""
    return v + lam * (first - v)


def sink_attention_core(q, k, v, scale, sink):
    """q ``[T, H, D]``, k ``[T, G, D]``, v ``[T, G, Dv]`` -> ``[T, H, Dv]``: causal softmax over the earlier keys, with
    one more term exp(sink_h) in each denominator that stands for no key."""
    T, H = q.shape[0], q.shape[1]
    per = H // k.shape[1]
    earlier = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    heads = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        s = torch.where(earlier, s, torch.full_like(s, float("-inf")))
        m = torch.maximum(s.max(-1, keepdim=True).values, sink[h])
        e = torch.exp(s - m)
        heads.append((e / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - m))) @ v[:, h // per])
    return torch.stack(heads, 1)


def attention(h, t, p, m, eps, first_values):
    """``(output, values)``: ``values`` are this layer's own, before any mixing."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(_r(h @ t[p + "q"].T).view(T, H, D), t[p + "q.norm"], eps)
    k = rms_norm(_r(h @ t[p + "k"].T).view(T, G, D), t[p + "k.norm"], eps)
    own = v = _r(h @ t[p + "v"].T).view(T, G, Dv)
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"], q.dtype)[:, None, None]
    if m.get("v_mix") and first_values is not None:
        v = mix_values(v, first_values, t[p + "vmix"])
    o = _r(sink_attention_core(_r(q), _r(k), _r(v), m["scale"], t[p + "sink"]))
    return o.reshape(T, H * Dv) @ t[p + "o"].T, own


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_feed_forward(h, t, p):
    return _r(gelu(_r(h @ t[p + "gate"].T)) * _r(h @ t[p + "up"].T)) @ t[p + "down"].T


def clamped_expert(h, t, p, limit):
    g = torch.minimum(_r(h @ t[p + ".gate"].T), torch.tensor(limit, dtype=h.dtype))
    u = _r(h @ t[p + ".up"].T).clamp(-limit, limit)
    return _r(g * torch.sigmoid(1.702 * g) * (u + 1)) @ t[p + ".down"].T


def route(z, top, scale):
    """``[T, E]`` weights: the softmax over all outputs at the ``top`` largest ones, made to sum to ``scale``."""
    s = torch.softmax(z, -1)
    chosen = torch.zeros_like(s, dtype=torch.bool).scatter_(-1, torch.topk(s, top, dim=-1).indices, True)
    w = torch.where(chosen, s, torch.zeros_like(s))
    return w / (w.sum(-1, keepdim=True) + 1e-20) * scale


def expert_feed_forward(h, t, p, f):
    r = f["router"]
    w = route(h @ t[p + "router"].T, r["top"], r.get("scale", 1.0))
    out = torch.zeros(h.shape[0], t[p + "e0.down"].shape[0], dtype=h.dtype)
    for e in range(r["experts"]):
        rows = torch.nonzero(w[:, e]).flatten()
        if rows.numel():
            out[rows] += w[rows, e, None] * _r(clamped_expert(h[rows], t, f"{p}e{e}", f["expert"]["limit"]))
    if f.get("shared"):
        out = out + _r(clamped_expert(h, t, p + "shared", f["shared"]["limit"]))
    return out


def feed_forward(h, t, p, f):
    return dense_feed_forward(h, t, p) if f["kind"] == "dense" else expert_feed_forward(h, t, p, f)


def forward(config, tensors, tokens, dtype=torch.float64, with_streams=False, activations=None):
    """Logits ``[T, vocab]`` of one sequence (and the stream after every layer).  ``activations``: a narrower type
    that sublayer inputs, products' results and sublayer outputs are rounded to, the stream, norms, routing, scores and
    softmax staying in ``dtype``."""
    global ACTIVATIONS
    ACTIVATIONS = activations
    try:
        return _forward(config, tensors, tokens, dtype, with_streams)
    finally:
        ACTIVATIONS = None


def _forward(config, tensors, tokens, dtype, with_streams):
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps, mult = config["norm"]["eps"], config.get("residual_mult", 1.0)
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    first_values, streams = None, []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y, own = attention(_r(rms_norm(x, t[p + "norm1"], eps)), t, p + "mix.", layer["mixer"], eps, first_values)
        if layer["mixer"].get("v_mix") and first_values is None:
            first_values = own
        x = x + mult * rms_norm(_r(y), t[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(_r(rms_norm(x, t[p + "norm2"], eps)), t, p + "mlp.", layer["mlp"])
            x = x + mult * rms_norm(_r(y), t[p + "norm2b"], eps)
        streams.append(x)
    logits = _r(rms_norm(x, t["final.norm"], eps)) @ t["embed"].T
    return (logits, torch.stack(streams)) if with_streams else logits
