"""Pevazen stated plainly: whole sequences, no cache, one function per mechanism, float64 or float32.

Nothing here is shared with the package.  A model is ``(config, tensors)``: ``config`` the dictionary of a
config.json, ``tensors`` name -> tensor.  Notation: ``X_0`` is the normed embedding, ``s_0 = X_0``; layer i
reads ``h = unit(s_i) * g_i`` and makes ``X_(i+1) = s_i + mixer(h) + ff(h)``; what layer i + 1 reads is
``s_(i+1) = sum_j w_i[j] X_j`` over ``j = 0 .. i + 1``.
"""

from __future__ import annotations

import torch

ACTIVATIONS = None  # a dtype: products' results and sublayer inputs are rounded to it (a model of 16-bit activations)


def _r(x):
    return x if ACTIVATIONS is None else x.to(ACTIVATIONS).to(x.dtype)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_length(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def depth_average(points, weights):
    """``points``: X_0 .. X_(i+1); ``weights``: one number each."""
    total = torch.zeros_like(points[0])
    for x, w in zip(points, weights):
        total = total + w * x
    return total


def frequencies(dims, base, dtype, factor=1.0):
    return torch.tensor([base ** (-2.0 * m / dims) / factor for m in range(dims // 2)], dtype=dtype)


def rotate(x, positions, freqs, direction=1.0):
    """x ``[T, heads, D]``: elements m and m + n of each head, n = len(freqs), turn by direction * position * f_m."""
    n = freqs.numel()
    ang = direction * positions.to(freqs.dtype)[:, None] * freqs[None, :]
    cos, sin = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * n:]], dim=-1)


def visible(T, chunk):
    i = torch.arange(T)
    seen = i[None, :] <= i[:, None]
    if chunk:
        seen = seen & ((i[None, :] // chunk) == (i[:, None] // chunk))
    return seen


def attention_core(q, k, v, scale, chunk):
    """q ``[T, H, D]``, k ``[T, G, D]``, v ``[T, G, Dv]`` -> ``[T, H, Dv]``: softmax over the visible keys."""
    T, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    seen = visible(T, chunk)
    outs = []
    for head in range(H):
        s = (q[:, head] @ k[:, head // rep].T) * scale
        w = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)
        outs.append(w @ v[:, head // rep])
    return torch.stack(outs, 1)


def turned_values_core(q, k, v, scale, chunk, base):
    """The same with every value turned by its own position before the sum and the sum turned back by the
    query's: what comes out depends on how far back a value lies."""
    T, Dv = v.shape[0], v.shape[2]
    pos = torch.arange(T)
    f = frequencies(Dv, base, v.dtype)
    return rotate(attention_core(q, k, _r(rotate(v, pos, f)), scale, chunk), pos, f, direction=-1.0)


def _qk_freqs(rot, dtype):
    if rot is None:
        return torch.zeros(0, dtype=dtype)
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    return frequencies(rot["dims"], rot["base"], dtype, factor)


def _chunk(m):
    return (m.get("mask") or {}).get("size")


def biased_attention(h, t, p, m, kept):
    """Grouped attention with biases on q, k and v; ``kept``: (keys, values) of the layer this one reads, or
    None.  Returns the output and the keys and values used."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    freqs = _qk_freqs(m.get("rot"), h.dtype)
    q = _r(rotate(_r(h @ t[p + "q"].T + t[p + "q.b"]).view(T, H, D), pos, freqs))
    if kept is None:
        k = _r(rotate(_r(h @ t[p + "k"].T + t[p + "k.b"]).view(T, G, D), pos, freqs))
        v = _r(h @ t[p + "v"].T + t[p + "v.b"]).view(T, G, Dv)
    else:
        k, v = kept
    o = _r(attention_core(q, k, v, m["scale"], _chunk(m)))
    return o.reshape(T, H * Dv) @ t[p + "o"].T, (k, v)


def turned_value_attention(h, t, p, m):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    freqs = _qk_freqs(m["rot"], h.dtype)
    q = _r(rotate(_r(h @ t[p + "q"].T).view(T, H, D), pos, freqs))
    k = _r(rotate(_r(h @ t[p + "k"].T).view(T, G, D), pos, freqs))
    v = _r(h @ t[p + "v"].T).view(T, G, Dv)
    o = _r(turned_values_core(q, k, v, m["scale"], _chunk(m), m["rot"]["base"]))
    return o.reshape(T, H * Dv) @ t[p + "o"].T


def silu(x):
    return x * torch.sigmoid(x)


def short_convolution(x, w):
    """x ``[T, C]``, w ``[C, taps]``: the last column weighs the token itself."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def channel_decay(z, a_log, dt_bias):
    """z ``[T, H, D]``: exp(-exp(a_log_h) * softplus(z + dt_bias))."""
    x = z + dt_bias
    soft = torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))
    return torch.exp(-torch.exp(a_log)[None, :, None] * soft)


def delta_rule(q, k, v, beta, decay, state=None):
    """q, k, decay ``[T, H, D]``, v ``[T, H, Dv]``, beta ``[T, H]`` -> (``[T, H, Dv]``, the state after)."""
    T, H, D = q.shape
    S = torch.zeros((H, D, v.shape[2]), dtype=q.dtype) if state is None else state.clone()
    outs = []
    for i in range(T):
        S = S * decay[i][:, :, None]
        guess = torch.einsum("hdv,hd->hv", S, k[i])
        u = beta[i][:, None] * (v[i] - guess)
        S = S + k[i][:, :, None] * u[:, None, :]
        outs.append(torch.einsum("hdv,hd->hv", S, q[i]))
    return torch.stack(outs), S


def delta_memory(h, t, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rep = H // G
    q, k, v = (_r(silu(short_convolution(_r(h @ t[p + n].T), t[p + n + ".conv"]))) for n in ("q", "k", "v"))
    q = (unit_length(q.view(T, G, D)) * D ** -0.5).repeat_interleave(rep, dim=1)
    k = unit_length(k.view(T, G, D)).repeat_interleave(rep, dim=1)
    beta = torch.sigmoid(_r(h @ t[p + "b"].T))
    z = _r(_r(h @ t[p + "a1"].T) @ t[p + "a2"].T).view(T, H, D)
    decay = channel_decay(z, t[p + "A_log"], t[p + "dt_bias"].view(H, D))
    o, _ = delta_rule(q, k, v.view(T, H, Dv), beta, decay)
    gate = torch.sigmoid(_r(_r(h @ t[p + "g1"].T) @ t[p + "g2"].T)).view(T, H, Dv)
    o = _r(unit_rms(o, eps) * t[p + "norm"] * gate)
    return o.reshape(T, H * Dv) @ t[p + "o"].T


def side_by_side(h, t, p, m, eps):
    left = _r(turned_value_attention(h, t, p + "left.", m["left"]))
    right = _r(delta_memory(h, t, p + "right.", m["right"], eps))
    return 0.5 * (unit_rms(left, eps) * t[p + "left.out"] + unit_rms(right, eps) * t[p + "right.out"])


def dense_feed_forward(h, t, p):
    return _r(_r(silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T)


def forward(config, tensors, tokens, dtype=torch.float64, with_streams=False, activations=None):
    """Logits ``[T, vocab]`` of one sequence (and the averaged stream after every layer).  ``activations``: a
    narrower type that sublayer inputs, products' results and sublayer outputs are rounded to, the stream, norms,
    scores, softmax and the recurrence staying in ``dtype``."""
    global ACTIVATIONS
    ACTIVATIONS = activations
    try:
        return _forward(config, tensors, tokens, dtype, with_streams)
    finally:
        ACTIVATIONS = None


def _forward(config, tensors, tokens, dtype, with_streams):
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = unit_rms(t["embed"][torch.as_tensor(tokens, dtype=torch.long)], eps) * t["embed.norm"]
    points, streams, kept = [x], [], {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = _r(unit_rms(x, eps) * t[p + "norm1"])
        if layer["type"] == "parallel":
            y = side_by_side(h, t, p + "mix.", m, eps)
        else:
            source = m.get("kv_from")
            y, kept[i] = biased_attention(h, t, p + "mix.", m, None if source is None else kept[source])
            y = _r(y)
        if layer.get("mlp") is not None:
            y = y + dense_feed_forward(h, t, p + "mlp.")
        points.append(x + y)
        x = depth_average(points, t[p + "dwa"])
        streams.append(x)
    logits = _r(unit_rms(x, eps) * t["final.norm"]) @ t["head"].T
    return (logits, torch.stack(streams)) if with_streams else logits
