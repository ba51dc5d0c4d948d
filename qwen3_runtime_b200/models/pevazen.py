"""Pevazen expressed as data for the generic decoder.

The embedding is normed before it enters the stream.  A layer has one norm (a single number as its weight) whose
output both the mixer and the feed-forward read; what goes on is a learned average of the embedding output and all
layers' results so far (``shared_norm`` blocks with ``depth_points``).  The mixer of a layer is attention under a
chunked mask with biases on q, k and v (``attention``), possibly on the keys and values another layer has stored, or
two mixers side by side (``parallel``): attention under a chunked mask whose values are turned by their positions, and
the gated delta rule; each of the two outputs is normed and half of their sum goes on.  The feed-forward is a dense
SwiGLU layer or absent.  Tensor names: ``embed``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``l<i>.dwa``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.pevazen_config import (ChunkedAttentionConfig, DeltaConfig, PevazenConfig, PevazenLayerConfig,
                                     SideBySideConfig)
from ..config.registry import register_architecture
from ..config.spec import LayerRun, ModelSpec, PartSpec
from ..config.tabisun_config import RotaryConfig


def _attention_spec(cfg: PevazenConfig, m: ChunkedAttentionConfig, **options) -> PartSpec:
    position = None
    if m.rot is not None:
        scaling = dict(m.rot.scaling, kind="linear") if m.rot.scaling else None
        position = PartSpec("rotary_scaled", dict(rotary_dim=m.rot.dims, theta=m.rot.base, pairing="half", scaling=scaling))
    return PartSpec("sink_window_attention", dict(
        hidden_size=cfg.width, num_heads=m.heads, num_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale,
        window=None, sink=None, gate=None, qk_norm_eps=None, chunk=m.chunk, position=position, **options))


def _mixer_spec(cfg: PevazenConfig, m) -> PartSpec:
    if isinstance(m, ChunkedAttentionConfig):
        return _attention_spec(cfg, m, qkv_bias=True, own_kv=m.kv_from is None)
    left = _attention_spec(cfg, m.left, value_turn=m.left.rot.base)
    d = m.right
    if not d.decay_rank or not d.gate_rank:
        raise ValueError("delta rule: the ranks are not known yet; they are the row counts of the stored a1 and g1 "
                         "(PevazenConfig.with_tensor_shapes)")
    right = PartSpec("gated_delta", dict(
        hidden_size=cfg.width, num_heads=d.heads, num_kv_heads=d.kv_heads, dim=d.dim, vdim=d.vdim, taps=d.conv,
        decay_rank=d.decay_rank, gate_rank=d.gate_rank, eps=cfg.norm_eps))
    return PartSpec("parallel", dict(
        hidden_size=cfg.width, branches=(("left.", left, 0.5), ("right.", right, 0.5)),
        out_norms=(("left.out", cfg.norm_eps), ("right.out", cfg.norm_eps))))


def pevazen_spec(cfg: PevazenConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", dict(size=cfg.width, eps=cfg.norm_eps, weight_name="", scalar=True))
    blocks = []
    for i, layer in enumerate(cfg.layers):
        params = dict(mixer=_mixer_spec(cfg, layer.mixer), norm=norm, mixer_prefix="mix.", norm_prefix="norm1",
                      feed_forward=None, depth_points=i + 2, depth_name="dwa")
        if layer.ff:
            params.update(feed_forward=PartSpec("gated_mlp", dict(
                hidden_size=cfg.width, intermediate_size=layer.ff, activation="silu",
                names=dict(gate="gate", up="up", down="down"))), feed_forward_prefix="mlp.")
        blocks.append(PartSpec("shared_norm", params))
    sources = [getattr(layer.mixer, "kv_from", None) for layer in cfg.layers]
    order = tuple(LayerRun(block=i, cache=i if j is None else j, writes=j is None) for i, j in enumerate(sources))
    embedding = PartSpec("normed_lookup", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, eps=cfg.norm_eps, scalar=True,
                                               embed_name="embed", weight_name="embed.norm"))
    return ModelSpec(vocab_size=cfg.vocab, hidden_size=cfg.width, blocks=tuple(blocks), order=order, final_norm=norm,
                     tie_word_embeddings=False, embed_name="embed", head_name="head", block_prefix="l{index}.",
                     final_norm_prefix="final.norm", embedding=embedding)


def tiny_pevazen_config() -> PevazenConfig:
    """A small model with every branch of the design: both mixers, keys and values of another layer under another
    mask, a layer without a feed-forward."""
    rot = RotaryConfig(dims=8, base=10000.0)
    own = ChunkedAttentionConfig(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.25, rot=rot, chunk=12)
    reader = ChunkedAttentionConfig(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.25, rot=rot, chunk=20, kv_from=1)
    side = SideBySideConfig(
        left=ChunkedAttentionConfig(heads=2, kv_heads=1, dim=16, vdim=8, scale=0.25, chunk=16,
                                    rot=RotaryConfig(dims=16, base=500.0, scaling=(("factor", 2.0),))),
        right=DeltaConfig(heads=4, kv_heads=2, dim=8, vdim=16, conv=3, decay_rank=8, gate_rank=8))
    layers = (PevazenLayerConfig("parallel", side, 48), PevazenLayerConfig("attention", own, 40),
              PevazenLayerConfig("parallel", side, None), PevazenLayerConfig("attention", reader, 40))
    return PevazenConfig(vocab=64, width=40, norm_eps=1e-5, layers=layers)


register_architecture(PevazenConfig.architecture, PevazenConfig, pevazen_spec, tiny_config=tiny_pevazen_config)
