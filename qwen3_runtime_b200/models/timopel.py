"""Timopel expressed as data for the generic decoder.

The token's row times a constant enters the stream.  Blocks norm both the input and the output of each sublayer
(``sandwich_norm``), a sublayer's normed output times ``residual_mult`` is added.  The mixer is causal attention with
grouped key/value heads, normed q and k, a learned sink per head and a query temperature in place of positions; the
values of every mixing layer but the first take a learned share of the first one's.  The feed-forward is a dense gated
gelu layer, routed clamped experts with a shared one, or absent.  The head is the embedding table.
Tensor names: ``embed``, ``l<i>.norm1 | norm1b | norm2 | norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``.
"""

from __future__ import annotations

from ..config.logesun_config import ExpertConfig
from ..config.registry import register_architecture
from ..config.spec import ModelSpec, PartSpec
from ..config.timopel_config import (DenseConfig, MixedValueAttentionConfig, MoeConfig, TemperatureConfig, TimopelConfig,
                                     TimopelLayerConfig)


def _mixer_spec(cfg: TimopelConfig, index: int) -> PartSpec:
    m = cfg.layers[index].mixer
    value_mix = None
    if m.v_mix:
        value_mix = "source" if index == cfg.first_mixing_layer() else "blend"
    return PartSpec("sink_window_attention", dict(
        hidden_size=cfg.width, num_heads=m.heads, num_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale,
        window=None, sink="learned", gate=None, qk_norm_eps=cfg.norm_eps, value_mix=value_mix,
        query_temperature=(m.q_temp.coef, m.q_temp.every) if m.q_temp else None))


def _feed_forward_spec(cfg: TimopelConfig, f: DenseConfig | MoeConfig) -> PartSpec:
    if isinstance(f, DenseConfig):
        return PartSpec("gated_mlp", dict(hidden_size=cfg.width, intermediate_size=f.ff, activation="gelu",
                                          names=dict(gate="gate", up="up", down="down")))
    return PartSpec("routed_experts", dict(
        hidden_size=cfg.width, num_experts=f.experts, top=f.top, expert_size=f.expert.ff, limit=f.expert.limit,
        alpha=1.702, up_offset=1.0, score="softmax_all", renormalize=True, weight_scale=f.scale, weight_on="output",
        shared_size=f.shared.ff if f.shared else 0, shared_limit=f.shared.limit if f.shared else None))


def timopel_spec(cfg: TimopelConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", dict(size=cfg.width, eps=cfg.norm_eps, weight_name=""))
    out_norm = PartSpec("rmsnorm", dict(size=cfg.width, eps=cfg.norm_eps, weight_name="", weight_scale=cfg.residual_mult))
    blocks = []
    for i, layer in enumerate(cfg.layers):
        params = dict(mixer=_mixer_spec(cfg, i), mixer_norm=norm, mixer_out_norm=out_norm, mixer_prefix="mix.",
                      mixer_norm_prefix="norm1", mixer_out_norm_prefix="norm1b", feed_forward=None)
        if layer.mlp is not None:
            params.update(feed_forward=_feed_forward_spec(cfg, layer.mlp), feed_forward_norm=norm,
                          feed_forward_out_norm=out_norm, feed_forward_prefix="mlp.", feed_forward_norm_prefix="norm2",
                          feed_forward_out_norm_prefix="norm2b")
        blocks.append(PartSpec("sandwich_norm", params))
    embedding = PartSpec("scaled_bigram", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, scale=cfg.embed_scale,
                                               embed_name="embed"))
    return ModelSpec(vocab_size=cfg.vocab, hidden_size=cfg.width, blocks=tuple(blocks),
                     order=ModelSpec.sequential_order(len(blocks)), final_norm=norm, tie_word_embeddings=True,
                     embed_name="embed", head_name="head", block_prefix="l{index}.", final_norm_prefix="final.norm",
                     embedding=embedding)


def tiny_timopel_config() -> TimopelConfig:
    """A small model with every branch of the design: layers that mix values and one that does not, with and without a
    query temperature, a dense and a routed feed-forward, a layer without one."""
    def attention(**kw):
        base = dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.25, q_temp=TemperatureConfig(0.4, 6), v_mix=True)
        return MixedValueAttentionConfig(**{**base, **kw})

    moe = MoeConfig(experts=4, top=2, scale=1.5, expert=ExpertConfig(16, 1.5), shared=ExpertConfig(24, 2.0))
    layers = (TimopelLayerConfig("attention", attention(), DenseConfig(48)),
              TimopelLayerConfig("attention", attention(heads=2, kv_heads=1, vdim=16, v_mix=False, q_temp=None), moe),
              TimopelLayerConfig("attention", attention(dim=24), None))
    return TimopelConfig(vocab=64, width=40, norm_eps=1e-5, layers=layers, embed_scale=2.0, residual_mult=0.5)


register_architecture(TimopelConfig.architecture, TimopelConfig, timopel_spec, tiny_config=tiny_timopel_config)
