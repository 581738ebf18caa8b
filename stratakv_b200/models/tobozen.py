"""The Tobozen decoder as a list of parts.

Embedding ``embed``, which is also the head; last norm ``final.norm``.  Every layer ``l<i>`` is a pre-norm block whose
norms work in groups (the vector in equal parts, each divided by its own root mean square).  Three mixers, chosen per
layer:

* ``attention``: grouped-query attention with one norm over all query heads and one over all key heads (``mix.q.norm``,
  ``mix.k.norm``), rotary positions in interleaved pairs, one added to the softmax's denominator, and in layers that mix
  values the first such layer's values taken in with the weight ``mix.vmix``;
* ``mamba2``: the Mamba-2 mixer (``mix.in``, ``mix.conv``, ``mix.dt_bias``, ``mix.A_log``, ``mix.D``, ``mix.norm``);
* ``lightning``: linear attention with a fixed decay per head, silu on queries, keys and values, and a gated norm over all
  heads (``mix.q/k/v/g``, ``mix.norm``).

The feed-forward is a mixture of clamped gated experts (``mlp.e<k>.gate/up/down``, ``mlp.router``) whose weights multiply
their inputs; a layer may have none.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tobozen import ARCHITECTURE, TobozenConfig
from ..parts.spec import (DecayAttentionSpec, EmbeddingSpec, HeadSpec, LayerSpec, Mamba2Spec, ModelSpec, NormedAttentionSpec,
                          NormSpec, RotarySpec, RoutedMlpSpec, ScheduleEntry)

# what the design fixes
EXPERT_ACTIVATION = "swiglu_clamp"
ROUTER_SCORES = "sigmoid"
ROTATION_INTERLEAVED = True
SINK_SCORE = 0.0                     # exp(0) = 1 is added to the softmax's denominator


def _mixer_spec(config: TobozenConfig, layer, p: str, keeps_values: bool):
    m = layer.mixer
    if layer.type == "attention":
        return NormedAttentionSpec(
            hidden_size=config.width, num_heads=m.heads, num_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale,
            eps=config.norm_eps, q_weight=p + "q", k_weight=p + "k", v_weight=p + "v", o_weight=p + "o",
            q_norm=p + "q.norm", k_norm=p + "k.norm",
            rope=RotarySpec(m.rot_dims, m.rot_base, interleaved=ROTATION_INTERLEAVED) if m.rot_dims else None,
            sink_score=SINK_SCORE, keeps_values=keeps_values,
            value_mix=p + "vmix" if m.v_mix and not keeps_values else None)
    if layer.type == "mamba2":
        return Mamba2Spec(
            hidden_size=config.width, num_heads=m.heads, vdim=m.vdim, state=m.state, groups=m.groups, taps=m.taps,
            norm_groups=m.norm_groups, eps=config.norm_eps, in_weight=p + "in", conv_weight=p + "conv",
            conv_bias=p + "conv.b", dt_bias=p + "dt_bias", a_log=p + "A_log", skip=p + "D", norm=p + "norm",
            o_weight=p + "o")
    return DecayAttentionSpec(
        hidden_size=config.width, num_heads=m.heads, dim=m.dim, vdim=m.vdim, decay=m.decay, eps=config.norm_eps,
        q_weight=p + "q", k_weight=p + "k", v_weight=p + "v", gate_weight=p + "g", norm=p + "norm", o_weight=p + "o")


def _mlp_spec(config: TobozenConfig, mlp, p: str):
    names = lambda part: tuple(f"{p}e{k}.{part}" for k in range(mlp.experts))
    return RoutedMlpSpec(
        hidden_size=config.width, intermediate_size=mlp.ff, experts=mlp.experts, top=mlp.top,
        activation=EXPERT_ACTIVATION, activation_param=mlp.limit, route_scale=1.0, router_weight=p + "router",
        up_weights=names("up"), down_weights=names("down"), gate_weights=names("gate"), score=ROUTER_SCORES,
        weigh_input=True)


def tobozen_spec(config: TobozenConfig) -> ModelSpec:
    norm = lambda name: NormSpec(config.width, config.norm_eps, name, groups=config.norm_groups)
    layers, ignorable, first_mixing = [], [], None
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        keeps = False
        if layer.type == "attention" and layer.mixer.v_mix and first_mixing is None:
            first_mixing, keeps = i, True
            ignorable.append(p + "mix.vmix")         # the first layer that mixes values has nobody's to take in
        ffn = ffn_norm = None
        if layer.mlp is not None:
            ffn, ffn_norm = _mlp_spec(config, layer.mlp, p + "mlp."), norm(p + "norm2")
        else:
            ignorable.append(p + "norm2")            # (a checkpoint may carry a second norm all the same)
        layers.append(LayerSpec(mixer_norm=norm(p + "norm1"), mixer=_mixer_spec(config, layer, p + "mix.", keeps),
                                ffn_norm=ffn_norm, ffn=ffn, arrangement="pre_norm"))
    return ModelSpec(
        architecture=config.architecture, hidden_size=config.width, vocab_size=config.vocab,
        embedding=EmbeddingSpec(config.vocab, config.width, "embed"), layers=tuple(layers),
        schedule=tuple(ScheduleEntry(layer=i, cache=i) for i in range(len(layers))), final_norm=norm("final.norm"),
        head=HeadSpec(config.vocab, config.width, "embed"), ignorable=tuple(ignorable))


register_architecture(ARCHITECTURE, TobozenConfig, tobozen_spec)
