"""The Vekanex decoder as a list of parts.

Embedding ``embed``, head ``head`` with capped logits, last norm ``final.norm``.  Every layer ``l<i>`` norms what its
sublayers give and not what they read, ``x += m norm1(mixer(x))`` and ``x += m norm2(mlp(x))`` with one factor m for the
model.  Three mixers, chosen per layer:

* ``mlstm``: a matrix memory with exponential gates and a running maximum (``mix.q/k/v/g``, ``mix.i``, ``mix.f`` with biases,
  ``mix.norm``, ``mix.o``);
* ``gla``: linear attention with a decay per key channel out of a low-rank projection (``mix.q/k/v/g``, ``mix.a1``,
  ``mix.a2``, ``mix.norm``, ``mix.o``);
* ``parallel``: two mixers side by side whose results are added with a weight each.  ``mix.left.*``: grouped-query attention
  with biased projections, one norm over all query heads and one over all key heads and rotary positions in half pairs.
  ``mix.right.*``: the gated delta rule behind a short convolution, with a decay per key channel and a low-rank gate.

The feed-forward is a mixture of gated experts (``mlp.e<k>.gate/up/down``, ``mlp.router``) weighed by a softmax over the
chosen ones' logits, with an expert that every token uses (``mlp.shared.gate/up/down``); a layer may have none.  A layer may
use another layer's tensors, with a cache entry of its own.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.vekanex import ARCHITECTURE, VekanexConfig
from ..parts.spec import (EmbeddingSpec, ExpGateMemorySpec, GatedDeltaRuleSpec, GatedLinearAttentionSpec, HeadSpec, LayerSpec,
                          MixerPairSpec, ModelSpec, NormedAttentionSpec, NormSpec, RotarySpec, RoutedMlpSpec, ScheduleEntry,
                          SharedExpertSpec)

# what the design fixes
DENOMINATOR_EPS = 1e-6               # beside the floor of an exponential-gate memory's denominator
UNIT_EPS = 1e-6                      # in the length of the delta rule's queries and keys
EXPERT_ACTIVATION = "silu"
ROUTER_SCORES = "softmax"            # over all experts, then renormalised: a softmax over the chosen ones' logits


def _mixer_spec(config: VekanexConfig, layer, p: str):
    m = layer.mixer
    if layer.type == "mlstm":
        return ExpGateMemorySpec(
            hidden_size=config.width, num_heads=m.heads, dim=m.dim, vdim=m.vdim, gate_cap=m.gate_cap,
            denominator_eps=DENOMINATOR_EPS, eps=config.norm_eps, q_weight=p + "q", k_weight=p + "k", v_weight=p + "v",
            input_weight=p + "i", input_bias=p + "i.b", forget_weight=p + "f", forget_bias=p + "f.b", gate_weight=p + "g",
            norm=p + "norm", o_weight=p + "o")
    if layer.type == "gla":
        return GatedLinearAttentionSpec(
            hidden_size=config.width, num_heads=m.heads, dim=m.dim, vdim=m.vdim, tau=m.tau, decay_rank=m.rank,
            eps=config.norm_eps, q_weight=p + "q", k_weight=p + "k", v_weight=p + "v", gate_weight=p + "g",
            decay_down=p + "a1", decay_up=p + "a2", decay_bias=p + "a2.b", norm=p + "norm", o_weight=p + "o")
    l, r, a, d = p + "left.", p + "right.", m.left, m.right
    left = NormedAttentionSpec(
        hidden_size=config.width, num_heads=a.heads, num_kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale,
        eps=config.norm_eps, q_weight=l + "q", k_weight=l + "k", v_weight=l + "v", o_weight=l + "o", q_norm=l + "q.norm",
        k_norm=l + "k.norm", rope=RotarySpec(a.rot_dims, a.rot_base) if a.rot_dims else None, q_bias=l + "q.b",
        k_bias=l + "k.b", v_bias=l + "v.b", o_bias=l + "o.b")
    right = GatedDeltaRuleSpec(
        hidden_size=config.width, num_heads=d.heads, num_kv_heads=d.kv_heads, dim=d.dim, vdim=d.vdim, taps=d.taps,
        decay_rank=d.decay_rank, gate_rank=d.gate_rank, unit_eps=UNIT_EPS, eps=config.norm_eps, q_weight=r + "q",
        k_weight=r + "k", v_weight=r + "v", q_conv=r + "q.conv", k_conv=r + "k.conv", v_conv=r + "v.conv",
        beta_weight=r + "b", a_log=r + "A_log", decay_down=r + "a1", decay_up=r + "a2", dt_bias=r + "dt_bias",
        gate_down=r + "g1", gate_up=r + "g2", norm=r + "norm", o_weight=r + "o")
    return MixerPairSpec(left, right, m.left_scale, m.right_scale)


def _mlp_spec(config: VekanexConfig, mlp, p: str):
    names = lambda part: tuple(f"{p}e{k}.{part}" for k in range(mlp.experts))
    shared = None
    if mlp.shared_ff:
        shared = SharedExpertSpec(mlp.shared_ff, p + "shared.up", p + "shared.down", unit_gate_weight=p + "shared.gate")
    return RoutedMlpSpec(
        hidden_size=config.width, intermediate_size=mlp.ff, experts=mlp.experts, top=mlp.top, activation=EXPERT_ACTIVATION,
        route_scale=1.0, router_weight=p + "router", up_weights=names("up"), down_weights=names("down"), renormalize=True,
        shared=shared, gate_weights=names("gate"), score=ROUTER_SCORES)


def vekanex_spec(config: VekanexConfig) -> ModelSpec:
    if config.needs_tensor_shapes():
        raise ValueError("Vekanex: the rank of a low-rank part is open; open the model through load_config, which reads it "
                         "from the checkpoint, or give it in the mixer's section")
    layers, place, ignorable = [], {}, []
    for i, layer in enumerate(config.layers):
        if layer.weights_of is not None:
            continue
        p = f"l{i}."
        norm = lambda name: NormSpec(config.width, config.norm_eps, p + name, weight_scale=config.residual_mult)
        extras = [("mixer_post_norm", "norm", norm("norm1"))]
        ffn = None
        if layer.mlp is not None:
            ffn = _mlp_spec(config, layer.mlp, p + "mlp.")
            extras.append(("ffn_post_norm", "norm", norm("norm2")))
        else:
            ignorable.append(p + "norm2")            # (a checkpoint may carry a second norm all the same)
        place[i] = len(layers)
        layers.append(LayerSpec(mixer_norm=None, mixer=_mixer_spec(config, layer, p + "mix."), ffn=ffn,
                                arrangement="output_norm", extras=tuple(extras)))
    # a layer that uses another's tensors is one more run of it, with a cache entry of its own
    schedule = tuple(ScheduleEntry(layer=place[config.owner(i)], cache=i) for i in range(len(config.layers)))
    return ModelSpec(
        architecture=config.architecture, hidden_size=config.width, vocab_size=config.vocab,
        embedding=EmbeddingSpec(config.vocab, config.width, "embed"), layers=tuple(layers), schedule=schedule,
        final_norm=NormSpec(config.width, config.norm_eps, "final.norm"),
        head=HeadSpec(config.vocab, config.width, "head", softcap=config.logit_softcap), ignorable=tuple(ignorable))


register_architecture(ARCHITECTURE, VekanexConfig, vekanex_spec)
