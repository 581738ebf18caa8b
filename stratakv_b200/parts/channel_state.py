"""Mixers whose memory of a sequence is a matrix per head that decays by one number per key channel and token
(``csrc/channel_state.cu``): gated linear attention and the gated delta rule.  With D_t the diagonal matrix of the decays::

    plain:  S_t = D_t S_(t-1) + k_t v_t^T                                                 o_t = S_t^T q_t
    delta:  S_t = D_t S_(t-1) + k_t (beta_t (v_t - (D_t S_(t-1))^T k_t))^T                 per head, float32, S = 0 at the start

between an input and an output projection, with a norm per head and a gate in front of the latter.  The decays come out of a
low-rank projection whose first half is part of the input projection.  The cache keeps nothing per position: per sequence its
state area holds S twice, in the half chosen by the parity of the last position written, and for the delta rule a ring with
the short convolution's last inputs.
"""
from __future__ import annotations

import torch

from .. import ops as _ops
from .attention import _residual_mode, _residual_stats
from .base import CacheRequest, TensorRequest
from .linear_state import _StateMixer
from .registry import register_mixer


def _transposed(weight):
    return weight.t().contiguous()


class GatedLinearAttention(_StateMixer):
    """One projection for ``[q | k | v | gate | decays' first half]``.  One token a sequence: ``matrix_step`` does everything
    up to the output projection.  Longer steps: ``low_rank`` (the decays' logarithms), ``channel_state``, ``gated_norm``."""

    def __init__(self, spec, runtime):
        if not spec.tau > 0.0 or spec.decay_rank <= 0:
            raise ValueError("gated_linear_attention: the decays' exponent and rank must be positive")
        self.qk_dim = spec.num_heads * spec.dim
        inner = spec.num_heads * spec.vdim
        self.v_at, self.gate_at = 2 * self.qk_dim, 2 * self.qk_dim + inner
        self.decay_at = self.gate_at + inner
        super().__init__(spec, runtime, inner, self.decay_at + spec.decay_rank)

    @classmethod
    def expected_tensors(cls, spec):
        qk, v, hidden = spec.num_heads * spec.dim, spec.num_heads * spec.vdim, spec.hidden_size
        return {spec.q_weight: TensorRequest((qk, hidden)), spec.k_weight: TensorRequest((qk, hidden)),
                spec.v_weight: TensorRequest((v, hidden)), spec.gate_weight: TensorRequest((v, hidden)),
                spec.decay_down: TensorRequest((spec.decay_rank, hidden)), spec.decay_up: TensorRequest((qk, spec.decay_rank)),
                spec.decay_bias: TensorRequest((qk,), "half_normal"), spec.norm: TensorRequest((spec.vdim,), "around_one"),
                spec.o_weight: TensorRequest((hidden, v))}

    @classmethod
    def cache_request(cls, spec):
        return CacheRequest(kind="none", state_bytes=4 * 2 * spec.num_heads * spec.dim * spec.vdim)

    def bind(self, tensors):
        s, rt = self.spec, self.rt
        self._bind_projections([rt.upload(tensors[name]) for name in (s.q_weight, s.k_weight, s.v_weight, s.gate_weight,
                                                                      s.decay_down)], rt.upload(tensors[s.o_weight]))
        self.decay_wt = _transposed(rt.upload(tensors[s.decay_up]))
        as_float = lambda name: rt.upload(tensors[name], torch.float32).reshape(-1)
        self.decay_bias = as_float(s.decay_bias).contiguous()
        self.norm = as_float(s.norm).repeat(s.num_heads).contiguous()

    def forward(self, step, h, x, cache_entry, writes_cache=True):
        s, rt = self.spec, self.rt
        ops = rt.kernels()
        get = rt.workspace.get
        n, heads = h.shape[0], s.num_heads
        fused = get("qkv", (n, self.fused_width), torch.float32)
        ops.linear(h, self.w_in, fused, _ops.MODE_STORE_F32)
        state = step.cache.state(cache_entry).view(torch.float32)
        meta = (step.positions, step.token_seq, step.cu_q, step.slot_ids)
        q_scale = s.dim ** -0.5
        if step.is_decode:
            mixed = self._mixed(n)
            ops.matrix_step(_ops.STEP_CHANNEL, fused, 0, self.qk_dim, self.v_at, mixed, state, meta, heads, heads, s.dim, s.vdim,
                            self.norm, s.eps, self.gate_at, q_scale=q_scale, decay_at=self.decay_at, decay_wt=self.decay_wt,
                            decay_bias=self.decay_bias, decay_mode=_ops.LOW_RANK_LOG_SIGMOID, decay_factor=1.0 / s.tau,
                            gate_silu=True)
            ops.linear(mixed, self.w_o, x, _residual_mode(step), stats=_residual_stats(step))
            return
        log_decay = get("channel_log_decays", (n, self.qk_dim), torch.float32)
        ops.low_rank(fused, self.decay_at, self.decay_wt, log_decay, bias=self.decay_bias, mode=_ops.LOW_RANK_LOG_SIGMOID,
                     factor=1.0 / s.tau)
        y = get("linear_state_y", (n, self.inner), torch.float32)
        need = ops.channel_state_scratch(n, step.n_seqs, step.max_q_len, heads, s.dim, s.vdim, False)
        ops.channel_state(fused, 0, self.qk_dim, self.v_at, log_decay, y, state, meta, heads, heads, s.dim, s.vdim,
                          step.max_q_len, get("channel_state_scratch", (need,), torch.float32), q_scale=q_scale)
        self._project_out(step, ops, y, fused[:, self.gate_at:], self.fused_width, heads, _ops.GATE_SILU, x)


class GatedDeltaRule(_StateMixer):
    """One projection for ``[q | k | v | beta | decays' first half | gate's first half]``; the first three are convolved.  One
    token a sequence: ``matrix_step`` does everything up to the output projection.  Longer steps: ``conv_silu``, ``low_rank``
    twice (the decays' logarithms, the gate's logits), ``channel_state`` with the delta rule, ``short_conv_remember``,
    ``gated_norm``.  ``state_offset`` (floats): where this mixer's state starts in its cache entry's rows; ``out_scale``: a
    factor on the mixer's result, for a mixer that is one side of a weighted pair."""
    honours_state_offset = True
    scales_output = True

    def __init__(self, spec, runtime):
        if spec.num_kv_heads <= 0 or spec.num_heads % spec.num_kv_heads:
            raise ValueError("gated_delta_rule: heads must be a multiple of the query and key heads")
        if spec.taps < 1 or spec.decay_rank <= 0 or spec.gate_rank <= 0:
            raise ValueError("gated_delta_rule: the convolution needs a tap and the low-rank parts a rank")
        self.qk_dim = spec.num_kv_heads * spec.dim
        inner = spec.num_heads * spec.vdim
        self.channels = 2 * self.qk_dim + inner
        self.beta_at = self.channels
        self.decay_at = self.beta_at + spec.num_heads
        self.gate_at = self.decay_at + spec.decay_rank
        self.state_offset, self.out_scale = 0, 1.0
        super().__init__(spec, runtime, inner, self.gate_at + spec.gate_rank)

    @classmethod
    def expected_tensors(cls, spec):
        qk, decays, v = spec.num_kv_heads * spec.dim, spec.num_heads * spec.dim, spec.num_heads * spec.vdim
        hidden, heads = spec.hidden_size, spec.num_heads
        return {spec.q_weight: TensorRequest((qk, hidden)), spec.k_weight: TensorRequest((qk, hidden)),
                spec.v_weight: TensorRequest((v, hidden)), spec.q_conv: TensorRequest((qk, spec.taps), "conv_taps"),
                spec.k_conv: TensorRequest((qk, spec.taps), "conv_taps"), spec.v_conv: TensorRequest((v, spec.taps), "conv_taps"),
                spec.beta_weight: TensorRequest((heads, hidden)), spec.a_log: TensorRequest((heads,), "log_rate"),
                spec.decay_down: TensorRequest((spec.decay_rank, hidden)), spec.decay_up: TensorRequest((decays, spec.decay_rank)),
                spec.dt_bias: TensorRequest((decays,), "decay_logit"), spec.gate_down: TensorRequest((spec.gate_rank, hidden)),
                spec.gate_up: TensorRequest((v, spec.gate_rank)), spec.norm: TensorRequest((spec.vdim,), "around_one"),
                spec.o_weight: TensorRequest((hidden, v))}

    @staticmethod
    def matrix_floats(spec) -> int:
        return 2 * spec.num_heads * spec.dim * spec.vdim

    @classmethod
    def cache_request(cls, spec):
        channels = 2 * spec.num_kv_heads * spec.dim + spec.num_heads * spec.vdim
        floats = cls.matrix_floats(spec) + (spec.taps * channels if spec.taps > 1 else 0)
        return CacheRequest(kind="none", state_bytes=4 * (-(-floats // 4) * 4))      # (rows of whole 16 bytes)

    def bind(self, tensors):
        s, rt = self.spec, self.rt
        self._bind_projections([rt.upload(tensors[name]) for name in (s.q_weight, s.k_weight, s.v_weight, s.beta_weight,
                                                                      s.decay_down, s.gate_down)], rt.upload(tensors[s.o_weight]))
        self.decay_wt, self.gate_wt = _transposed(rt.upload(tensors[s.decay_up])), _transposed(rt.upload(tensors[s.gate_up]))
        as_float = lambda name: rt.upload(tensors[name], torch.float32)
        self.conv_w = torch.cat([as_float(name) for name in (s.q_conv, s.k_conv, s.v_conv)], dim=0).contiguous()
        self.decay_rate = torch.exp(as_float(s.a_log).reshape(-1)).contiguous()
        self.dt_bias = as_float(s.dt_bias).reshape(-1).contiguous()
        self.norm = (as_float(s.norm).reshape(-1).repeat(s.num_heads) * self.out_scale).contiguous()

    def forward(self, step, h, x, cache_entry, writes_cache=True):
        s, rt = self.spec, self.rt
        ops = rt.kernels()
        get = rt.workspace.get
        n, heads = h.shape[0], s.num_heads
        fused = get("qkv", (n, self.fused_width), torch.float32)
        ops.linear(h, self.w_in, fused, _ops.MODE_STORE_F32)
        state = step.cache.state(cache_entry).view(torch.float32)
        meta = (step.positions, step.token_seq, step.cu_q, step.slot_ids)
        ring_offset = self.state_offset + self.matrix_floats(s)
        shape = (heads, s.num_kv_heads, s.dim, s.vdim)
        q_scale = s.dim ** -0.5
        if step.is_decode:
            mixed = self._mixed(n)
            ops.matrix_step(_ops.STEP_DELTA, fused, 0, self.qk_dim, 2 * self.qk_dim, mixed, state, meta, *shape, self.norm, s.eps,
                            self.gate_at, q_scale=q_scale, unit_eps=s.unit_eps, conv_w=self.conv_w, ring_offset=ring_offset,
                            decay_at=self.decay_at, decay_wt=self.decay_wt, decay_bias=self.dt_bias,
                            decay_mode=_ops.LOW_RANK_SOFTPLUS, decay_rate=self.decay_rate, beta_at=self.beta_at,
                            gate_wt=self.gate_wt, state_offset=self.state_offset)
            ops.linear(mixed, self.w_o, x, _residual_mode(step), stats=_residual_stats(step))
            return
        convolved = get("conv_rows", (n, self.channels), torch.float32)
        ops.conv_silu(fused, self.conv_w, None, convolved, meta, state, ring_offset)
        log_decay = get("channel_log_decays", (n, heads * s.dim), torch.float32)
        ops.low_rank(fused, self.decay_at, self.decay_wt, log_decay, bias=self.dt_bias, mode=_ops.LOW_RANK_SOFTPLUS,
                     rate=self.decay_rate)
        gate = get("channel_gates", (n, self.inner), torch.float32)
        ops.low_rank(fused, self.gate_at, self.gate_wt, gate)
        y = get("linear_state_y", (n, self.inner), torch.float32)
        need = ops.channel_state_scratch(n, step.n_seqs, step.max_q_len, heads, s.dim, s.vdim, True)
        ops.channel_state(convolved, 0, self.qk_dim, 2 * self.qk_dim, log_decay, y, state, meta, *shape, step.max_q_len,
                          get("channel_state_scratch", (need,), torch.float32), q_scale=q_scale, beta_rows=fused,
                          beta_at=self.beta_at, unit_eps=s.unit_eps, state_offset=self.state_offset)
        ops.short_conv_remember(fused, None, self.channels, s.taps, step.n_seqs, meta, state, ring_offset)
        self._project_out(step, ops, y, gate, self.inner, heads, _ops.GATE_SIGMOID, x)


register_mixer("gated_linear_attention", GatedLinearAttention)
register_mixer("gated_delta_rule", GatedDeltaRule)
