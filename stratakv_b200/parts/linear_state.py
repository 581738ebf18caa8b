"""Mixers whose memory of a sequence is a matrix per head that decays by one number a token (``csrc/linear_state.cu``):
Mamba-2, whose decay, keys, queries and values come out of a convolution and a step size, Lightning attention, whose
decay is fixed per head, and memories with exponential gates (the mLSTM), whose output is divided by what a key sum of the
same decays says.  All are::

    S_t = d_t S_(t-1) + c_t k_t v_t^T,   o_t = S_t^T q_t + skip v_t          per head, float32, S = 0 before the first token

between an input and an output projection, with a gated norm in front of the latter.  The cache keeps nothing per
position: per sequence its state area holds S twice, in the half chosen by the parity of the last position written,
for Mamba-2 a ring with the convolution's last inputs, and for exponential gates the key sums (behind each half's S) and the
running maxima.
"""
from __future__ import annotations

import torch

from .. import ops as _ops
from .attention import _residual_mode, _residual_stats
from .base import CacheRequest, Mixer, TensorRequest
from .registry import register_mixer


class _StateMixer(Mixer):
    graph_safe = True
    stores_branch = True

    def __init__(self, spec, runtime, inner: int, in_rows: int):
        super().__init__(spec, runtime)
        if runtime.dtype == torch.bfloat16 and spec.hidden_size % 8 != 0:
            raise ValueError(f"{spec.kind}: hidden size {spec.hidden_size} is not supported in bfloat16 "
                             "(rows of 16 bytes are needed: a multiple of 8); float32 takes any size")
        self.inner = inner
        self.fused_width = -(-in_rows // 8) * 8
        self.out_width = -(-inner // 8) * 8                # whole 16 bytes for the output projection

    def _bind_projections(self, parts, w_o):
        """``parts``: the input projection's rows in the order the kernels read them."""
        hidden = self.spec.hidden_size
        missing = self.fused_width - sum(part.shape[0] for part in parts)
        if missing:                                        # (zero rows: what they produce is never read)
            parts = list(parts) + [parts[0].new_zeros(missing, hidden)]
        self.w_in = torch.cat(parts, dim=0).contiguous()
        if self.out_width != self.inner:
            w_o = torch.cat([w_o, w_o.new_zeros(hidden, self.out_width - self.inner)], dim=1)
        self.w_o = w_o.contiguous()

    def _scratch(self, ops, step, heads, dim, vdim, with_floor=False):
        need = ops.linear_state_scratch(step.n_seqs, step.max_q_len, heads, dim, vdim, with_floor)
        return self.rt.workspace.get("linear_state_chunks", (need,), torch.float32) if need else None

    def _mixed(self, n):
        """The output projection's input."""
        return self.rt.workspace.get("linear_state_out", (n, self.out_width), self.rt.dtype)

    def _project_out(self, step, ops, y, gate, gate_stride, groups, mode, x):
        mixed = self._mixed(y.shape[0])
        ops.gated_norm(y, gate, gate_stride, self.norm, groups, self.spec.eps, mode, mixed)
        ops.linear(mixed, self.w_o, x, _residual_mode(step), stats=_residual_stats(step))


class DecayAttention(_StateMixer):
    """``o = norm(sum of decayed k v^T, read by q) * sigmoid(Wg h)``: one projection for q, k, v and the gate's logits,
    ``linear_state`` with silu on what it reads, ``gated_norm``, the output projection."""

    def __init__(self, spec, runtime):
        if len(spec.decay) != spec.num_heads:
            raise ValueError("decay_attention: one decay per head is needed")
        if not all(0.0 <= d <= 1.0 for d in spec.decay):
            raise ValueError("decay_attention: decays lie between 0 and 1")
        self.qk_dim = spec.num_heads * spec.dim
        inner = spec.num_heads * spec.vdim
        super().__init__(spec, runtime, inner, 2 * self.qk_dim + 2 * inner)

    @classmethod
    def expected_tensors(cls, spec):
        qk, v = spec.num_heads * spec.dim, spec.num_heads * spec.vdim
        return {spec.q_weight: TensorRequest((qk, spec.hidden_size)), spec.k_weight: TensorRequest((qk, spec.hidden_size)),
                spec.v_weight: TensorRequest((v, spec.hidden_size)), spec.gate_weight: TensorRequest((v, spec.hidden_size)),
                spec.norm: TensorRequest((v,), "around_one"), spec.o_weight: TensorRequest((spec.hidden_size, v))}

    @classmethod
    def cache_request(cls, spec):
        return CacheRequest(kind="none", state_bytes=4 * 2 * spec.num_heads * spec.dim * spec.vdim)

    def bind(self, tensors):
        s, rt = self.spec, self.rt
        self._bind_projections([rt.upload(tensors[name]) for name in (s.q_weight, s.k_weight, s.v_weight, s.gate_weight)],
                               rt.upload(tensors[s.o_weight]))
        self.norm = rt.upload(tensors[s.norm], torch.float32).contiguous()
        self.decay = torch.tensor(list(s.decay), dtype=torch.float32).to(rt.device)

    def forward(self, step, h, x, cache_entry, writes_cache=True):
        s, rt = self.spec, self.rt
        ops = rt.kernels()
        n = h.shape[0]
        fused = rt.workspace.get("qkv", (n, self.fused_width), torch.float32)
        ops.linear(h, self.w_in, fused, _ops.MODE_STORE_F32)
        y = rt.workspace.get("linear_state_y", (n, self.inner), torch.float32)
        ops.linear_state(fused, 0, self.qk_dim, 2 * self.qk_dim, y, step.cache.state(cache_entry).view(torch.float32),
                         (step.positions, step.token_seq, step.cu_q, step.slot_ids), s.num_heads, s.num_heads, s.dim, s.vdim,
                         step.max_q_len, decay=self.decay, silu=True,
                         scratch=self._scratch(ops, step, s.num_heads, s.dim, s.vdim))
        self._project_out(step, ops, y, fused[:, 2 * self.qk_dim + self.inner:], self.fused_width, 1, _ops.GATE_SIGMOID, x)


class Mamba2(_StateMixer):
    """The input projection's rows are kept in the order ``[x | B | C | z | dt]`` (the checkpoint's are ``[z | x | B | C |
    dt]``), so that the convolved channels lie first.  One token a sequence: ``mamba2_step`` does convolution, step size
    and recurrence.  Longer steps: ``conv_silu``, ``step_sizes``, ``linear_state`` in chunks, ``short_conv_remember``.  Then
    ``gated_norm`` with silu(z) before the norm, and the output projection."""

    def __init__(self, spec, runtime):
        if spec.groups <= 0 or spec.num_heads % spec.groups:
            raise ValueError("mamba2: heads must be a multiple of the groups")
        if spec.taps < 1:
            raise ValueError("mamba2: the convolution needs at least one tap")
        inner = spec.num_heads * spec.vdim
        if spec.norm_groups < 1 or inner % spec.norm_groups:
            raise ValueError("mamba2: the norm's groups must split the inner width into equal parts")
        self.channels = inner + 2 * spec.groups * spec.state
        self.z_at, self.dt_at = self.channels, self.channels + inner
        super().__init__(spec, runtime, inner, self.dt_at + spec.num_heads)

    @classmethod
    def expected_tensors(cls, spec):
        inner = spec.num_heads * spec.vdim
        channels = inner + 2 * spec.groups * spec.state
        return {spec.in_weight: TensorRequest((inner + channels + spec.num_heads, spec.hidden_size)),
                spec.conv_weight: TensorRequest((channels, spec.taps), "conv_taps"), spec.conv_bias: TensorRequest((channels,)),
                spec.dt_bias: TensorRequest((spec.num_heads,), "decay_logit"), spec.a_log: TensorRequest((spec.num_heads,), "log_rate"),
                spec.skip: TensorRequest((spec.num_heads,), "around_one"), spec.norm: TensorRequest((inner,), "around_one"),
                spec.o_weight: TensorRequest((spec.hidden_size, inner))}

    @staticmethod
    def matrix_floats(spec) -> int:
        return 2 * spec.num_heads * spec.state * spec.vdim

    @classmethod
    def cache_request(cls, spec):
        channels = spec.num_heads * spec.vdim + 2 * spec.groups * spec.state
        floats = cls.matrix_floats(spec) + (spec.taps * channels if spec.taps > 1 else 0)
        return CacheRequest(kind="none", state_bytes=4 * (-(-floats // 4) * 4))      # (rows of whole 16 bytes)

    def bind(self, tensors):
        s, rt = self.spec, self.rt
        z, xbc, dt = torch.split(rt.upload(tensors[s.in_weight]), [self.inner, self.channels, s.num_heads], dim=0)
        self._bind_projections([xbc, z, dt], rt.upload(tensors[s.o_weight]))
        as_float = lambda name: rt.upload(tensors[name], torch.float32).contiguous()
        self.conv_w, self.conv_b = as_float(s.conv_weight), as_float(s.conv_bias)
        self.dt_bias, self.a_log, self.skip, self.norm = (as_float(name) for name in (s.dt_bias, s.a_log, s.skip, s.norm))
        self.ring_offset = self.matrix_floats(s)

    def forward(self, step, h, x, cache_entry, writes_cache=True):
        s, rt = self.spec, self.rt
        ops = rt.kernels()
        get = rt.workspace.get
        n, heads = h.shape[0], s.num_heads
        fused = get("qkv", (n, self.fused_width), torch.float32)
        ops.linear(h, self.w_in, fused, _ops.MODE_STORE_F32)
        state = step.cache.state(cache_entry).view(torch.float32)
        meta = (step.positions, step.token_seq, step.cu_q, step.slot_ids)
        y = get("linear_state_y", (n, self.inner), torch.float32)
        if step.is_decode:
            ops.mamba2_step(fused, self.conv_w, self.conv_b, self.dt_at, self.dt_bias, self.a_log, self.skip, y, state, meta,
                            heads, s.groups, s.state, s.vdim, 0, self.ring_offset)
        else:
            convolved = get("conv_rows", (n, self.channels), torch.float32)
            ops.conv_silu(fused, self.conv_w, self.conv_b, convolved, meta, state, self.ring_offset)
            dt, log_decay = get("step_sizes", (n, heads), torch.float32), get("log_decays", (n, heads), torch.float32)
            ops.step_sizes(fused, self.dt_at, self.dt_bias, self.a_log, dt, log_decay)
            group_width = s.groups * s.state
            ops.linear_state(convolved, self.inner + group_width, self.inner, 0, y, state, meta, heads, s.groups, s.state,
                             s.vdim, step.max_q_len, log_decay=log_decay, key_scale=dt, skip=self.skip,
                             scratch=self._scratch(ops, step, heads, s.state, s.vdim))
            ops.short_conv_remember(fused, None, self.channels, s.taps, step.n_seqs, meta, state, self.ring_offset)
        self._project_out(step, ops, y, fused[:, self.z_at:], self.fused_width, s.norm_groups, _ops.GATE_SILU_FIRST, x)


class ExpGateMemory(_StateMixer):
    """One projection for ``[q | k | v | output gate | input gates | forget gates]``.  One token a sequence: ``matrix_step``
    does everything up to the output projection.  Longer steps: ``exp_gates`` turns the gates' logits into decays and key
    factors (and the floor of the denominator), then ``linear_state`` in chunks and ``gated_norm`` with a part per head."""

    def __init__(self, spec, runtime):
        if not spec.gate_cap > 0.0:
            raise ValueError("exp_gate_memory: the gates' cap must be positive")
        self.qk_dim = spec.num_heads * spec.dim
        inner = spec.num_heads * spec.vdim
        self.v_at, self.gate_at = 2 * self.qk_dim, 2 * self.qk_dim + inner
        self.input_at, self.forget_at = self.gate_at + inner, self.gate_at + inner + spec.num_heads
        super().__init__(spec, runtime, inner, self.forget_at + spec.num_heads)

    @classmethod
    def expected_tensors(cls, spec):
        qk, v, heads, hidden = spec.num_heads * spec.dim, spec.num_heads * spec.vdim, spec.num_heads, spec.hidden_size
        return {spec.q_weight: TensorRequest((qk, hidden)), spec.k_weight: TensorRequest((qk, hidden)),
                spec.v_weight: TensorRequest((v, hidden)), spec.gate_weight: TensorRequest((v, hidden)),
                spec.input_weight: TensorRequest((heads, hidden)), spec.input_bias: TensorRequest((heads,)),
                spec.forget_weight: TensorRequest((heads, hidden)), spec.forget_bias: TensorRequest((heads,), "half_normal"),
                spec.norm: TensorRequest((v,), "around_one"), spec.o_weight: TensorRequest((hidden, v))}

    @staticmethod
    def half_floats(spec) -> int:
        return spec.num_heads * spec.dim * (spec.vdim + 1)

    @classmethod
    def cache_request(cls, spec):
        floats = 2 * cls.half_floats(spec) + 2 * spec.num_heads
        return CacheRequest(kind="none", state_bytes=4 * (-(-floats // 4) * 4))      # (rows of whole 16 bytes)

    def bind(self, tensors):
        s, rt = self.spec, self.rt
        self._bind_projections([rt.upload(tensors[name]) for name in (s.q_weight, s.k_weight, s.v_weight, s.gate_weight,
                                                                      s.input_weight, s.forget_weight)],
                               rt.upload(tensors[s.o_weight]))
        as_float = lambda name: rt.upload(tensors[name], torch.float32).contiguous()
        self.norm, self.input_bias, self.forget_bias = as_float(s.norm), as_float(s.input_bias), as_float(s.forget_bias)

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
            ops.matrix_step(_ops.STEP_EXP, fused, 0, self.qk_dim, self.v_at, mixed, state, meta, heads, heads, s.dim, s.vdim,
                            self.norm, s.eps, self.gate_at, q_scale=q_scale, input_at=self.input_at, forget_at=self.forget_at,
                            input_bias=self.input_bias, forget_bias=self.forget_bias, cap=s.gate_cap,
                            denominator_eps=s.denominator_eps)
            ops.linear(mixed, self.w_o, x, _residual_mode(step), stats=_residual_stats(step))
            return
        log_decay, key_scale, floor = (get(name, (n, heads), torch.float32) for name in ("log_decays", "key_scales", "floors"))
        ops.exp_gates(fused, self.input_at, self.forget_at, self.input_bias, self.forget_bias, s.gate_cap, log_decay, key_scale,
                      floor, meta, state, 2 * self.half_floats(s))
        y = get("linear_state_y", (n, self.inner), torch.float32)
        ops.linear_state(fused, 0, self.qk_dim, self.v_at, y, state, meta, heads, heads, s.dim, s.vdim, step.max_q_len,
                         log_decay=log_decay, key_scale=key_scale, scratch=self._scratch(ops, step, heads, s.dim, s.vdim, True),
                         out_scale=q_scale, floor=floor, floor_eps=s.denominator_eps)
        self._project_out(step, ops, y, fused[:, self.gate_at:], self.fused_width, heads, _ops.GATE_SIGMOID, x)


register_mixer("decay_attention", DecayAttention)
register_mixer("exp_gate_memory", ExpGateMemory)
register_mixer("mamba2", Mamba2)
