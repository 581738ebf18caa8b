"""Causal grouped-query attention with a norm over all query heads and one over all key heads, rotary positions, a
constant sink in the softmax, and values that later layers may mix in.

For the mixer's input h, H query heads on G key heads of d numbers (values of dv)::

    q, k = norm(Wq h + bq) q_norm, norm(Wk h + bk) k_norm      one root mean square over ALL heads of q, one over all of k
    q, k = rot(q), rot(k)                             rotary positions on the first rope.dims numbers of every head
    v    = Wv h + bv,  or (1 - m) Wv h + m v_kept          v_kept: the values of an earlier layer for the same token
    out  = softmax with exp(sink_score) as one more term of the denominator, times v;   x += Wo out + bo

Kernels: one projection ``[q | k | v]`` (float32 out), ``normed_rotary`` (norms, rotation, mixing, queries out, keys and
values into the paged cache), attention over the cache, the output projection.  Heads of at most 128 numbers are cached
and attended at the width a compiled kernel has (64 or 128, the further numbers zero), so that every such size runs on
the tensor-core kernels in bfloat16; wider ones run on the kernel with run-time head sizes.
"""
from __future__ import annotations

import torch

from .. import ops as _ops
from .attention import _residual_mode, _residual_stats, attend_with_sink
from .base import CacheRequest, Mixer, TensorRequest
from .position import RotaryTable
from .registry import register_mixer


class NormedAttention(Mixer):
    graph_safe = True
    stores_branch = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        if spec.num_heads % spec.num_kv_heads != 0:
            raise ValueError("normed_attention: heads must be a multiple of kv heads")
        if spec.rope is not None and (spec.rope.dims > spec.dim or spec.rope.dims % 2):
            raise ValueError("normed_attention: the rotated numbers must be an even count within a head")
        if spec.vdim > 512:
            raise ValueError(f"normed_attention: value heads of {spec.vdim} numbers are not supported (at most 512)")
        if runtime.dtype == torch.bfloat16 and spec.hidden_size % 8 != 0:
            raise ValueError(f"normed_attention: hidden size {spec.hidden_size} is not supported in bfloat16 "
                             "(rows of 16 bytes are needed: a multiple of 8); float32 takes any size")
        self.key_width, self.value_width = self.widths(spec)
        self.v_dim = spec.num_kv_heads * spec.vdim
        rows = spec.num_heads * spec.dim + spec.num_kv_heads * spec.dim + self.v_dim
        self.fused_width = -(-rows // 8) * 8
        self.ctx_width = -(-spec.num_heads * self.value_width // 8) * 8      # whole 16 bytes for the output projection
        self.position = RotaryTable(spec.rope, runtime) if spec.rope is not None else None

    @staticmethod
    def widths(spec):
        """How wide keys and values are cached."""
        return (spec.kernel_head_dim or spec.dim), (spec.kernel_head_dim or spec.vdim)

    @classmethod
    def expected_tensors(cls, spec):
        q, k, v = spec.num_heads * spec.dim, spec.num_kv_heads * spec.dim, spec.num_kv_heads * spec.vdim
        wanted = {spec.q_weight: TensorRequest((q, spec.hidden_size)), spec.k_weight: TensorRequest((k, spec.hidden_size)),
                  spec.v_weight: TensorRequest((v, spec.hidden_size)),
                  spec.o_weight: TensorRequest((spec.hidden_size, spec.num_heads * spec.vdim))}
        for name, width in ((spec.q_bias, q), (spec.k_bias, k), (spec.v_bias, v), (spec.o_bias, spec.hidden_size)):
            if name:
                wanted[name] = TensorRequest((width,))
        if spec.q_norm:
            wanted[spec.q_norm] = TensorRequest((q,), "around_one")
        if spec.k_norm:
            wanted[spec.k_norm] = TensorRequest((k,), "around_one")
        if spec.value_mix:
            wanted[spec.value_mix] = TensorRequest((), "unit_interval")
        return wanted

    @classmethod
    def cache_request(cls, spec):
        key_width, value_width = cls.widths(spec)
        return CacheRequest("kv", spec.num_kv_heads, key_width, v_head_dim=value_width if value_width != key_width else 0)

    def bind(self, tensors):
        s, rt = self.spec, self.rt
        parts = [rt.upload(tensors[name]) for name in (s.q_weight, s.k_weight, s.v_weight)]
        missing = self.fused_width - sum(part.shape[0] for part in parts)
        if missing:                                        # (zero rows: what they produce is never read)
            parts.append(parts[0].new_zeros(missing, s.hidden_size))
        self.w_qkv = torch.cat(parts, dim=0).contiguous()
        del parts
        w_o = rt.upload(tensors[s.o_weight])
        if self.value_width != s.vdim:                     # zero columns meet the numbers that pad a head
            w_o = torch.nn.functional.pad(w_o.view(s.hidden_size, s.num_heads, s.vdim), (0, self.value_width - s.vdim))
            w_o = w_o.reshape(s.hidden_size, s.num_heads * self.value_width)
        if self.ctx_width != w_o.shape[1]:
            w_o = torch.cat([w_o, w_o.new_zeros(s.hidden_size, self.ctx_width - w_o.shape[1])], dim=1)
        self.w_o = w_o.contiguous()
        as_float = lambda name: rt.upload(tensors[name], torch.float32).reshape(-1).contiguous() if name else None
        self.q_norm, self.k_norm, self.mix = as_float(s.q_norm), as_float(s.k_norm), as_float(s.value_mix)
        self.bias = None
        if s.q_bias or s.k_bias or s.v_bias:
            widths = (s.num_heads * s.dim, s.num_kv_heads * s.dim, self.v_dim)
            self.bias = torch.cat([as_float(name) if name else torch.zeros(width, dtype=torch.float32, device=rt.device)
                                   for name, width in zip((s.q_bias, s.k_bias, s.v_bias), widths)]).contiguous()
        self.output_bias = as_float(s.o_bias)
        self.sink = None
        if s.sink_score is not None:
            self.sink = torch.full((s.num_heads,), float(s.sink_score), dtype=torch.float32, device=rt.device)

    def forward(self, step, h, x, cache_entry, writes_cache=True):
        s, rt = self.spec, self.rt
        ops = rt.kernels()
        n = h.shape[0]
        fused = rt.workspace.get("qkv", (n, self.fused_width), torch.float32)
        ops.linear(h, self.w_qkv, fused, _ops.MODE_STORE_F32)
        k_cache, v_cache = step.cache.entry_kv(cache_entry)
        table = step.block_tables[step.cache.entry_group_index(cache_entry)]
        keep = first = None
        if s.keeps_values:
            keep = rt.workspace.get("kept_values", (n, self.v_dim), torch.float32)
            step.scratch["kept_values"] = keep
        if self.mix is not None:
            first = step.scratch.get("kept_values")
            if first is None or tuple(first.shape) != (n, self.v_dim):
                raise ValueError("normed_attention: no earlier layer has kept values of this layer's size")
        q = rt.workspace.get("q", (n, s.num_heads * self.key_width), rt.dtype)
        ops.normed_rotary(fused, q, k_cache, v_cache, step.positions, step.token_seq, table, s.num_heads, s.num_kv_heads,
                          s.dim, s.vdim, step.cache.block_size, eps=s.eps, q_weight=self.q_norm, k_weight=self.k_norm,
                          cos_sin=self.position.fusion_table(step.max_ctx) if self.position is not None else None,
                          rotated=s.rope.dims if s.rope is not None else 0,
                          interleaved=bool(s.rope is not None and s.rope.interleaved), mix=self.mix, first=first, keep=keep,
                          write_kv=writes_cache, bias=self.bias)
        ctx = rt.workspace.get("attn_ctx", (n, self.ctx_width), rt.dtype)
        attend_with_sink(step, rt, q, ctx, k_cache, v_cache, table, s.num_heads, s.num_kv_heads, self.key_width,
                         self.value_width, s.scale, sink=self.sink)
        ops.linear(ctx, self.w_o, x, _residual_mode(step), stats=_residual_stats(step))
        if self.output_bias is not None and not self.leaves_output_bias:
            ops.add_biased(x, None, self.output_bias, 1.0)


register_mixer("normed_attention", NormedAttention)
