"""A stand-in for the CUDA kernel library, used only by CPU tests of the engine's
bookkeeping (batch packing, cache slots and block tables, the order of parts).

It has the call signatures of ``stratakv_b200.ops.Kernels`` and computes each
call with plain torch on whatever device the tensors are on.  The package never
imports it; the product path has no CPU backend.
"""
from __future__ import annotations

import torch

MODE_STORE, MODE_STORE_F32, MODE_ADD_F32, MODE_GATED = 0, 1, 2, 3
MODE_ACT = 5
ACTIVATIONS = {"silu": lambda z: z * torch.sigmoid(z), "relu2": lambda z: torch.relu(z) ** 2,
               "gelu_tanh": lambda z: torch.nn.functional.gelu(z, approximate="tanh")}


class DoubleKernels:
    def __init__(self, dtype, head_dim):
        self.dtype = dtype
        self.head_dim = head_dim
        self.calls = []

    def embed(self, table, ids, out, flag=None, stats=None):
        self.calls.append("embed")
        out.copy_(table[ids.long()].float())

    def rmsnorm(self, x, gamma, eps, out, rows=None, groups=1):
        self.calls.append("rmsnorm")
        src = x if rows is None else x[rows.long()]
        if groups > 1:
            parts = src.view(src.shape[0], groups, -1)
            parts = parts / torch.sqrt((parts * parts).mean(dim=-1, keepdim=True) + eps)
            out.copy_((parts.reshape(src.shape) * gamma).to(out.dtype))
            return
        inv = 1.0 / torch.sqrt((src * src).mean(dim=-1, keepdim=True) + eps)
        out.copy_((src * inv * gamma).to(out.dtype))

    def linear(self, a, w, out, mode=MODE_STORE, activation="silu", flag=None, stats=None, activation_param=0.0):
        self.calls.append("linear")
        result = a.float() @ w.float().T
        if mode == MODE_GATED:
            tiles = result.view(result.shape[0], -1, 2, 8)
            gate, up = tiles[:, :, 0, :], tiles[:, :, 1, :]
            if activation == "swiglu_clamp":
                gate = gate.clamp(max=activation_param)
                product = gate * torch.sigmoid(1.702 * gate) * (up.clamp(-activation_param, activation_param) + 1.0)
            else:
                product = ACTIVATIONS[activation](gate) * up
            out.copy_(product.reshape(result.shape[0], -1).to(out.dtype))
        elif mode == MODE_ADD_F32:
            out.add_(result)
        elif mode == MODE_ACT:
            out.copy_(ACTIVATIONS[activation](result).to(out.dtype))
        else:
            out.copy_(result.to(out.dtype))

    def rope_kv_write(self, qkv, cos_sin, positions, token_seq, block_table, q_out, k_cache, v_cache,
                      num_heads, num_kv_heads, head_dim, block_size, write_kv):
        self.calls.append("rope_kv_write")
        n = qkv.shape[0]
        q_dim, kv_dim, half = num_heads * head_dim, num_kv_heads * head_dim, head_dim // 2
        q = qkv[:, :q_dim].view(n, num_heads, head_dim)
        k = qkv[:, q_dim:q_dim + kv_dim].view(n, num_kv_heads, head_dim)
        v = qkv[:, q_dim + kv_dim:].view(n, num_kv_heads, head_dim)

        def rotate(x):
            if cos_sin is None:
                return x
            cs = cos_sin[positions.long()]                        # [n, half, 2]
            c, s = cs[:, None, :, 0], cs[:, None, :, 1]
            x1, x2 = x[..., :half], x[..., half:]
            return torch.cat([x1 * c - x2 * s, x1 * s + x2 * c], dim=-1)

        q_out.copy_(rotate(q).reshape(n, q_dim).to(q_out.dtype))
        if write_kv:
            k = rotate(k)
            for t in range(n):
                pos = int(positions[t])
                block = int(block_table[int(token_seq[t]), pos // block_size])
                k_cache[block, :, pos % block_size, :] = k[t].to(k_cache.dtype)
                v_cache[block, :, pos % block_size, :] = v[t].to(v_cache.dtype)

    def attention(self, q, k_cache, v_cache, block_table, positions, token_seq, out, num_heads,
                  num_kv_heads, head_dim, block_size, scale, window=0):
        self.calls.append("attention")
        n = q.shape[0]
        group = num_heads // num_kv_heads
        qh = q.view(n, num_heads, head_dim).float()
        result = torch.zeros(n, num_heads, head_dim)
        for t in range(n):
            pos, seq = int(positions[t]), int(token_seq[t])
            lo = max(0, pos - window + 1) if window > 0 else 0
            keys = torch.stack([k_cache[int(block_table[seq, j // block_size]), :, j % block_size, :]
                                for j in range(lo, pos + 1)]).float()       # [ctx, kv_heads, d]
            values = torch.stack([v_cache[int(block_table[seq, j // block_size]), :, j % block_size, :]
                                  for j in range(lo, pos + 1)]).float()
            for h in range(num_heads):
                g = h // group
                weights = torch.softmax((keys[:, g, :] @ qh[t, h]) * scale, dim=0)
                result[t, h] = weights @ values[:, g, :]
        out.copy_(result.reshape(n, num_heads * head_dim).to(out.dtype))

    def embed_sum(self, table, ids, out, positions, token_seq, cu_q, slot_ids, flag=None, pair_table=None,
                  last_ids=None, mul_prev=0, mul_cur=0, position_table=None, position_scale=1.0, stats=None):
        self.calls.append("embed_sum")
        x = table[ids.long()].float()
        if pair_table is not None:
            buckets = pair_table.shape[0] - 1
            for t in range(ids.numel()):
                seq, pos, row = int(token_seq[t]), int(positions[t]), buckets
                if pos > 0:
                    slot = int(slot_ids[seq])
                    previous = int(ids[t - 1]) if t > int(cu_q[seq]) else int(last_ids[2 * slot + ((pos - 1) & 1)])
                    row = (previous * mul_prev + int(ids[t]) * mul_cur) % buckets
                x[t] += pair_table[row].float()
            for seq in range(slot_ids.numel()):
                last = int(cu_q[seq + 1]) - 1
                last_ids[2 * int(slot_ids[seq]) + (int(positions[last]) & 1)] = ids[last]
        if position_table is not None:
            x += position_table[positions.long()].float() * position_scale
        out.copy_(x)

    def qkv_finish(self, qkv, q_out, k_cache, v_cache, positions, token_seq, block_table, num_heads, num_kv_heads,
                   dim, vdim, block_size, q_bias=None, k_bias=None, v_bias=None, value_norm_eps=None, write_kv=True,
                   q_norm=False, k_norm=False, qk_norm_eps=0.0, k_norm_weight=None, q_temperature=None, key_dim=0):
        self.calls.append("qkv_finish")
        n = qkv.shape[0]
        key_dim = key_dim or dim
        unit = lambda x, eps: x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
        a = num_heads * dim
        q = qkv[:, :a]
        q = (q + q_bias if q_bias is not None else q).view(n, num_heads, dim)
        if q_norm:
            q = unit(q, qk_norm_eps)
        if q_temperature is not None:
            coef, every = q_temperature
            steps = torch.div(positions.long() + 1, every, rounding_mode="floor").float()
            q = q * (1.0 + coef * torch.log(steps + 1.0))[:, None, None]
        q_out.copy_(q.reshape(n, a).to(q_out.dtype))
        if not write_kv:
            return
        b = a + num_kv_heads * key_dim
        k = qkv[:, a:b]
        k = (k + k_bias if k_bias is not None else k).view(n, num_kv_heads, key_dim)
        if k_norm:
            k = unit(k, qk_norm_eps)
            if k_norm_weight is not None:
                k = k * k_norm_weight.view(num_kv_heads, key_dim)
        v = None
        if vdim > 0:
            v = qkv[:, b:b + num_kv_heads * vdim]
            v = (v + v_bias if v_bias is not None else v).view(n, num_kv_heads, vdim)
            if value_norm_eps is not None:
                v = unit(v, value_norm_eps)
        for t in range(n):
            pos = int(positions[t])
            block = int(block_table[int(token_seq[t]), pos // block_size])
            k_cache[block, :, pos % block_size, :] = k[t].to(k_cache.dtype)
            if v is not None:
                v_cache[block, :, pos % block_size, :] = v[t].to(v_cache.dtype)

    def attention_general(self, q, k_cache, v_cache, block_table, positions, token_seq, out, num_heads, num_kv_heads,
                          dim, vdim, block_size, scale, window=0, r1=None, r2=None, gate=None, gate_stride=0,
                          softcap=0.0, gate_per_element=False, sink=None, value_stride=0, splits=1, scratch_o=None, scratch_ml=None):
        self.calls.append("attention_general")
        n = q.shape[0]
        group = num_heads // num_kv_heads
        qh = q.view(n, num_heads, dim).float()
        out.zero_()
        for t in range(n):
            pos, seq = int(positions[t]), int(token_seq[t])
            lo = max(0, pos - window + 1) if window > 0 else 0
            where = [(int(block_table[seq, j // block_size]), j % block_size) for j in range(lo, pos + 1)]
            keys = torch.stack([k_cache[b, :, r, :] for b, r in where]).float()
            values = torch.stack([v_cache[b, :, r, :vdim] for b, r in where]).float()
            distance = torch.arange(pos - lo, -1, -1, dtype=torch.float32)
            for h in range(num_heads):
                score = (keys[:, h // group, :] @ qh[t, h]) * scale
                if r1 is not None:
                    score = score - r1[h] * torch.log1p(r2[h] * distance)
                if softcap > 0.0:
                    score = softcap * torch.tanh(score / softcap)
                if sink is not None:                # one more term in the denominator, with no value
                    result = torch.softmax(torch.cat([score, sink[h].view(1)]), dim=0)[:-1] @ values[:, h // group, :]
                else:
                    result = torch.softmax(score, dim=0) @ values[:, h // group, :]
                if gate is not None and gate_per_element:
                    result = result * torch.sigmoid(gate[t, h * vdim:(h + 1) * vdim])
                elif gate is not None:
                    result = result * torch.sigmoid(gate[t, h])
                out[t, h * vdim:(h + 1) * vdim] = result.to(out.dtype)

    def rmsnorm_add(self, y, gamma, eps, x, next_gamma=None, next_eps=0.0, next_out=None):
        self.calls.append("rmsnorm_add")
        x.add_(y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps) * gamma)
        if next_out is not None:
            normed = x if next_gamma is None else x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + next_eps) * next_gamma
            next_out.copy_(normed.to(next_out.dtype))

    def token_side(self, x, ids, table, offset, dim, gate_w, proj_t, norm_w, eps, next_gamma=None, next_eps=0.0,
                   next_out=None, branch=None, post_gamma=None, post_eps=0.0):
        self.calls.append("token_side")
        if branch is not None:
            self.rmsnorm_add(branch, post_gamma, post_eps, x)
        e = table[ids.long()][:, offset:offset + dim].float()
        g = torch.nn.functional.gelu(x @ gate_w.float().T, approximate="tanh") * e
        self.rmsnorm_add(g @ proj_t.float(), norm_w, eps, x, next_gamma, next_eps, next_out)

    def headwise_linear(self, x, w, out, heads, zero_pad=False, out_head_stride=0):
        self.calls.append("headwise_linear")
        n, out_dim, in_dim = x.shape[0], w.shape[1], w.shape[2]
        parts = x[:, :heads * in_dim].float().view(n, heads, in_dim)
        if zero_pad:
            out.zero_()
        result = torch.einsum("thi,hoi->tho", parts, w.float()).to(out.dtype)
        if out_head_stride and out_head_stride != out_dim:
            for h in range(heads):
                out[:, h * out_head_stride:h * out_head_stride + out_dim] = result[:, h]
        else:
            out[:, :heads * out_dim] = result.reshape(n, heads * out_dim)

    def stream_mix(self, streams, count, source=None, branch=None, mix=None, write=None, read=None, gamma=None,
                   eps=0.0, normed_out=None, sum_out=None):
        self.calls.append("stream_mix")
        old = streams.clone() if source is None else source[None].repeat(count, 1, 1)
        if branch is not None:
            old = torch.einsum("sr,stw->rtw", mix.view(count, count), old) + write[:, None, None] * branch[None]
            streams.copy_(old)
        if normed_out is not None:
            u = torch.einsum("s,stw->tw", read, old)
            normed_out.copy_((u / torch.sqrt((u * u).mean(dim=-1, keepdim=True) + eps) * gamma).to(normed_out.dtype))
        if sum_out is not None:
            sum_out.copy_(old.sum(dim=0))

    def retention_scratch(self, n_seqs, max_q_len, heads, dim, vdim):
        return 0

    @staticmethod
    def _turn(x, cos_sin, positions, rotated):
        """x [n, ..., width]: the first ``rotated`` numbers of the last axis turned by the table's angles."""
        if cos_sin is None or rotated == 0:
            return x
        half = rotated // 2
        cs = cos_sin[positions.long()]
        shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
        c, s = cs[:, :, 0].view(shape), cs[:, :, 1].view(shape)
        u, v = x[..., :half], x[..., half:rotated]
        return torch.cat([u * c - v * s, v * c + u * s, x[..., rotated:]], dim=-1)

    def retention(self, fused, cos_sin, rotated, decay, eps, out, state, step_meta, heads, dim, vdim, max_q_len, scratch=None):
        self.calls.append("retention")
        positions, token_seq, cu_q, slot_ids = step_meta
        n = fused.shape[0]
        a, b = heads * dim, heads * vdim
        q = self._turn(fused[:, :a].view(n, heads, dim), cos_sin, positions, rotated)
        k = self._turn(fused[:, a:2 * a].view(n, heads, dim), cos_sin, positions, rotated) * dim ** -0.5
        v = fused[:, 2 * a:2 * a + b].view(n, heads, vdim)
        gate = fused[:, 2 * a + b:2 * a + 2 * b]
        size = heads * dim * vdim
        out.zero_()
        for s in range(slot_ids.numel()):
            first, last = int(cu_q[s]), int(cu_q[s + 1]) - 1
            row = state[int(slot_ids[s])]
            p_first = int(positions[first])
            S = (row[((p_first - 1) & 1) * size:][:size].clone().view(heads, dim, vdim) if p_first > 0
                 else torch.zeros(heads, dim, vdim))
            for t in range(first, last + 1):
                S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
                o = torch.einsum("hde,hd->he", S, q[t])
                o = o / torch.sqrt((o * o).mean(dim=-1, keepdim=True) + eps)
                out[t, :b] = (o.reshape(b) * gate[t] * torch.sigmoid(gate[t])).to(out.dtype)
            row[((p_first + last - first) & 1) * size:][:size] = S.reshape(size)

    def latent_finish(self, fused, q_plain, q_folded, cache, positions, token_seq, block_table, heads, dim, rope_dim,
                      latent_dim, block_size, rotation=None, rotated=0, latent_offset=0, latent_gamma=None, eps=0.0,
                      write_cache=True, q_whole=None):
        self.calls.append("latent_finish")
        assert q_whole is None, "whole query heads are the bfloat16 prompt path's"
        n, key_dim = fused.shape[0], latent_dim + rope_dim
        q = fused[:, :heads * (dim + rope_dim)].view(n, heads, dim + rope_dim)
        q_plain.copy_(q[:, :, :dim].reshape(n, heads * dim).to(q_plain.dtype))
        if rope_dim:
            turned = self._turn(q[:, :, dim:], rotation, positions, rotated)
            q_folded.view(n, heads, key_dim)[:, :, latent_dim:] = turned.to(q_folded.dtype)
        if not write_cache:
            return
        c = fused[:, latent_offset:latent_offset + latent_dim]
        c = c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * latent_gamma
        rows = torch.cat([c, self._turn(fused[:, latent_offset + latent_dim:latent_offset + key_dim], rotation, positions,
                                        rotated)], dim=-1)
        for t in range(n):
            pos = int(positions[t])
            block = int(block_table[int(token_seq[t]), pos // block_size])
            cache[block, 0, pos % block_size, :] = rows[t].to(cache.dtype)

    def route_tokens(self, h, router_w, correction, top, scale, renormalize, chosen, weights, shared_gate_weight=None,
                     shared_gate_out=None, softmax=False, groups=0, keep=0, renorm_eps=0.0):
        self.calls.append("route_tokens")
        logits = h.float() @ router_w.float().T
        s = torch.softmax(logits, dim=-1) if softmax else torch.sigmoid(logits)
        choice = s + correction if correction is not None else s
        if groups > 1:
            size = s.shape[1] // groups
            best = choice.view(-1, groups, size).max(dim=-1).values
            kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(keep, dim=-1).indices, True)
            choice = choice.masked_fill(~kept.repeat_interleave(size, dim=1), -float("inf"))
        picked = torch.topk(choice, top, dim=-1).indices
        w = torch.gather(s, 1, picked)
        if renormalize:
            w = w / (w.sum(dim=-1, keepdim=True) + renorm_eps)
        chosen.copy_(picked.to(torch.int32))
        weights.copy_(w * scale)
        if shared_gate_out is not None:
            shared_gate_out.copy_(torch.sigmoid(h.float() @ shared_gate_weight.float()))

    def sort_by_expert(self, chosen, experts, offsets, order, place):
        self.calls.append("sort_by_expert")
        flat = chosen.reshape(-1).long()
        sorted_pairs = torch.argsort(flat, stable=True)
        counts = torch.bincount(flat, minlength=experts)
        offsets[0] = 0
        offsets[1:] = torch.cumsum(counts, 0).to(torch.int32)
        order.copy_((sorted_pairs // chosen.shape[1]).to(torch.int32))
        place.view(-1)[sorted_pairs] = torch.arange(flat.numel(), dtype=torch.int32)

    def expert_rows_sorted_first(self, hidden):
        return False

    def expert_linear(self, a, w, offsets, out, rows=None, activation=None, flag=None, gated=False,
                      activation_param=0.0):
        self.calls.append("expert_linear")
        for e in range(w.shape[0]):
            lo, hi = int(offsets[e]), int(offsets[e + 1])
            if hi == lo:
                continue
            src = a[rows[lo:hi].long()] if rows is not None else a[lo:hi]
            result = src.float() @ w[e].float().T
            if gated:                               # tiles of 8 gate rows and their 8 up rows
                tiles = result.view(result.shape[0], -1, 2, 8)
                gate, up = tiles[:, :, 0], tiles[:, :, 1]
                if activation == "swiglu_clamp":
                    gate = gate.clamp(max=activation_param)
                    product = gate * torch.sigmoid(1.702 * gate) * (up.clamp(-activation_param, activation_param) + 1.0)
                else:
                    product = ACTIVATIONS[activation](gate) * up
                result = product.reshape(result.shape[0], -1)
            elif activation is not None:
                result = ACTIVATIONS[activation](result)
            out[lo:hi] = result.to(out.dtype)

    def scatter_rows(self, a, place, weights, out):
        self.calls.append("scatter_rows")
        rows = (a.float()[:, None, :] * weights[:, :, None]).to(out.dtype)
        out[place.reshape(-1).long()] = rows.reshape(-1, a.shape[1])

    def combine_experts(self, results, place, weights, shared, share, x, add=True):
        self.calls.append("combine_experts")
        total = results[place.long()]
        total = (total * weights[:, :, None] if weights is not None else total).sum(dim=1)
        if shared is not None:
            total = total + (shared * share[:, None] if share is not None else shared)
        if add:
            x.add_(total)
        else:
            x.copy_(total)

    def rglru_conv(self, yx, x_offset, x_bias, conv_w, conv_b, u, step_meta, state):
        self.calls.append("rglru_conv")
        positions, token_seq, cu_q, slot_ids = step_meta
        channels, taps = conv_w.shape
        for t in range(u.shape[0]):
            p, s = int(positions[t]), int(token_seq[t])
            ring = state[int(slot_ids[s]), 2 * channels:(2 + taps) * channels].view(taps, channels)
            total = conv_b.clone()
            for k in range(taps):
                back = taps - 1 - k
                if p - back < 0:
                    continue
                inside = t - back >= int(cu_q[s])
                value = yx[t - back, x_offset:x_offset + channels] + x_bias if inside else ring[(p - back) % taps]
                total = total + conv_w[:, k] * value
            u[t] = total

    def rglru_rate(self, lam, rate):
        rate.copy_(8.0 * torch.nn.functional.softplus(lam))
        return rate

    def rglru_gates(self, gates, u, yx, y_bias, r_bias, i_bias, rate, part):
        self.calls.append("rglru_gates")
        n, channels = u.shape
        pairs = gates.view(n, channels // part, 2, part)
        r = torch.sigmoid(pairs[:, :, 0, :] + r_bias.view(-1, part))
        i = torch.sigmoid(pairs[:, :, 1, :] + i_bias.view(-1, part))
        a = torch.exp(-r * rate.view(-1, part))
        driven = torch.sqrt(1.0 - a * a) * i * u.view(n, -1, part)
        pairs[:, :, 0, :] = a
        pairs[:, :, 1, :] = driven
        yx[:, :channels] = torch.nn.functional.gelu(yx[:, :channels] + y_bias, approximate="tanh")

    def rglru_scan_scratch(self, n_seqs, max_q_len, channels):
        return 0

    def rglru_scan(self, gates, yx, x_offset, x_bias, out, part, taps, step_meta, state, max_q_len=0, summary=None):
        self.calls.append("rglru_scan")
        positions, token_seq, cu_q, slot_ids = step_meta
        n, channels = gates.shape[0], gates.shape[1] // 2
        pairs = gates.view(n, channels // part, 2, part)
        for s in range(slot_ids.numel()):
            first, last = int(cu_q[s]), int(cu_q[s + 1]) - 1
            row = state[int(slot_ids[s])]
            p_first = int(positions[first])
            S = row[((p_first - 1) & 1) * channels:][:channels].clone() if p_first > 0 else torch.zeros(channels)
            for t in range(first, last + 1):
                S = pairs[t, :, 0, :].reshape(-1) * S + pairs[t, :, 1, :].reshape(-1)
                out[t, :channels] = (S * yx[t, :channels]).to(out.dtype)
            p_last = p_first + last - first
            row[(p_last & 1) * channels:][:channels] = S
            ring = row[2 * channels:(2 + taps) * channels].view(taps, channels)
            for back in range(min(taps, last - first + 1)):
                ring[(p_last - back) % taps] = yx[last - back, x_offset:x_offset + channels] + x_bias

    def add_scaled(self, out, other, factor):
        self.calls.append("add_scaled")
        out.add_(other * factor)

    def add_biased(self, out, other, bias, factor):
        self.calls.append("add_biased")
        out.add_(((other if other is not None else 0.0) + bias) * factor)

    def softcap_inplace(self, x, cap):
        self.calls.append("softcap_inplace")
        x.copy_(cap * torch.tanh(x / cap))

    def projection_norm(self, rows, eps, segments):
        self.calls.append("projection_norm")
        for offset, width, bias, weight in segments:
            x = rows[:, offset:offset + width] + (bias if bias is not None else 0.0)
            rows[:, offset:offset + width] = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight

    def short_conv_rotary(self, rows, bias, conv_w, taps, cos_sin, rotated, interleaved, block_table, q_out, k_cache,
                          v_cache, num_heads, num_kv_heads, dim, block_size, write_kv, step_meta, state, state_offset=0):
        self.calls.append("short_conv_rotary")
        positions, token_seq, cu_q, slot_ids = step_meta
        n, channels = rows.shape[0], (num_heads + num_kv_heads) * dim
        u = rows[:, :channels] + (bias if bias is not None else 0.0)
        y = torch.zeros(n, channels)
        for t in range(n):
            seq, p = int(token_seq[t]), int(positions[t])
            first = int(cu_q[seq])
            if taps == 0:
                y[t] = u[t]
                continue
            ring = (state[int(slot_ids[seq])][state_offset:state_offset + taps * channels].view(taps, channels)
                    if taps > 1 else None)
            for j in range(taps):
                back = taps - 1 - j
                if p - back >= 0:
                    y[t] += conv_w[:, j] * (u[t - back] if t - back >= first else ring[(p - back) % taps])
        heads = y.view(n, num_heads + num_kv_heads, dim)
        turned = heads.clone()
        if rotated:
            cs = cos_sin[positions.long()]                            # [n, rotated / 2, 2]
            c, sn = cs[:, None, :, 0], cs[:, None, :, 1]
            if interleaved:
                a, b = heads[..., 0:rotated:2], heads[..., 1:rotated:2]
                turned[..., 0:rotated:2], turned[..., 1:rotated:2] = a * c - b * sn, b * c + a * sn
            else:
                half = rotated // 2
                a, b = heads[..., :half], heads[..., half:rotated]
                turned[..., :half], turned[..., half:rotated] = a * c - b * sn, b * c + a * sn
        q_out.copy_(turned[:, :num_heads].reshape(n, num_heads * dim).to(q_out.dtype))
        if not write_kv:
            return
        for t in range(n):
            pos = int(positions[t])
            block = int(block_table[int(token_seq[t]), pos // block_size])
            k_cache[block, :, pos % block_size, :] = turned[t, num_heads:].to(k_cache.dtype)
            if v_cache is not None:
                v_cache[block, :, pos % block_size, :] = heads[t, num_heads:].to(v_cache.dtype)

    def short_conv_remember(self, rows, bias, channels, taps, n_seqs, step_meta, state, state_offset=0):
        self.calls.append("short_conv_remember")
        if taps <= 1:
            return
        positions, token_seq, cu_q, slot_ids = step_meta
        for seq in range(n_seqs):
            first, end = int(cu_q[seq]), int(cu_q[seq + 1])
            ring = state[int(slot_ids[seq])][state_offset:state_offset + taps * channels].view(taps, channels)
            for t in range(max(first, end - (taps - 1)), end):
                ring[int(positions[t]) % taps] = rows[t, :channels] + (bias if bias is not None else 0.0)

    def time_mix_state_floats(self, hidden, heads, dim):
        return 2 * heads * dim * dim + 2 * hidden

    def token_shift_mix(self, h, mu, mixes, heads, dim, step_meta, state, state_offset=0):
        self.calls.append("token_shift_mix")
        positions, token_seq, cu_q, slot_ids = step_meta
        hidden = h.shape[1]
        base = state_offset + 2 * heads * dim * dim
        for t in range(h.shape[0]):
            seq, p = int(token_seq[t]), int(positions[t])
            if t > int(cu_q[seq]):
                before = h[t - 1].float()
            elif p > 0:
                before = state[int(slot_ids[seq])][base + ((p - 1) & 1) * hidden:][:hidden]
            else:
                before = torch.zeros(hidden)
            now = h[t].float()
            for m in range(mixes.shape[0]):
                mixes[m, t] = (now + (before - now) * mu[m]).to(mixes.dtype)

    def time_mix_decay(self, lora, rank, w2, w0, decay):
        self.calls.append("time_mix_decay")
        decay.copy_(torch.exp(-torch.exp(torch.tanh(lora[:, :rank]) @ w2.float() + w0)))       # (w2 is [rank, channels])

    def time_mix_scan(self, r, k, v, decay, bonus, out, h, n_seqs, heads, dim, step_meta, state, state_offset=0):
        self.calls.append("time_mix_scan")
        positions, token_seq, cu_q, slot_ids = step_meta
        hidden, size = h.shape[1], heads * dim * dim
        u = bonus.view(heads, dim)
        for seq in range(n_seqs):
            first, end = int(cu_q[seq]), int(cu_q[seq + 1])
            if end <= first:
                continue
            row = state[int(slot_ids[seq])]
            p0 = int(positions[first])
            S = (row[state_offset + ((p0 - 1) & 1) * size:][:size].clone().view(heads, dim, dim) if p0 > 0
                 else torch.zeros(heads, dim, dim))
            for t in range(first, end):
                kv = k[t].view(heads, dim)[:, :, None] * v[t].view(heads, dim)[:, None, :]
                out[t] = torch.einsum("hi,hij->hj", r[t].view(heads, dim), S + u[:, :, None] * kv).reshape(-1)
                S = decay[t].view(heads, dim)[:, :, None] * S + kv
            last = p0 + end - first - 1
            row[state_offset + (last & 1) * size:][:size] = S.reshape(size)
            row[state_offset + 2 * size + (last & 1) * hidden:][:hidden] = h[end - 1].float()

    def time_mix_finish(self, o, gate, norm, eps, out_scale, out, heads, dim):
        self.calls.append("time_mix_finish")
        n = o.shape[0]
        heads_o = o.view(n, heads, dim)
        unit = heads_o / torch.sqrt((heads_o * heads_o).mean(dim=-1, keepdim=True) + eps)
        out.zero_()
        out[:, :heads * dim] = (unit.reshape(n, -1) * norm * gate * torch.sigmoid(gate) * out_scale).to(out.dtype)

    def normed_rotary(self, rows, q_out, k_cache, v_cache, positions, token_seq, block_table, num_heads, num_kv_heads, dim,
                      vdim, block_size, eps=0.0, q_weight=None, k_weight=None, cos_sin=None, rotated=0, interleaved=False,
                      mix=None, first=None, keep=None, write_kv=True, bias=None):
        self.calls.append("normed_rotary")
        n = rows.shape[0]
        if bias is not None:
            rows = rows[:, :bias.numel()] + bias
        a, b, c = num_heads * dim, num_kv_heads * dim, num_kv_heads * vdim

        def turned(x, weight, heads):
            if weight is not None:
                x = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight
            x = x.view(n, heads, dim)
            out = x.clone()
            if rotated:
                cs = cos_sin[positions.long()]
                co, sn = cs[:, None, :, 0], cs[:, None, :, 1]
                even, odd = (slice(0, rotated, 2), slice(1, rotated, 2)) if interleaved else \
                    (slice(0, rotated // 2), slice(rotated // 2, rotated))
                out[..., even] = x[..., even] * co - x[..., odd] * sn
                out[..., odd] = x[..., odd] * co + x[..., even] * sn
            return out

        q, k = turned(rows[:, :a], q_weight, num_heads), turned(rows[:, a:a + b], k_weight, num_kv_heads)
        v = rows[:, a + b:a + b + c]
        if keep is not None:
            keep.copy_(v)
        if mix is not None:
            v = (1.0 - mix) * v + mix * first
        v = v.reshape(n, num_kv_heads, vdim)
        wide = q_out.view(n, num_heads, k_cache.shape[-1])
        wide.zero_()
        wide[..., :dim] = q.to(wide.dtype)
        if not write_kv:
            return
        for t in range(n):
            pos = int(positions[t])
            block = int(block_table[int(token_seq[t]), pos // block_size])
            for cache, value in ((k_cache, k[t]), (v_cache, v[t])):
                row = cache[block, :, pos % block_size, :]
                row.zero_()
                row[:, :value.shape[-1]] = value.to(cache.dtype)

    def linear_state_scratch(self, n_seqs, max_q_len, heads, dim, vdim, with_floor=False):
        return 0

    def linear_state(self, rows, q_at, k_at, v_at, out, state, step_meta, heads, groups, dim, vdim, max_q_len, decay=None,
                     log_decay=None, key_scale=None, skip=None, silu=False, scratch=None, state_offset=0, out_scale=1.0,
                     floor=None, floor_eps=0.0):
        self.calls.append("linear_state")
        positions, token_seq, cu_q, slot_ids = step_meta
        n = rows.shape[0]
        act = ACTIVATIONS["silu"] if silu else (lambda z: z)
        spread = lambda x: x.repeat_interleave(heads // groups, dim=1)
        q = spread(act(rows[:, q_at:q_at + groups * dim]).view(n, groups, dim))
        k = spread(act(rows[:, k_at:k_at + groups * dim]).view(n, groups, dim))
        v = act(rows[:, v_at:v_at + heads * vdim]).view(n, heads, vdim)
        if key_scale is not None:
            k = k * key_scale[:, :, None]
        d = decay.expand(n, heads) if decay is not None else torch.exp(log_decay)
        size = heads * dim * vdim
        half = size + (heads * dim if floor is not None else 0)
        for s in range(slot_ids.numel()):
            first, last = int(cu_q[s]), int(cu_q[s + 1]) - 1
            row = state[int(slot_ids[s])][state_offset:]
            p_first = int(positions[first])
            before = row[((p_first - 1) & 1) * half:][:half].clone() if p_first > 0 else torch.zeros(half)
            S, sums = before[:size].view(heads, dim, vdim), before[size:].view(-1, dim)
            for t in range(first, last + 1):
                S = d[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
                o = torch.einsum("hnp,hn->hp", S, q[t]) * out_scale
                if floor is not None:
                    sums = d[t][:, None] * sums + k[t]
                    dot = (sums * q[t]).sum(dim=-1).abs() * out_scale
                    o = o / (torch.maximum(dot, floor[t]) + floor_eps)[:, None]
                out[t] = (o + skip[:, None] * v[t] if skip is not None else o).reshape(-1)
            after = row[((p_first + last - first) & 1) * half:]
            after[:size] = S.reshape(-1)
            after[size:half] = sums.reshape(-1)

    def conv_silu(self, rows, conv_w, conv_b, out, step_meta, state, ring_offset=0):
        self.calls.append("conv_silu")
        positions, token_seq, cu_q, slot_ids = step_meta
        channels, taps = conv_w.shape
        for t in range(rows.shape[0]):
            seq, p = int(token_seq[t]), int(positions[t])
            first = int(cu_q[seq])
            y = conv_b.clone() if conv_b is not None else torch.zeros(channels)
            for j in range(taps):
                back = taps - 1 - j
                if p - back < 0:
                    continue
                if t - back >= first:
                    u = rows[t - back, :channels]
                else:
                    ring = state[int(slot_ids[seq])][ring_offset:ring_offset + taps * channels].view(taps, channels)
                    u = ring[(p - back) % taps]
                y = y + conv_w[:, j] * u
            out[t] = ACTIVATIONS["silu"](y)

    def step_sizes(self, rows, dt_at, dt_bias, a_log, dt, log_decay):
        self.calls.append("step_sizes")
        dt.copy_(torch.nn.functional.softplus(rows[:, dt_at:dt_at + dt.shape[1]] + dt_bias))
        log_decay.copy_(-torch.exp(a_log) * dt)

    def mamba2_step(self, rows, conv_w, conv_b, dt_at, dt_bias, a_log, skip, out, state, step_meta, heads, groups, dim, vdim,
                    state_offset, ring_offset):
        self.calls.append("mamba2_step")
        n, (channels, taps) = rows.shape[0], conv_w.shape
        convolved = torch.zeros(n, channels)
        self.conv_silu(rows, conv_w, conv_b, convolved, step_meta, state, ring_offset)
        dt, log_decay = torch.zeros(n, heads), torch.zeros(n, heads)
        self.step_sizes(rows, dt_at, dt_bias, a_log, dt, log_decay)
        inner = heads * vdim
        self.linear_state(convolved, inner + groups * dim, inner, 0, out, state, step_meta, heads, groups, dim, vdim, 1,
                          log_decay=log_decay, key_scale=dt, skip=skip, state_offset=state_offset)
        self.short_conv_remember(rows, None, channels, taps, n, step_meta, state, ring_offset)

    def gated_norm(self, y, gate, gate_stride, weight, groups, eps, mode, out):
        self.calls.append("gated_norm")
        n, width = y.shape
        g = gate[:, :width]
        x = y * ACTIVATIONS["silu"](g) if mode == 1 else y
        parts = x.view(n, groups, -1)
        x = (parts / torch.sqrt((parts * parts).mean(dim=-1, keepdim=True) + eps)).reshape(n, width) * weight
        out.zero_()
        out[:, :width] = (x * {0: torch.sigmoid(g), 1: 1.0, 2: ACTIVATIONS["silu"](g)}[mode]).to(out.dtype)

    def exp_gates(self, rows, input_at, forget_at, input_bias, forget_bias, cap, log_decay, key_scale, floor, step_meta, state,
                  m_offset=0):
        self.calls.append("exp_gates")
        positions, token_seq, cu_q, slot_ids = step_meta
        heads = input_bias.numel()
        i = cap * torch.tanh((rows[:, input_at:input_at + heads] + input_bias) / cap)
        f = torch.nn.functional.logsigmoid(cap * torch.tanh((rows[:, forget_at:forget_at + heads] + forget_bias) / cap))
        for s in range(slot_ids.numel()):
            first, end = int(cu_q[s]), int(cu_q[s + 1])
            kept = state[int(slot_ids[s])][m_offset:m_offset + 2 * heads].view(2, heads)
            p = int(positions[first])
            m = kept[(p - 1) & 1].clone() if p > 0 else torch.zeros(heads)
            for t in range(first, end):
                top = torch.maximum(f[t] + m, i[t])
                log_decay[t], key_scale[t], floor[t] = f[t] + m - top, torch.exp(i[t] - top), torch.exp(-top)
                m = top
            kept[(p + end - first - 1) & 1] = m

    def low_rank(self, rows, at, wt, out, bias=None, mode=0, factor=1.0, rate=None):
        self.calls.append("low_rank")
        z = rows[:, at:at + wt.shape[0]] @ wt.float()
        if bias is not None:
            z = z + bias
        if mode == 1:
            z = torch.nn.functional.logsigmoid(z) * factor
        elif mode == 2:
            z = -torch.nn.functional.softplus(z) * rate.repeat_interleave(z.shape[1] // rate.numel())
        out.copy_(z)

    def channel_state_scratch(self, n_tokens, n_seqs, max_q_len, heads, dim, vdim, delta):
        return 4

    def channel_state(self, rows, q_at, k_at, v_at, log_decay, out, state, step_meta, heads, groups, dim, vdim, max_q_len, scratch,
                      q_scale=1.0, beta_rows=None, beta_at=0, unit_eps=None, state_offset=0):
        self.calls.append("channel_state")
        positions, token_seq, cu_q, slot_ids = step_meta
        n = rows.shape[0]
        unit = (lambda x: x) if unit_eps is None else (lambda x: x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + unit_eps))
        spread = lambda at: unit(rows[:, at:at + groups * dim].view(n, groups, dim)).repeat_interleave(heads // groups, dim=1)
        q, k, v = spread(q_at) * q_scale, spread(k_at), rows[:, v_at:v_at + heads * vdim].view(n, heads, vdim)
        d = torch.exp(log_decay).view(n, heads, dim)
        size = heads * dim * vdim
        for s in range(slot_ids.numel()):
            first, end = int(cu_q[s]), int(cu_q[s + 1])
            row = state[int(slot_ids[s])][state_offset:]
            p = int(positions[first])
            S = row[((p - 1) & 1) * size:][:size].clone().view(heads, dim, vdim) if p > 0 else torch.zeros(heads, dim, vdim)
            for t in range(first, end):
                S = d[t][:, :, None] * S
                u = v[t]
                if beta_rows is not None:
                    u = torch.sigmoid(beta_rows[t, beta_at:beta_at + heads])[:, None] * (u - torch.einsum("hnp,hn->hp", S, k[t]))
                S = S + k[t][:, :, None] * u[:, None, :]
                out[t] = torch.einsum("hnp,hn->hp", S, q[t]).reshape(-1)
            row[((p + end - first - 1) & 1) * size:][:size] = S.reshape(-1)

    def matrix_step(self, kind, rows, q_at, k_at, v_at, out, state, step_meta, heads, groups, dim, vdim, norm, eps, gate_at,
                    q_scale=1.0, unit_eps=None, conv_w=None, ring_offset=0, decay_at=0, decay_wt=None, decay_bias=None, decay_mode=1,
                    decay_factor=1.0, decay_rate=None, beta_at=0, input_at=0, forget_at=0, input_bias=None, forget_bias=None,
                    cap=1.0, denominator_eps=0.0, gate_wt=None, gate_silu=False, state_offset=0):
        self.calls.append("matrix_step")
        n, hp = rows.shape[0], heads * vdim
        y = torch.zeros(n, hp)
        if kind == 2:
            decay, scale, floor = torch.zeros(n, heads), torch.zeros(n, heads), torch.zeros(n, heads)
            self.exp_gates(rows, input_at, forget_at, input_bias, forget_bias, cap, decay, scale, floor, step_meta, state,
                           state_offset + 2 * heads * dim * (vdim + 1))
            self.linear_state(rows, q_at, k_at, v_at, y, state, step_meta, heads, groups, dim, vdim, 1, log_decay=decay,
                              key_scale=scale, state_offset=state_offset, out_scale=q_scale, floor=floor, floor_eps=denominator_eps)
        else:
            log_decay = torch.zeros(n, heads * dim)
            self.low_rank(rows, decay_at, decay_wt, log_decay, decay_bias, decay_mode, decay_factor, decay_rate)
            inputs, beta = rows, None
            if kind == 1:
                inputs, beta = torch.zeros(n, conv_w.shape[0]), rows
                self.conv_silu(rows, conv_w, None, inputs, step_meta, state, ring_offset)
                self.short_conv_remember(rows, None, conv_w.shape[0], conv_w.shape[1], n, step_meta, state, ring_offset)
            self.channel_state(inputs, q_at, k_at, v_at, log_decay, y, state, step_meta, heads, groups, dim, vdim, 1, None,
                               q_scale, beta, beta_at, unit_eps, state_offset)
        gate = rows[:, gate_at:gate_at + hp]
        if gate_wt is not None:
            gate = rows[:, gate_at:gate_at + gate_wt.shape[0]] @ gate_wt.float()
        self.gated_norm(y, gate, 0, norm, heads, eps, 2 if gate_silu else 0, out)

    def scale_inplace(self, x, factor):
        x.mul_(factor)

    def add_inplace(self, out, other):
        out.add_(other)

    def argmax(self, logits, out, flag=None):
        out.copy_(torch.argmax(logits, dim=-1).to(torch.int32))


def double_loader():
    made = {}

    def load(dtype, head_dim):
        key = (dtype, head_dim)
        if key not in made:
            made[key] = DoubleKernels(dtype, head_dim)
        return made[key]
    return load
