"""The mechanisms of the Tobozen decoder one at a time, each kernel against the plain implementation's function
(tests/plain_tobozen.py): the norm in groups; the norms over all heads with rotation, value mixing and the cache write,
heads stored wider than they are; attention with one added to the denominator where one key is made to dominate at page
borders, far back, at the first position and at the query itself, in prompts and in one-token steps, and where no key is
worth looking at; the matrix-state recurrence over portions, batches, used slots and steps that run twice, at chunk
borders, with decays per head and per token, a token hundreds back that a slow head keeps, and a token that forgets
everything; the convolution and step sizes; the gated norms; the experts."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_tobozen as plain

pytestmark = pytest.mark.gpu

F64 = torch.float64
DTYPES = [torch.float32, torch.bfloat16]


def kernels(dtype, head_dim=64):
    from stratakv_b200 import ops
    return ops.kernels_for(dtype, head_dim, verbose=False)


def i32(values):
    return torch.as_tensor(values, dtype=torch.int32).cuda()


def close(got, want, dtype, what="", loose=1.0):
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape, what
    allowed = (2e-5 if dtype == torch.float32 else 1.2e-2) * loose * max(1.0, float(want.abs().max()))
    worst = float((got - want).abs().max())
    assert worst <= allowed, f"{what}: off by {worst:.3e} (allowed {allowed:.3e})"


def table_of(rot, positions):
    """[positions, dims / 2, 2] float32 of (cos, sin)."""
    f = torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)], dtype=F64)
    angle = torch.arange(positions, dtype=F64)[:, None] * f[None, :]
    return torch.stack([torch.cos(angle), torch.sin(angle)], dim=-1).float().cuda()


def batch_meta(at, counts, slots):
    positions = [p for b, c in zip(at, counts) for p in range(b, b + c)]
    token_seq = [s for s, c in enumerate(counts) for _ in range(c)]
    cu_q = [0]
    for c in counts:
        cu_q.append(cu_q[-1] + c)
    return (i32(positions), i32(token_seq), i32(cu_q), i32(slots)), cu_q


# ---- the norm in groups -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,hidden,groups", [(3, 96, 4), (5, 44, 11), (700, 256, 2), (1100, 64, 1), (2, 4096, 8), (9, 30, 3)])
def test_norm_in_groups(dtype, rows, hidden, groups):
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(rows)
    x = torch.randn(rows, hidden, generator=g) * torch.rand(hidden, generator=g) * 4.0
    weight = torch.rand(hidden, generator=g) + 0.5
    out = torch.empty(rows, hidden, dtype=dtype, device="cuda")
    ops.rmsnorm(x.cuda(), weight.cuda(), 1e-5, out, groups=groups)
    want = plain.grouped_norm(x.double(), weight.double(), groups, 1e-5)
    close(out, want, dtype, "all rows")
    some = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32)
    picked = torch.empty(3, hidden, dtype=dtype, device="cuda")
    ops.rmsnorm(x.cuda(), weight.cuda(), 1e-5, picked, some.cuda(), groups=groups)
    close(picked, want[some.long()], dtype, "rows by index")


# ---- norms over all heads, rotation, value mixing, cache write ----------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 16, 24, 12, 64), (6, 3, 20, 16, 20, 64), (2, 1, 96, 112, 32, 128), (3, 1, 10, 6, 4, 0),
                                   (2, 2, 64, 64, 64, 64), (16, 2, 144, 136, 50, 0)])
def test_norms_over_all_heads_rotation_mixing_and_cache(dtype, shape):
    H, G, d, dv, rotated, width = shape
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(d)
    block, counts, at = 16, [5, 1, 37], [0, 33, 14]
    n = sum(counts)
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "rot": {"dims": rotated, "base": 300.0}, "v_mix": True}
    kw, vw = width or d, width or dv
    rows = torch.randn(n, H * d + G * d + G * dv + 4, generator=g)
    rows = rows[:, :(rows.shape[1] // 4) * 4].contiguous() if (rows.shape[1] % 4 and d % 4 == 0) else rows
    P = {"q.norm": torch.rand(H * d, generator=g).double() + 0.5, "k.norm": torch.rand(G * d, generator=g).double() + 0.5,
         "vmix": torch.tensor(0.3, dtype=F64)}
    first = torch.randn(n, G * dv, generator=g)
    (positions, token_seq, _, _), _ = batch_meta(at, counts, [0, 1, 2])
    tables = (torch.randperm(12, generator=g) + 1).view(3, 4).to(torch.int32)
    q_out = torch.full((n, H * kw), 7.0, dtype=dtype, device="cuda")
    k_cache = torch.full((14, G, block, kw), 7.0, dtype=dtype, device="cuda")
    v_cache = torch.full((14, G, block, vw), 7.0, dtype=dtype, device="cuda")
    keep = torch.empty(n, G * dv, device="cuda")
    ops.normed_rotary(rows.cuda(), q_out, k_cache, v_cache, positions, token_seq, tables.cuda(), H, G, d, dv, block, eps=1e-5,
                      q_weight=P["q.norm"].float().cuda(), k_weight=P["k.norm"].float().cuda(),
                      cos_sin=table_of(m["rot"], 80), rotated=rotated, interleaved=True,
                      mix=P["vmix"].float().reshape(1).cuda(), first=first.cuda(), keep=keep)
    # the plain functions on the projections themselves
    wide = rows.double()
    q = plain.grouped_norm(wide[:, :H * d], P["q.norm"], 1, 1e-5).view(n, H, d)
    k = plain.grouped_norm(wide[:, H * d:(H + G) * d], P["k.norm"], 1, 1e-5).view(n, G, d)
    own = wide[:, (H + G) * d:(H + G) * d + G * dv]
    v = plain.mixed_values(own, P, "", first.double()).view(n, G, dv)
    where = positions.cpu().long()
    q, k = plain.rotate_pairs(q, where, m["rot"]), plain.rotate_pairs(k, where, m["rot"])
    got_q = q_out.view(n, H, kw)
    close(got_q[..., :d], q, dtype, "queries", 0.5)
    assert float(got_q[..., d:].float().abs().sum()) == 0.0
    close(keep, own, torch.float32, "the values before mixing")
    for t in range(n):
        p, s = int(where[t]), int(token_seq[t])
        page = int(tables[s, p // block])
        close(k_cache[page, :, p % block, :d], k[t], dtype, f"key of token {t}", 0.5)
        close(v_cache[page, :, p % block, :dv], v[t], dtype, f"value of token {t}", 0.5)
        assert float(k_cache[page, :, p % block, d:].float().abs().sum() + v_cache[page, :, p % block, dv:].float().abs().sum()) == 0.0
    # not one norm per head: the heads of a row share one root mean square
    per_head = plain.unit_rms(wide[:, :H * d].view(n, H, d), 1e-5).reshape(n, H * d) * P["q.norm"]
    assert H == 1 or float((plain.rotate_pairs(per_head.view(n, H, d), where, m["rot"]) - q).abs().max()) > 0.05
    # a page nobody was given stays as it was
    assert float((k_cache[0].float() - 7.0).abs().max()) == 0.0


def test_split_half_pairs_without_norm_or_mixing():
    """The other pair layout and every switch off (another design's use of the kernel)."""
    ops = kernels(torch.float32)
    g = torch.Generator().manual_seed(3)
    H, G, d, dv, rotated = 2, 1, 12, 8, 8
    rows = torch.randn(4, H * d + G * (d + dv), generator=g)
    table = table_of({"dims": rotated, "base": 100.0}, 8)
    q_out = torch.empty(4, H * d, device="cuda")
    k_cache, v_cache = torch.zeros(2, G, 16, d, device="cuda"), torch.zeros(2, G, 16, dv, device="cuda")
    ops.normed_rotary(rows.cuda(), q_out, k_cache, v_cache, i32([2, 3, 4, 5]), i32([0, 0, 0, 0]), i32([[1]]), H, G, d, dv, 16,
                      cos_sin=table, rotated=rotated)
    cs = table.cpu()[2:6].double()
    x = rows[:, :H * d].double().view(4, H, d)
    want = x.clone()
    c, s = cs[:, None, :, 0], cs[:, None, :, 1]
    want[..., :4], want[..., 4:8] = x[..., :4] * c - x[..., 4:8] * s, x[..., 4:8] * c + x[..., :4] * s
    close(q_out.view(4, H, d), want, torch.float32, "queries")
    close(v_cache[1, 0, 2:6], rows[:, (H + G) * d:].double(), torch.float32, "values")


# ---- attention with one more in the denominator -------------------------------------------------------------------------
def run_attention(dtype, q, k, v, scale, before, width, block=16, decode=False):
    """Queries of the last T - before positions through ``attend_with_sink`` over a paged cache with scattered pages."""
    from stratakv_b200.parts.attention import attend_with_sink
    from stratakv_b200.parts.workspace import Workspace
    T, H, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    kw, vw = width or d, width or dv
    pages = -(-T // block)
    order = (torch.randperm(pages, generator=torch.Generator().manual_seed(T)) + 1).to(torch.int32)
    k_cache = torch.full((pages + 2, G, block, kw), 3.0, dtype=dtype)          # (rows nobody wrote must not be read)
    v_cache = torch.full((pages + 2, G, block, vw), 3.0, dtype=dtype)
    for t in range(T):
        page = int(order[t // block])
        for cache, x in ((k_cache, k), (v_cache, v)):
            cache[page, :, t % block] = 0.0
            cache[page, :, t % block, :x.shape[2]] = x[t].to(dtype)
    new = T - before
    wide_q = torch.zeros(new, H, kw, dtype=dtype)
    wide_q[..., :d] = q[before:].to(dtype)
    rt = SimpleNamespace(dtype=dtype, device=torch.device("cuda"), workspace=Workspace("cuda"), sm_count=148,
                         kernels=lambda head_dim=64: kernels(dtype, head_dim))
    step = SimpleNamespace(n_seqs=1, max_q_len=new, max_ctx=T, is_decode=new == 1, positions=i32(list(range(before, T))),
                           token_seq=i32([0] * new), cu_q=i32([0, new]), ctx_after=i32([T]), cache=SimpleNamespace(block_size=block))
    ctx = torch.full((new, H * vw), 9.0, dtype=dtype, device="cuda")
    sink = torch.zeros(H, device="cuda")
    attend_with_sink(step, rt, wide_q.reshape(new, H * kw).cuda(), ctx, k_cache.cuda(), v_cache.cuda(), order.view(1, -1).cuda(), H, G, kw,
                     vw, scale, sink=sink)
    out = ctx.view(new, H, vw)
    assert float(out[..., dv:].float().abs().sum()) == 0.0
    return out[..., :dv]


ATTENTION = [(torch.float32, (4, 2, 16, 24), 64), (torch.float32, (2, 1, 144, 136), 0), (torch.bfloat16, (4, 2, 16, 24), 64),
             (torch.bfloat16, (2, 2, 64, 64), 64), (torch.bfloat16, (6, 2, 96, 112), 128), (torch.bfloat16, (2, 1, 144, 136), 0)]


@pytest.mark.parametrize("dtype,shape,width", ATTENTION)
@pytest.mark.parametrize("before,total", [(0, 5), (0, 150), (97, 160), (149, 150), (0, 1), (1500, 1501)])
def test_attention_with_a_key_that_stands_out(dtype, shape, width, before, total):
    """One key is made to score far above the rest for every query: at the first position, on both sides of a page's
    border, far back, and the query's own; the queries before it do not see it."""
    H, G, d, dv = shape
    for spot in sorted({0, 15, 16, 63, 64, total // 2, total - 2, total - 1}):
        if not 0 <= spot < total:
            continue
        g = torch.Generator().manual_seed(spot + total)
        q, k, v = (torch.randn(total, h, w, generator=g) for h, w in ((H, d), (G, d), (G, dv)))
        q[..., 0] = 3.0
        k[..., 0] = -0.5
        k[spot, :, 0] = 3.5
        v[spot] += 5.0
        q, k, v = (x.to(dtype).double() for x in (q, k, v))
        scale = d ** -0.5
        want = plain.attend(q, k, v, scale)[before:]
        close(run_attention(dtype, q, k, v, scale, before, width), want, dtype, f"key {spot} of {total}")


@pytest.mark.parametrize("dtype,shape,width", ATTENTION)
@pytest.mark.parametrize("before,total", [(0, 70), (199, 200)])
def test_attention_where_no_key_is_worth_looking_at(dtype, shape, width, before, total):
    """All scores far below zero: the one in the denominator takes nearly all the weight, and with a plain softmax the
    outputs would be of the values' size."""
    H, G, d, dv = shape
    g = torch.Generator().manual_seed(total)
    q, k, v = (torch.randn(total, h, w, generator=g) * 0.1 for h, w in ((H, d), (G, d), (G, dv)))
    q[..., 0], k[..., 0] = 4.0, -3.0
    v = v * 10.0 + 2.0
    q, k, v = (x.to(dtype).double() for x in (q, k, v))
    want = plain.attend(q, k, v, 0.8)[before:]
    assert float(want.abs().max()) < 0.2
    got = run_attention(dtype, q, k, v, 0.8, before, width)
    allowed = (1e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())
    assert float((got.double().cpu() - want).abs().max()) <= allowed


# ---- the matrix-state recurrence ----------------------------------------------------------------------------------------
SHAPES = [(3, 3, 8, 12), (4, 2, 16, 20), (2, 1, 128, 64), (1, 1, 72, 100), (3, 3, 7, 9), (2, 1, 200, 40), (4, 4, 64, 130)]


def state_inputs(n, H, G, dim, vdim, generator):
    rows = torch.randn(n, 2 * G * dim + H * vdim + 5, generator=generator)
    return rows, 3 if (dim % 4 or vdim % 4) else 4


@pytest.mark.parametrize("per_token", [False, True])
@pytest.mark.parametrize("shape", SHAPES)
def test_recurrence_over_portions_batches_and_used_slots(shape, per_token):
    """Three sequences in one packed step after another, in portions around the chunks' length, in slots whose state holds
    1e30; one-token steps run twice; a head keeps nearly all and a head loses nearly all of what it has."""
    H, G, dim, vdim = shape
    ops = kernels(torch.float32)
    g = torch.Generator().manual_seed(dim + vdim)
    lengths = [150, 131, 67]
    portions = [(64, 1, 65), (1, 1, 1), (63, 129, 0), (1, 0, 1), (1, 0, 0), (20, 0, 0)]
    assert [sum(p[i] for p in portions) for i in range(3)] == lengths
    offset, width = 8, 2 * G * dim + H * vdim
    at_q, at_k, at_v = 4, 4 + G * dim, 4 + 2 * G * dim
    stride = -(-(4 + width) // 4) * 4
    rows = [torch.randn(n, stride, generator=g) for n in lengths]
    decay = torch.linspace(0.2, 0.999, H) if H > 1 else torch.tensor([0.95])
    log_decay = [-torch.rand(n, H, generator=g) ** 4 * 6.0 for n in lengths]
    scale = [torch.rand(n, H, generator=g) + 0.2 for n in lengths]
    skip = torch.randn(H, generator=g) if per_token else None
    slots = [4, 1, 2]
    state = torch.full((6, offset + 2 * H * dim * vdim + 4), 1e30, device="cuda")
    want = []
    for r, l, c in zip(rows, log_decay, scale):
        spread = lambda x: x.double().view(-1, G, dim).repeat_interleave(H // G, dim=1)
        q, k = spread(r[:, at_q:at_q + G * dim]), spread(r[:, at_k:at_k + G * dim])
        v = r[:, at_v:at_v + H * vdim].double().view(-1, H, vdim)
        if per_token:
            o = plain.decayed_sums(q, k * c.double()[:, :, None], v, torch.exp(l.double())) + skip.double()[:, None] * v
        else:
            o = plain.decayed_sums(plain.silu(q), plain.silu(k), plain.silu(v), decay.double().expand(len(r), H))
        want.append(o.reshape(len(r), -1))
    got, at = [[] for _ in lengths], [0, 0, 0]
    for portion in portions:
        live = [i for i in range(3) if portion[i]]
        counts = [portion[i] for i in live]
        meta, cu = batch_meta([at[i] for i in live], counts, [slots[i] for i in live])
        pick = lambda parts: torch.cat([parts[i][at[i]:at[i] + portion[i]] for i in live]).cuda()
        fused = pick(rows)
        more = dict(log_decay=pick(log_decay), key_scale=pick(scale), skip=skip.cuda()) if per_token else \
            dict(decay=decay.cuda(), silu=True)
        need = ops.linear_state_scratch(len(live), max(counts), H, dim, vdim)
        scratch = torch.full((max(need, 1),), 1e30, device="cuda")
        for turn in range(2 if max(counts) == 1 else 1):
            out = torch.empty(sum(counts), H * vdim, device="cuda")
            ops.linear_state(fused, at_q, at_k, at_v, out, state, meta, H, G, dim, vdim, max(counts), scratch=scratch,
                             state_offset=offset, **more)
        for s, i in enumerate(live):
            got[i].append(out[cu[s]:cu[s + 1]])
            at[i] += portion[i]
    for i in range(3):
        close(torch.cat(got[i]), want[i], torch.float32, f"sequence {i}", 2.0)
    assert bool((state[[0, 3, 5]] == state.new_tensor(1e30)).all())              # nobody else's slot was touched


@pytest.mark.parametrize("dim", [320, 600])
def test_recurrence_with_keys_too_wide_for_long_chunks(dim):
    ops = kernels(torch.float32)
    g = torch.Generator().manual_seed(dim)
    n, vdim = 83, 8
    rows = torch.randn(n, 2 * dim + vdim, generator=g) * 0.3
    meta, _ = batch_meta([0], [n], [0])
    state = torch.full((1, 2 * dim * vdim), 1e30, device="cuda")
    out = torch.empty(n, vdim, device="cuda")
    scratch = torch.empty(ops.linear_state_scratch(1, n, 1, dim, vdim), device="cuda")
    ops.linear_state(rows.cuda(), 0, dim, 2 * dim, out, state, meta, 1, 1, dim, vdim, n, decay=torch.tensor([0.9]).cuda(), scratch=scratch)
    r = rows.double()
    want = plain.decayed_sums(r[:, None, :dim], r[:, None, dim:2 * dim], r[:, None, 2 * dim:], torch.full((n, 1), 0.9, dtype=F64))
    close(out, want[:, 0], torch.float32, "wide keys", 2.0)


@pytest.mark.parametrize("decode", [False, True])
def test_a_token_hundreds_back_is_kept_and_lost(decode):
    """One token with a large key and value, then 400 near nothing: a head with decay 0.9995 still has it, one with 0.9
    has lost it, and a later token that forgets everything takes it away for good."""
    ops = kernels(torch.float32)
    n, dim, vdim, H = 402, 16, 24, 2
    rows = torch.full((n, 2 * H * dim + H * vdim), 1e-4)
    rows[:, :H * dim] = 1.0
    rows[3, H * dim:] = 2.0
    log_decay = torch.log(torch.tensor([0.9995, 0.9])).repeat(n, 1)
    log_decay[401] = -200.0
    state = torch.full((2, 2 * H * dim * vdim), 1e30, device="cuda")
    outs = []
    for lo, hi in ((0, 2), *((t, t + 1) for t in range(2, n))) if decode else ((0, n),):
        meta, _ = batch_meta([lo], [hi - lo], [1])
        out = torch.empty(hi - lo, H * vdim, device="cuda")
        need = ops.linear_state_scratch(1, hi - lo, H, dim, vdim)
        ops.linear_state(rows[lo:hi].cuda().contiguous(), 0, H * dim, 2 * H * dim, out, state, meta, H, H, dim, vdim, hi - lo,
                         log_decay=log_decay[lo:hi].cuda().contiguous(), scratch=torch.empty(max(1, need), device="cuda"))
        outs.append(out)
    got = torch.cat(outs).cpu().view(n, H, vdim)
    held = dim * 4.0 * 0.9995 ** 397
    assert float((got[400, 0] - held).abs().max()) < 1e-3 * held and held > 50
    assert float(got[400, 1].abs().max()) < 1e-3
    assert float(got[401].abs().max()) < 1e-5                    # only that token's own product is left


def test_a_token_that_forgets_does_not_cost_precision():
    """Decays of e^-60 in the middle of a chunk: the sums behind them are made from the tokens between, so the weights of
    neighbours stay exact where a difference of two running sums would be off."""
    ops = kernels(torch.float32)
    g = torch.Generator().manual_seed(9)
    n, dim, vdim = 64, 16, 16
    rows = torch.randn(n, 2 * dim + vdim, generator=g)
    log_decay = -torch.rand(n, 1, generator=g) * 1e-3
    log_decay[::7] = -60.0
    log_decay[30] = -4000.0
    meta, _ = batch_meta([0], [n], [0])
    state = torch.zeros(1, 2 * dim * vdim, device="cuda")
    out = torch.empty(n, vdim, device="cuda")
    scratch = torch.empty(ops.linear_state_scratch(1, n, 1, dim, vdim), device="cuda")
    ops.linear_state(rows.cuda(), 0, dim, 2 * dim, out, state, meta, 1, 1, dim, vdim, n, log_decay=log_decay.cuda(), scratch=scratch)
    r = rows.double()
    want = plain.decayed_sums(r[:, None, :dim], r[:, None, dim:2 * dim], r[:, None, 2 * dim:], torch.exp(log_decay.double()))[:, 0]
    assert float((out.double().cpu() - want).abs().max()) <= 3e-6 * float(want.abs().max())


# ---- Mamba-2's own steps --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("shape", [(4, 2, 8, 12, 4), (6, 1, 14, 10, 1), (2, 1, 16, 64, 8), (3, 3, 9, 7, 2), (2, 2, 6, 18, 11)])
def test_mamba2_between_its_projections(shape):
    """Convolution, step sizes and recurrence over portions (shorter and longer than the convolution reaches) and one-token
    steps that run twice, in used slots, against the plain functions on the whole sequences."""
    H, G, N, dv, taps = shape
    ops = kernels(torch.float32)
    g = torch.Generator().manual_seed(taps)
    inner, gn = H * dv, G * N
    channels = inner + 2 * gn
    dt_at, stride = channels, -(-(channels + H) // 8) * 8
    lengths = [40, 75]
    portions = [(1, 2), (1, 1), (2, 70), (1, 1), (1, 1), (34, 0)]
    rows = [torch.randn(n, stride, generator=g) for n in lengths]
    P = {"conv": torch.randn(channels, taps, generator=g).double() / taps, "conv.b": torch.randn(channels, generator=g).double(),
         "dt_bias": torch.randn(H, generator=g).double() - 1.0, "A_log": torch.rand(H, generator=g).double() * 2.0, "D": torch.randn(H, generator=g).double()}
    f = {k: v.float().cuda().contiguous() for k, v in P.items()}
    want = []
    for r in rows:
        u = plain.silu(plain.causal_convolution(r[:, :channels].double(), P["conv"], P["conv.b"]))
        T = r.shape[0]
        dt = plain.softplus(r[:, dt_at:dt_at + H].double() + P["dt_bias"])
        want.append(plain.mamba2_sums(u[:, :inner].view(T, H, dv), u[:, inner:inner + gn].view(T, G, N), u[:, inner + gn:].view(T, G, N), dt, P, "").reshape(T, -1))
    ring = 2 * H * N * dv
    state = torch.full((5, -(-(ring + taps * channels) // 4) * 4), 1e30, device="cuda")
    slots, at, got = [3, 0], [0, 0], [[], []]
    for portion in portions:
        live = [i for i in range(2) if portion[i]]
        counts = [portion[i] for i in live]
        meta, cu = batch_meta([at[i] for i in live], counts, [slots[i] for i in live])
        fused = torch.cat([rows[i][at[i]:at[i] + portion[i]] for i in live]).cuda()
        out = torch.empty(sum(counts), inner, device="cuda")
        if max(counts) == 1:
            for _ in range(2):
                ops.mamba2_step(fused, f["conv"], f["conv.b"], dt_at, f["dt_bias"], f["A_log"], f["D"], out, state, meta, H, G, N, dv, 0, ring)
        else:
            u = torch.empty(sum(counts), channels, device="cuda")
            dt, log_decay = torch.empty(sum(counts), H, device="cuda"), torch.empty(sum(counts), H, device="cuda")
            ops.conv_silu(fused, f["conv"], f["conv.b"], u, meta, state, ring)
            ops.step_sizes(fused, dt_at, f["dt_bias"], f["A_log"], dt, log_decay)
            scratch = torch.empty(ops.linear_state_scratch(len(live), max(counts), H, N, dv), device="cuda")
            ops.linear_state(u, inner + gn, inner, 0, out, state, meta, H, G, N, dv, max(counts), log_decay=log_decay, key_scale=dt,
                             skip=f["D"], scratch=scratch)
            ops.short_conv_remember(fused, None, channels, taps, len(live), meta, state, ring)
        for s, i in enumerate(live):
            got[i].append(out[cu[s]:cu[s + 1]])
            at[i] += portion[i]
    for i in range(2):
        close(torch.cat(got[i]), want[i], torch.float32, f"sequence {i}", 2.0)


def test_step_sizes_far_from_zero():
    ops = kernels(torch.float32)
    rows = torch.tensor([[-90.0, -3.0, 0.0, 19.0, 21.0, 80.0]]).T.contiguous().cuda()
    dt, log_decay = torch.empty(6, 1, device="cuda"), torch.empty(6, 1, device="cuda")
    ops.step_sizes(rows, 0, torch.tensor([0.5]).cuda(), torch.tensor([1.0]).cuda(), dt, log_decay)
    want = plain.softplus(rows.cpu().double() + 0.5)
    torch.testing.assert_close(dt.cpu().double(), want, rtol=1e-6, atol=0.0)
    torch.testing.assert_close(log_decay.cpu().double(), -math.e * want, rtol=1e-6, atol=0.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,groups", [(5, 48, 3), (5, 60, 1), (5, 126, 2), (5, 4096, 2), (5, 63, 7), (900, 48, 3), (1030, 1016, 2)])
def test_gated_norms(dtype, n, width, groups):
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(width)
    padded = -(-width // 8) * 8
    y, rows, weight = torch.randn(n, width, generator=g) * 3, torch.randn(n, width + 12, generator=g), torch.rand(width, generator=g) + 0.5
    gate = rows[:, 4:4 + width].double()
    view = rows.cuda()
    for gate_first in (True, False):
        out = torch.full((n, padded), 5.0, dtype=dtype, device="cuda")
        ops.gated_norm(y.cuda(), view[:, 4:], width + 12, weight.cuda(), groups, 1e-5, gate_first, out)
        want = (plain.grouped_norm(y.double() * plain.silu(gate), weight.double(), groups, 1e-5) if gate_first
                else plain.grouped_norm(y.double(), weight.double(), groups, 1e-5) * plain.sigmoid(gate))
        close(out[:, :width], want, dtype, f"gate first {gate_first}", 0.5)
        assert float(out[:, width:].float().abs().sum()) == 0.0


# ---- the experts --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,hidden,ff,experts,top,limit", [(37, 64, 24, 6, 2, 0.7), (5, 72, 36, 3, 3, 0.5), (300, 128, 72, 12, 1, 1.0)])
def test_experts_whose_weights_multiply_their_inputs(dtype, n, hidden, ff, experts, top, limit):
    """The part itself against ``plain.moe``, and against the same experts with the weight on their output, which it must
    not be; one expert gets nobody."""
    from stratakv_b200.parts.base import Runtime
    from stratakv_b200.parts.routed_mlp import RoutedMlp
    from stratakv_b200.parts.spec import RoutedMlpSpec
    from stratakv_b200.parts.workspace import Workspace
    g = torch.Generator().manual_seed(n)
    names = lambda part: tuple(f"e{k}.{part}" for k in range(experts))
    spec = RoutedMlpSpec(hidden, ff, experts, top, "swiglu_clamp", 1.0, "router", names("up"), names("down"), gate_weights=names("gate"),
                         activation_param=limit, weigh_input=True)
    tensors = {"router": torch.randn(experts, hidden, generator=g) * 0.3}
    for k in range(experts):
        for part, shape in (("gate", (ff, hidden)), ("up", (ff, hidden)), ("down", (hidden, ff))):
            tensors[f"e{k}.{part}"] = torch.randn(*shape, generator=g) * 0.3
    if experts > top:
        tensors["router"][1] = 0.0
        tensors["router"][1, 0] = -40.0
    tensors = {k: v.to(dtype) for k, v in tensors.items()}
    h = torch.randn(n, hidden, generator=g)
    h[:, 0] = h[:, 0].abs() + 1.0
    h = h.to(dtype)
    rt = Runtime(dtype, "cuda", Workspace("cuda"), lambda d, head_dim: kernels(d, 64), 64)
    part = RoutedMlp(spec, rt)
    part.bind(tensors)
    x = torch.zeros(n, hidden, device="cuda")
    seen = []
    step = SimpleNamespace(choice_probe=lambda run, step, chosen: seen.append(chosen.cpu().long()), run_index=0, store_branch=False)
    part.forward(step, h.cuda(), x)
    P = {k: v.double() for k, v in tensors.items()}
    mlp = {"expert": {"limit": limit}, "router": {"experts": experts, "top": top}}
    want = plain.moe(h.double(), P, "", mlp, seen[0])
    close(x, want, dtype, "experts", 1.0 if dtype == torch.float32 else 1.5)
    if experts > top:
        assert not bool((seen[0] == 1).any())
    chosen, weights = plain.route(h.double(), P, "", mlp["router"], seen[0])
    other = torch.zeros_like(want)
    for k in range(experts):
        t, c = torch.nonzero(chosen == k, as_tuple=True)
        if t.numel():
            other.index_add_(0, t, weights[t, c][:, None] * plain.expert(h[t].double(), P, f"e{k}.", limit))
    assert float((other - want).abs().max()) > 0.1 * float(want.abs().max())
