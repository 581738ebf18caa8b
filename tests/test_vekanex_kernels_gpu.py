"""The mechanisms of the Vekanex decoder one at a time, each kernel against the plain implementation's function
(tests/plain_vekanex.py): attention's inputs with biases, norms over all heads and rotation in half pairs, and attention
where one key dominates; the low-rank decays and gates; exponential gates, and the memory with its denominator; the
recurrences with a decay per key channel over portions, batches, used slots and steps that run twice, at chunk borders, with
a token hundreds back that a slow channel keeps and a fast one has lost, and channels that forget everything; the one-token
kernel against all of that; norms with gates, output biases, the stream that is handed on as it is, the cap on the logits,
the router's shares and the shared expert."""
import math

import pytest
import torch

import plain_vekanex as plain

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


# Portions of three sequences step by step: around a chunk's 16 or 32 tokens, down to one token, and one long step.
STEPS = [([0, 0, 0], [33, 1, 16]), ([33, 1, 16], [1, 31, 2]), ([34, 32, 18], [1, 1, 1]), ([35, 33, 19], [2, 64, 15]),
         ([37, 97, 34], [1, 1, 1]), ([38, 98, 35], [95, 2, 33])]
SLOTS = [4, 1, 2]
TOTAL = [133, 100, 68]


def used_state(floats):
    """State rows as an earlier user left them."""
    return torch.full((6, (floats + 3) // 4 * 4), 1e30, device="cuda")


def pieces(tensors, at, counts):
    """The rows of this step, packed."""
    return torch.cat([t[a:a + c] for t, a, c in zip(tensors, at, counts)])


# ---- attention's inputs ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 16, 24, 8, 64), (4, 2, 16, 24, 12, 64), (2, 1, 96, 112, 96, 128), (3, 1, 10, 6, 4, 0), (6, 1, 64, 64, 16, 64),
                                   (2, 2, 144, 136, 50, 0), (1, 1, 32, 32, 0, 64)])
def test_biases_norms_over_all_heads_and_half_pairs(dtype, shape):
    H, G, d, dv, rotated, width = shape
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(d + rotated)
    block, counts, at = 16, [5, 1, 37], [0, 33, 14]
    n, total = sum(counts), (H + G) * d + G * dv
    kw, vw = width or d, width or dv
    rows = torch.randn(n, -(-total // 8) * 8, generator=g)
    bias = torch.randn(total, generator=g)
    weights = [torch.rand(count * d, generator=g) + 0.5 for count in (H, G)]
    (positions, token_seq, _, _), _ = batch_meta(at, counts, [0, 1, 2])
    tables = (torch.randperm(12, generator=g) + 1).view(3, 4).to(torch.int32)
    q_out = torch.full((n, H * kw), 7.0, dtype=dtype, device="cuda")
    k_cache = torch.full((14, G, block, kw), 7.0, dtype=dtype, device="cuda")
    v_cache = torch.full((14, G, block, vw), 7.0, dtype=dtype, device="cuda")
    rot = {"dims": rotated, "base": 300.0}
    ops.normed_rotary(rows.cuda(), q_out, k_cache, v_cache, positions, token_seq, tables.cuda(), H, G, d, dv, block, eps=1e-5,
                      q_weight=weights[0].cuda(), k_weight=weights[1].cuda(), cos_sin=table_of(rot, 80) if rotated else None,
                      rotated=rotated, bias=bias.cuda())
    # the plain function on the identity as projections
    P = {}
    for name, lo, hi in (("q", 0, H * d), ("k", H * d, (H + G) * d), ("v", (H + G) * d, total)):
        P[name] = torch.eye(total, dtype=F64)[lo:hi]
        P[name + ".b"] = bias[lo:hi].double()
    P["q.norm"], P["k.norm"] = weights[0].double(), weights[1].double()
    where = positions.cpu().long()
    q, k, v = plain.attention_inputs(rows[:, :total].double(), P, "", {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "rot": rot}, 1e-5, where)
    got_q = q_out.view(n, H, kw)
    close(got_q[..., :d], q, dtype, "queries", 0.5)
    assert float(got_q[..., d:].float().abs().sum()) == 0.0
    for t in range(n):
        p, s = int(where[t]), int(token_seq[t])
        page = int(tables[s, p // block])
        close(k_cache[page, :, p % block, :d], k[t], dtype, f"key of token {t}", 0.5)
        close(v_cache[page, :, p % block, :dv], v[t], dtype, f"value of token {t}", 0.5)
        assert float(k_cache[page, :, p % block, d:].float().abs().sum() + v_cache[page, :, p % block, dv:].float().abs().sum()) == 0.0
    assert float((k_cache[0].float() - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,width,count,start", [(4, 2, 64, 300, 0), (2, 1, 128, 260, 0), (6, 1, 64, 40, 150), (4, 4, 64, 1, 259),
                                                              (6, 1, 128, 1, 200), (2, 1, 144, 70, 90), (3, 1, 64, 2, 64)])
def test_attention_where_one_key_dominates(dtype, heads, kv_heads, width, count, start):
    """One key scores far above all others for one query: the first position, both sides of a page's border, hundreds back
    and the query itself; prompts, a portion behind a prefix, one token, without a sink."""
    from types import SimpleNamespace
    from stratakv_b200.parts.attention import attend_with_sink
    ops = kernels(dtype, width if width in (64, 128) else 64)
    g = torch.Generator().manual_seed(width + count)
    block, total = 64, start + count
    scale = width ** -0.5
    q = torch.randn(total, heads, width, generator=g)
    k = torch.randn(total, kv_heads, width, generator=g)
    v = torch.randn(total, kv_heads, width, generator=g)
    targets = sorted({t for t in (0, 63, 64, 127, 128, start, total - 1, total // 2) if t < total})
    asked = []
    for j, target in enumerate(targets):           # (queries from the last one back, each for one target)
        i = total - 1 - j
        if i < max(start, target):
            continue
        q[i] = 0.0
        q[i, :, j] = 30.0 * width ** 0.5 / 8.0
        k[:, :, j] = 0.0
        k[target, :, j] = 8.0
        asked.append((i, target))
    rounded = [x.to(dtype) for x in (q, k, v)]
    pages = -(-total // block)
    table = (torch.randperm(pages, generator=g) + 1).to(torch.int32).view(1, -1)
    k_cache = torch.zeros(pages + 2, kv_heads, block, width, dtype=dtype)
    v_cache = torch.zeros(pages + 2, kv_heads, block, width, dtype=dtype)
    for p in range(total):
        k_cache[table[0, p // block], :, p % block] = rounded[1][p]
        v_cache[table[0, p // block], :, p % block] = rounded[2][p]
    meta, cu = batch_meta([start], [count], [0])
    scratch = {}

    def get(name, shape, kind):
        return scratch.setdefault((name, shape), torch.empty(shape, dtype=kind, device="cuda"))

    step = SimpleNamespace(is_decode=count == 1, max_q_len=count, n_seqs=1, max_ctx=total, positions=meta[0], token_seq=meta[1], cu_q=meta[2],
                           ctx_after=i32([total]), cache=SimpleNamespace(block_size=block))
    rt = SimpleNamespace(dtype=dtype, device=torch.device("cuda"), sm_count=148, workspace=SimpleNamespace(get=get),
                         kernels=lambda head_dim=None: ops)
    out = torch.empty(count, heads * width, dtype=dtype, device="cuda")
    attend_with_sink(step, rt, rounded[0][start:].reshape(count, -1).cuda(), out, k_cache.cuda(), v_cache.cuda(), table.cuda(), heads, kv_heads,
                     width, width, scale)
    want = plain.attend(*(x.double() for x in rounded), scale)[start:]
    close(out.view(count, heads, width), want, dtype, "attention")
    assert asked
    for i, target in asked:
        near = want[i - start] - rounded[2][target].double().repeat_interleave(heads // kv_heads, dim=0)
        assert float(near.abs().max()) < 0.05, f"query {i} does not single out key {target}: the test would not show a lost one"


# ---- low-rank projections --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,rank,heads,dim", [(3, 5, 3, 12), (300, 24, 4, 80), (1, 1, 1, 7), (257, 130, 2, 33)])
def test_low_rank_ends(dtype, n, rank, heads, dim):
    from stratakv_b200 import ops as O
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(rank)
    rows = torch.randn(n, rank + 9, generator=g) * 2.0
    wt = (torch.randn(rank, heads * dim, generator=g) / rank ** 0.5 * 4.0).to(dtype)
    bias, rate = torch.randn(heads * dim, generator=g) * 3.0, torch.rand(heads, generator=g) * 5.0
    z = rows[:, 3:3 + rank].double() @ wt.double()
    for mode, b, want in ((O.LOW_RANK_PLAIN, None, z), (O.LOW_RANK_LOG_SIGMOID, bias, plain.log_sigmoid(z + bias.double()) / 7.0),
                          (O.LOW_RANK_SOFTPLUS, bias, -plain.softplus(z + bias.double()) * rate.double().repeat_interleave(dim))):
        out = torch.empty(n, heads * dim, device="cuda")
        ops.low_rank(rows.cuda(), 3, wt.cuda(), out, bias=b.cuda() if b is not None else None, mode=mode, factor=1.0 / 7.0,
                     rate=rate.cuda() if mode == O.LOW_RANK_SOFTPLUS else None)
        close(out, want, torch.float32, f"mode {mode}")
    # far from zero: a gate that is shut keeps exp(z), one that is open loses exp(-z)
    far = torch.tensor([[60.0, -60.0, 12.0, -12.0]])
    out = torch.empty(1, 4, device="cuda")
    ops.low_rank(far.cuda(), 0, torch.eye(4).to(dtype).cuda(), out, mode=O.LOW_RANK_LOG_SIGMOID)
    want = plain.log_sigmoid(far.double())
    assert float(((out.cpu().double() - want) / want).abs()[0, 1:].max()) < 1e-5 and abs(float(out[0, 0])) < 1e-20


# ---- recurrences with a decay per key channel -----------------------------------------------------------------------------------
CHANNEL_SHAPES = [(4, 2, 12, 8), (3, 3, 64, 64), (2, 1, 128, 40), (2, 2, 9, 7), (1, 1, 290, 21), (2, 2, 48, 132), (1, 1, 4, 3)]


def channel_case(heads, groups, dim, vdim, seed, fast=3.0):
    g = torch.Generator().manual_seed(seed)
    made = lambda *shape: [torch.randn(t, *shape, generator=g) for t in TOTAL]
    q, k, v, beta = made(groups * dim), made(groups * dim), made(heads * vdim), made(heads)
    # decays from "keeps for hundreds" to "forgets at once", channel by channel, moving with the token
    rate = torch.exp(torch.linspace(-7.0, fast, heads * dim))[torch.randperm(heads * dim, generator=g)]
    log_decay = [-rate * torch.rand(t, heads * dim, generator=g) for t in TOTAL]
    return q, k, v, beta, log_decay


def plain_channels(q, k, v, beta, log_decay, heads, groups, dim, vdim, q_scale, delta):
    T = q.shape[0]
    spread = lambda x: x.double().view(T, groups, dim).repeat_interleave(heads // groups, dim=1)
    q, k, v, l = spread(q), spread(k), v.double().view(T, heads, vdim), log_decay.double().view(T, heads, dim)
    if delta:
        o = plain.delta_sums(plain.unit_vectors(q) * q_scale, plain.unit_vectors(k), v, plain.sigmoid(beta.double()), l)
    else:
        o = plain.channel_sums(q * q_scale, k, v, l)
    return o.reshape(T, -1)


def run_channels(case, heads, groups, dim, vdim, q_scale, delta, state, offset, at, counts):
    ops = kernels(torch.float32)
    q, k, v, beta, log_decay = (pieces(t, at, counts) for t in case)
    n = sum(counts)
    rows = torch.cat([q, k, v], dim=1)
    width = -(-rows.shape[1] // 4) * 4
    rows = torch.cat([rows, torch.full((n, width - rows.shape[1]), 1e9)], dim=1).cuda()
    beta_rows = torch.cat([torch.full((n, 3), 1e9), beta], dim=1).cuda()
    meta, _ = batch_meta(at, counts, SLOTS)
    out = torch.full((n, heads * vdim), 5.0, device="cuda")
    need = ops.channel_state_scratch(n, len(counts), max(counts), heads, dim, vdim, delta)
    more = dict(beta_rows=beta_rows, beta_at=3, unit_eps=1e-6) if delta else {}
    ops.channel_state(rows, 0, groups * dim, 2 * groups * dim, log_decay.contiguous().cuda(), out, state, meta, heads, groups, dim, vdim,
                      max(counts), torch.full((need,), 3e30, device="cuda"), q_scale=q_scale, state_offset=offset, **more)
    return out


@pytest.mark.parametrize("delta", [False, True])
@pytest.mark.parametrize("shape", CHANNEL_SHAPES)
def test_channel_state_over_portions_batches_and_used_slots(shape, delta):
    heads, groups, dim, vdim = shape
    case = channel_case(*shape, seed=dim)
    q_scale = dim ** -0.5
    refs = [plain_channels(*(t[i] for t in case), *shape, q_scale, delta) for i in range(3)]
    offset = 8
    state = used_state(offset + 2 * heads * dim * vdim)
    for at, counts in STEPS:
        out = run_channels(case, *shape, q_scale, delta, state, offset, at, counts)
        close(out, pieces(refs, at, counts), torch.float32, f"steps of {counts} from {at}")
        if max(counts) == 1:                        # a one-token step that runs again gives the same
            again = run_channels(case, *shape, q_scale, delta, state, offset, at, counts)
            assert torch.equal(out, again)
    untouched = state[[0, 3, 5]]
    assert bool((untouched == 1e30).all()) and bool((state[:, :offset] == 1e30).all())


@pytest.mark.parametrize("delta", [False, True])
def test_a_far_key_stays_in_a_slow_channel_and_leaves_a_fast_one(delta):
    """A key 400 tokens back in one channel that keeps and one that forgets, everything between writing elsewhere."""
    heads, dim, vdim, T = 2, 8, 4, 420
    k = torch.zeros(T, heads * dim)
    k.view(T, heads, dim)[:, :, 3:] = torch.randn(T, heads, dim - 3, generator=torch.Generator().manual_seed(1))
    k.view(T, heads, dim)[5, :, :] = 0.0
    k.view(T, heads, dim)[5, :, :2] = 1.0
    q = torch.zeros(T, heads * dim)
    q.view(T, heads, dim)[:, 0, 0] = 1.0             # head 0 asks for the slow channel, head 1 for the fast one
    q.view(T, heads, dim)[:, 1, 1] = 1.0
    v = torch.ones(T, heads * vdim)
    l = torch.full((T, heads * dim), -0.05)
    l.view(T, heads, dim)[:, :, 0], l.view(T, heads, dim)[:, :, 1] = -1e-4, -0.9
    beta = torch.full((T, heads), 3.0)
    ops = kernels(torch.float32)
    rows = torch.cat([q, k, v], dim=1).cuda()
    meta, _ = batch_meta([0], [T], [2])
    out = torch.empty(T, heads * vdim, device="cuda")
    need = ops.channel_state_scratch(T, 1, T, heads, dim, vdim, delta)
    more = dict(beta_rows=beta.cuda(), unit_eps=1e-6) if delta else {}
    ops.channel_state(rows, 0, heads * dim, 2 * heads * dim, l.cuda(), out, used_state(2 * heads * dim * vdim), meta, heads, heads, dim, vdim, T,
                      torch.empty(need, device="cuda"), **more)
    want = plain_channels(q, k, v, beta, l, heads, heads, dim, vdim, 1.0, delta)
    close(out, want, torch.float32, "far key")
    assert float(want[405, 0]) > 0.5 and abs(float(want[405, vdim])) < 1e-6


@pytest.mark.parametrize("delta", [False, True])
def test_channels_that_forget_everything_cost_no_precision(delta):
    """Log-decays down to -80 a token: every exponent is a sum of the numbers between, so what comes behind is exact."""
    shape = (2, 2, 24, 16)
    case = channel_case(*shape, seed=9, fast=math.log(80.0))
    for i in range(3):
        case[4][i][7::11] = -80.0                   # now and then all channels at once
    refs = [plain_channels(*(t[i] for t in case), *shape, 0.2, delta) for i in range(3)]
    state = used_state(2 * 2 * 24 * 16)
    at, counts = [0, 0, 0], TOTAL
    close(run_channels(case, *shape, 0.2, delta, state, 0, at, counts), pieces(refs, at, counts), torch.float32, "whole", 0.5)


def test_keys_that_come_again_are_overwritten():
    """The delta rule with beta near one and the same few keys again and again: the triangle inside a chunk has large entries,
    and what is read is the value written last."""
    heads, dim, vdim, T = 2, 16, 8, 130
    g = torch.Generator().manual_seed(4)
    basis = torch.linalg.qr(torch.randn(dim, dim, generator=g))[0]
    which = torch.randint(0, 3, (T,), generator=g)
    k = basis[which].repeat(1, heads)
    v = torch.randn(T, heads * vdim, generator=g)
    beta, l = torch.full((T, heads), 25.0), torch.zeros(T, heads * dim)
    ops = kernels(torch.float32)
    meta, _ = batch_meta([0], [T], [1])
    out = torch.empty(T, heads * vdim, device="cuda")
    need = ops.channel_state_scratch(T, 1, T, heads, dim, vdim, True)
    ops.channel_state(torch.cat([k, k, v], dim=1).cuda(), 0, heads * dim, 2 * heads * dim, l.cuda(), out, used_state(2 * heads * dim * vdim), meta,
                      heads, heads, dim, vdim, T, torch.empty(need, device="cuda"), beta_rows=beta.cuda(), unit_eps=1e-6)
    close(out, v, torch.float32, "the value written last")


# ---- exponential gates ------------------------------------------------------------------------------------------------------------
def gate_case(heads, dim, vdim, seed):
    g = torch.Generator().manual_seed(seed)
    made = lambda width, scale=1.0: [torch.randn(t, width, generator=g) * scale for t in TOTAL]
    return made(heads * dim), made(heads * dim), made(heads * vdim), made(heads, 3.0), made(heads, 3.0)


def plain_memory(q, k, v, i_logits, f_logits, P, cap, heads, dim, vdim):
    T = q.shape[0]
    eye = {"i": torch.eye(2 * heads, dtype=F64)[:heads], "f": torch.eye(2 * heads, dtype=F64)[heads:], "i.b": P["i.b"].double(), "f.b": P["f.b"].double()}
    i, f = plain.mlstm_gates(torch.cat([i_logits, f_logits], dim=1).double(), eye, "", {"gate_cap": cap})
    return plain.mlstm_memory(q.double().view(T, heads, dim) * dim ** -0.5, k.double().view(T, heads, dim), v.double().view(T, heads, vdim), i, f)


def memory_rows(case, at, counts):
    q, k, v, i, f = (pieces(t, at, counts) for t in case)
    rows = torch.cat([q, k, v, i, f], dim=1)
    return torch.cat([rows, torch.full((rows.shape[0], -rows.shape[1] % 4), 1e9)], dim=1).cuda()


@pytest.mark.parametrize("heads,dim,vdim", [(2, 16, 24), (3, 64, 64), (1, 128, 40), (3, 10, 8), (2, 5, 7), (1, 200, 130)])
def test_exponential_gates_and_the_denominator(heads, dim, vdim):
    cap = 5.0
    case = gate_case(heads, dim, vdim, dim)
    P = {"i.b": torch.linspace(-1.5, 1.0, heads), "f.b": torch.linspace(0.0, 4.0, heads)}
    refs = [plain_memory(*(t[s] for t in case), P, cap, heads, dim, vdim).reshape(TOTAL[s], -1) for s in range(3)]
    ops = kernels(torch.float32)
    half, offset = heads * dim * (vdim + 1), 4
    state = used_state(offset + 2 * half + 2 * heads)
    v_at, input_at = 2 * heads * dim, heads * (2 * dim + vdim)
    for at, counts in STEPS:
        rows = memory_rows(case, at, counts)
        n = rows.shape[0]
        meta, _ = batch_meta(at, counts, SLOTS)
        for _ in range(2 if max(counts) == 1 else 1):            # a one-token step that runs again gives the same
            log_decay, key_scale, floor = (torch.empty(n, heads, device="cuda") for _ in range(3))
            ops.exp_gates(rows, input_at, input_at + heads, P["i.b"].cuda(), P["f.b"].cuda(), cap, log_decay, key_scale, floor, meta, state,
                          offset + 2 * half)
            out = torch.full((n, heads * vdim), 5.0, device="cuda")
            need = ops.linear_state_scratch(3, max(counts), heads, dim, vdim, True)
            ops.linear_state(rows, 0, heads * dim, v_at, out, state, meta, heads, heads, dim, vdim, max(counts), log_decay=log_decay,
                             key_scale=key_scale, scratch=torch.full((need,), 3e30, device="cuda"), state_offset=offset,
                             out_scale=dim ** -0.5, floor=floor, floor_eps=1e-6)
            # where the keys' weights nearly cancel, the quotient is as sensitive as it is large
            close(out, pieces(refs, at, counts), torch.float32, f"steps of {counts} from {at}", 4.0)
    assert bool((state[[0, 3, 5]] == 1e30).all()) and bool((state[:, :offset] == 1e30).all())


def test_the_denominators_floor_and_the_maximums_start():
    """One key of weight w: o = v (k . q) w / max(|k . q| w, 1) whatever the gates did before; and input gates that stay below
    zero leave the maximum at the decayed start, where the floor exp(-m) counts."""
    heads, dim, vdim, T, cap = 1, 4, 3, 70, 15.0
    q, k, v = torch.zeros(T, dim), torch.zeros(T, dim), torch.randn(T, vdim, generator=torch.Generator().manual_seed(2))
    k[0, 0], q[:, 0] = 1.0, torch.linspace(0.1, 60.0, T)
    i, f = torch.full((T, 1), -3.0), torch.full((T, 1), 6.0)
    i[50:] = -30.0
    case = [[x] for x in (q, k, v, i, f)]
    P = {"i.b": torch.zeros(1), "f.b": torch.zeros(1)}
    want = plain_memory(q, k, v, i, f, P, cap, heads, dim, vdim).reshape(T, -1)
    gates = plain.mlstm_gates(torch.cat([i, f], dim=1).double(), {"i": torch.eye(2, dtype=F64)[:1], "f": torch.eye(2, dtype=F64)[1:], "i.b": torch.zeros(1, dtype=F64),
                                                                  "f.b": torch.zeros(1, dtype=F64)}, "", {"gate_cap": cap})
    kept = torch.exp(gates[0][0] + torch.cumsum(gates[1][:, 0], 0) - gates[1][0])           # the key's weight over time
    dots = q[:, 0].double() * dim ** -0.5 * kept
    by_hand = v[0].double() * (dots / torch.maximum(dots.abs(), torch.ones_like(dots)))[:, None]
    assert float((want - by_hand).abs().max()) < 1e-5 and float(dots.min()) < 0.1 and float(dots.max()) > 0.9
    ops = kernels(torch.float32)
    state, half = used_state(2 * dim * (vdim + 1) + 2), dim * (vdim + 1)
    rows, (meta, _) = memory_rows(case, [0], [T]), batch_meta([0], [T], [3])
    log_decay, key_scale, floor = (torch.empty(T, 1, device="cuda") for _ in range(3))
    ops.exp_gates(rows, 2 * dim + vdim, 2 * dim + vdim + 1, P["i.b"].cuda(), P["f.b"].cuda(), cap, log_decay, key_scale, floor, meta, state, 2 * half)
    out = torch.empty(T, vdim, device="cuda")
    ops.linear_state(rows, 0, dim, 2 * dim, out, state, meta, 1, 1, dim, vdim, T, log_decay=log_decay, key_scale=key_scale,
                     scratch=torch.empty(ops.linear_state_scratch(1, T, 1, dim, vdim, True), device="cuda"), out_scale=dim ** -0.5, floor=floor,
                     floor_eps=1e-6)
    close(out, want, torch.float32, "floor")


def test_gates_of_a_long_prompt_in_one_step():
    """More tokens than one round of the scan takes, with stretches where the maximum only decays."""
    heads, n, cap = 3, 2500, 6.0
    g = torch.Generator().manual_seed(6)
    logits = torch.randn(n, 2 * heads, generator=g) * 4.0
    logits[700:1500, :heads] = -50.0
    ops = kernels(torch.float32)
    meta, _ = batch_meta([0], [n], [1])
    log_decay, key_scale, floor = (torch.empty(n, heads, device="cuda") for _ in range(3))
    zeros = torch.zeros(heads, device="cuda")
    ops.exp_gates(logits.cuda(), 0, heads, zeros, zeros, cap, log_decay, key_scale, floor, meta, used_state(2 * heads), 0)
    i = cap * torch.tanh(logits[:, :heads].double() / cap)
    f = plain.log_sigmoid(cap * torch.tanh(logits[:, heads:].double() / cap))
    m, tops = torch.zeros(heads, dtype=F64), []
    for t in range(n):
        m = torch.maximum(f[t] + m, i[t])
        tops.append(m)
    tops = torch.stack(tops)
    before = torch.cat([torch.zeros(1, heads, dtype=F64), tops[:-1]])
    close(log_decay, f + before - tops, torch.float32, "decays")
    close(key_scale, torch.exp(i - tops), torch.float32, "key factors")
    close(floor / torch.exp(-tops).float().cuda(), torch.ones(n, heads), torch.float32, "floors")


# ---- the one-token kernel -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["channel", "delta", "exp"])
@pytest.mark.parametrize("shape", [(4, 2, 12, 8, 4, 6, 9), (2, 2, 64, 64, 3, 24, 16), (2, 1, 128, 132, 1, 5, 70), (3, 1, 7, 9, 10, 3, 1), (1, 1, 300, 21, 2, 2, 3),
                                   (1, 1, 16, 260, 4, 4, 4), (1, 1, 6, 270, 2, 3, 2)])
def test_one_token_at_a_time(dtype, kind, shape):
    """Forty tokens one by one in a batch of two used slots, every step run twice: convolution, decays, memory, norm and gate
    against the plain mixers with identity projections."""
    from stratakv_b200 import ops as O
    heads, groups, dim, vdim, taps, rank, gate_rank = shape
    if kind != "delta":
        groups = heads
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(dim + vdim)
    qk, hn, hv, T, eps = groups * dim, heads * dim, heads * vdim, 40, 1e-5
    widths = {"q": qk, "k": qk, "v": hv}
    if kind == "channel":
        widths.update(g=hv, a1=rank)
    elif kind == "delta":
        widths.update(b=heads, a1=rank, g1=gate_rank)
    else:
        widths.update(g=hv, i=heads, f=heads)
    total = sum(widths.values())
    places, at = {}, 0
    P = {}
    for name, width in widths.items():
        P[name] = torch.eye(total, dtype=F64)[at:at + width]
        places[name], at = at, at + width
    up = lambda r, c: (torch.randn(c, r, generator=g) / r ** 0.5 * 2.0).to(dtype)
    P["norm"] = (torch.rand(hv if kind == "exp" else vdim, generator=g) + 0.5).double()
    P["o"] = torch.eye(hv, dtype=F64)
    m = {"heads": heads, "kv_heads": groups, "dim": dim, "vdim": vdim, "tau": 3.0, "gate_cap": 4.0}
    more, decay_wt, gate_wt = {}, None, None
    if kind != "exp":
        P["a2"] = up(rank, hn).double()
        decay_wt = P["a2"].t().contiguous().to(dtype).cuda()
    if kind == "channel":
        P["a2.b"] = torch.randn(hn, generator=g).double() * 2.0
        more = dict(decay_bias=P["a2.b"].float().cuda(), decay_mode=O.LOW_RANK_LOG_SIGMOID, decay_factor=1.0 / 3.0, gate_silu=True)
    elif kind == "delta":
        P["g2"] = up(gate_rank, hv).double()
        gate_wt = P["g2"].t().contiguous().to(dtype).cuda()
        P["dt_bias"], P["A_log"] = torch.randn(hn, generator=g).double() - 2.0, torch.randn(heads, generator=g).double()
        for name in ("q", "k", "v"):
            P[name + ".conv"] = torch.randn(widths[name], taps, generator=g).double()
        conv_w = torch.cat([P[name + ".conv"] for name in ("q", "k", "v")]).float().cuda()
        more = dict(decay_bias=P["dt_bias"].float().cuda(), decay_mode=O.LOW_RANK_SOFTPLUS, decay_rate=torch.exp(P["A_log"]).float().cuda(),
                    unit_eps=1e-6, conv_w=conv_w, beta_at=places["b"])
    else:
        P["i.b"], P["f.b"] = torch.randn(heads, generator=g).double(), torch.rand(heads, generator=g).double() * 4.0
        more = dict(input_at=places["i"], forget_at=places["f"], input_bias=P["i.b"].float().cuda(), forget_bias=P["f.b"].float().cuda(), cap=4.0,
                    denominator_eps=1e-6)
    offset = 4
    matrix = 2 * heads * dim * (vdim + (1 if kind == "exp" else 0))
    floats = offset + matrix + (2 * heads if kind == "exp" else 0) + (taps * (2 * qk + hv) if kind == "delta" else 0)
    state = used_state(floats)
    rows = [torch.randn(T, total, generator=g) for _ in range(2)]
    norm = (P["norm"] if kind == "exp" else P["norm"].repeat(heads)).float().cuda()
    mixer = {"channel": plain.gla_mixer, "delta": plain.delta_side, "exp": plain.mlstm_mixer}[kind]
    refs = [mixer(r.double(), P, "", m, eps) for r in rows]
    gate_at = places["g1"] if kind == "delta" else places["g"]
    stride = -(-total // 4) * 4
    for t in range(T):
        step_rows = torch.full((2, stride), 1e9)
        step_rows[:, :total] = torch.stack([rows[1][t], rows[0][t]])
        meta, _ = batch_meta([t, t], [1, 1], [3, 1])
        outs = []
        for _ in range(2):
            out = torch.full((2, hv + 5), 7.0, dtype=dtype, device="cuda")
            ops.matrix_step({"channel": O.STEP_CHANNEL, "delta": O.STEP_DELTA, "exp": O.STEP_EXP}[kind], step_rows.cuda(), 0, qk, 2 * qk, out, state,
                            meta, heads, groups, dim, vdim, norm, eps, gate_at, q_scale=dim ** -0.5, ring_offset=offset + matrix,
                            decay_at=places.get("a1", 0), decay_wt=decay_wt, gate_wt=gate_wt, state_offset=offset, **more)
            outs.append(out)
        assert torch.equal(outs[0], outs[1]) and float(outs[0][:, hv:].float().abs().sum()) == 0.0
        close(outs[0][:, :hv], torch.stack([refs[1][t], refs[0][t]]), dtype, f"token {t}", 6.0 if dtype == torch.float32 else 1.0)
    assert bool((state[[0, 2, 4, 5]] == 1e30).all()) and bool((state[:, :offset] == 1e30).all())


# ---- what stands around -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,groups,size", [(3, 4, 20), (700, 4, 64), (2, 1, 7), (1500, 2, 260)])
def test_a_norm_per_head_with_either_gate(dtype, n, groups, size):
    from stratakv_b200 import ops as O
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(size)
    width = groups * size
    y, gate, weight = torch.randn(n, width, generator=g) * 3.0, torch.randn(n, width + 4, generator=g), torch.rand(width, generator=g) + 0.5
    unit = plain.unit_rms(y.double().view(n, groups, size), 1e-5).reshape(n, width) * weight.double()
    for mode, act in ((O.GATE_SIGMOID, plain.sigmoid), (O.GATE_SILU, plain.silu)):
        out = torch.empty(n, width + 4, dtype=dtype, device="cuda")
        ops.gated_norm(y.cuda(), gate.cuda()[:, 4:] if width % 4 else gate.cuda(), width + 4, weight.cuda(), groups, 1e-5, mode, out)
        z = gate[:, 4:] if width % 4 else gate[:, :width]
        close(out[:, :width], unit * act(z.double()), dtype, f"mode {mode}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,hidden", [(3, 64), (5, 44), (130, 1024), (2, 30)])
def test_the_stream_is_handed_on_as_it_is(dtype, n, hidden):
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(hidden)
    y, x, gamma = torch.randn(n, hidden, generator=g), torch.randn(n, hidden, generator=g), torch.rand(hidden, generator=g)
    stream, out = x.clone().cuda(), torch.empty(n, hidden, dtype=dtype, device="cuda")
    ops.rmsnorm_add(y.cuda(), gamma.cuda(), 1e-5, stream, next_out=out)
    want = x.double() + plain.rms_norm(y.double(), gamma.double(), 1e-5)
    close(stream, want, torch.float32, "stream")
    assert torch.equal(out, stream.to(dtype))


@pytest.mark.parametrize("n,width", [(3, 64), (5, 30), (300, 512)])
def test_output_bias_and_capped_logits(n, width):
    ops = kernels(torch.float32)
    g = torch.Generator().manual_seed(width)
    x, branch, bias = torch.randn(n, width, generator=g), torch.randn(n, width, generator=g), torch.randn(width, generator=g)
    for other in (branch, None):
        out = x.clone().cuda()
        ops.add_biased(out, other.cuda() if other is not None else None, bias.cuda(), 0.7)
        close(out, x.double() + 0.7 * ((other if other is not None else 0.0) + bias).double(), torch.float32, "bias")
    logits = (x * 40.0).cuda()
    ops.softcap_inplace(logits, 6.0)
    close(logits, plain.softcap((x * 40.0).double(), 6.0), torch.float32, "cap")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scale", [1.0, 60.0])
def test_router_shares_among_the_chosen(dtype, scale):
    """Also where logits lie so far apart that all shares but the first few are zero: the choice is made by the logits."""
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(3)
    n, hidden, experts, top = 50, 64, 11, 4
    h = torch.randn(n, hidden, generator=g).to(dtype)
    w = (torch.randn(experts, hidden, generator=g) * scale / hidden ** 0.5).to(dtype)
    chosen, weights = torch.empty(n, top, dtype=torch.int32, device="cuda"), torch.empty(n, top, device="cuda")
    ops.route_tokens(h.cuda(), w.cuda(), None, top, 1.0, True, chosen, weights, softmax=True)
    want, shares = plain.route(h.double(), {"router": w.double()}, "", {"experts": experts, "top": top})
    assert torch.equal(chosen.cpu().long(), want)
    close(weights, shares, torch.float32, "shares", 5.0 * scale)
    assert scale == 1.0 or float(torch.softmax(h.double() @ w.double().T, dim=-1).gather(1, want)[:, -1].min()) < 1e-45


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [3, 70])
def test_experts_and_a_gated_shared_expert(dtype, tokens):
    """The routed feed-forward part alone: chosen experts by their shares and the gated unit that every token uses."""
    from types import SimpleNamespace
    from stratakv_b200 import ops as O
    from stratakv_b200.parts.routed_mlp import RoutedMlp
    from stratakv_b200.parts.spec import RoutedMlpSpec, SharedExpertSpec
    ops = kernels(dtype)
    g = torch.Generator().manual_seed(8)
    hidden, ff, shared, experts, top = 64, 20, 44, 5, 2
    names = lambda part: tuple(f"e{e}.{part}" for e in range(experts))
    spec = RoutedMlpSpec(hidden, ff, experts, top, "silu", 1.0, "router", names("up"), names("down"), renormalize=True,
                         shared=SharedExpertSpec(shared, "shared.up", "shared.down", unit_gate_weight="shared.gate"), gate_weights=names("gate"), score="softmax")
    made = {name: (torch.randn(*request.shape, generator=g) * 0.2).to(dtype) for name, request in RoutedMlp.expected_tensors(spec).items()}
    scratch = {}

    def get(name, shape, kind):
        return scratch.setdefault((name, shape), torch.empty(shape, dtype=kind, device="cuda"))

    rt = SimpleNamespace(dtype=dtype, device=torch.device("cuda"), workspace=SimpleNamespace(get=get), kernels=lambda head_dim=None: ops,
                         upload=lambda t, kind=None: t.to("cuda", kind or dtype))
    part = RoutedMlp(spec, rt)
    part.bind(made)
    h = torch.randn(tokens, hidden, generator=g).to(dtype)
    x = torch.full((tokens, hidden), 3.0, device="cuda")
    part.forward(SimpleNamespace(choice_probe=None, store_branch=True), h.cuda(), x)
    want = plain.moe(h.double(), {name: t.double() for name, t in made.items()}, "", {"router": {"experts": experts, "top": top}, "shared": {"ff": shared}})
    close(x, want, dtype, "mixture")
