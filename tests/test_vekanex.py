"""The Vekanex decoder on the CPU: its configuration and refusals, tensor names and cache entries, hand-worked numbers for
the mechanisms of the plain implementation (tests/plain_vekanex.py), that a fault in any mechanism moves the plain logits
by far more than rounding, and the engine's bookkeeping (portions, batches, slots, pages and states used again, steps
that run twice, layers that use another's tensors) with torch stand-ins for the kernels (tests/ops_double.py)."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_vekanex as plain
from helpers import random_tokens
from ops_double import double_loader
from stratakv_b200 import Engine, EngineConfig, StepEntry
from stratakv_b200.config import ConfigError, VekanexConfig, load_config
from stratakv_b200.engine.model import cache_requests, default_head_dim, expected_tensors
from stratakv_b200.models.vekanex import vekanex_spec
from stratakv_b200.weights.loader import load_checkpoint
from vekanex_models import VEKANEX, make_folder

F64 = torch.float64


def near12(got, want):
    np.testing.assert_allclose(np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64), rtol=1e-12, atol=1e-300)


def test_configuration_round_trip_and_refusals():
    for raw in VEKANEX.values():
        typed = VekanexConfig.from_dict(raw)
        assert VekanexConfig.from_dict(typed.to_dict()) == typed
    va, vb = VekanexConfig.from_dict(VEKANEX["VA"]), VekanexConfig.from_dict(VEKANEX["VB"])
    assert (va.vocab, va.width, va.norm_eps, va.residual_mult, va.logit_softcap) == (101, 64, 1e-5, 0.6, 6.0)
    assert va.layers[0].mixer.tau == 4.0 and va.layers[1].mixer.left.rot_dims == 12 and va.layers[1].mixer.right.taps == 4
    assert va.layers[2].mlp is None and va.layers[0].mlp.shared_ff == 40 and vb.layers[0].mlp.shared_ff == 0
    assert [va.owner(i) for i in range(5)] == [0, 1, 2, 1, 2] and vb.logit_softcap == 0.0

    def broken(change):
        raw = copy.deepcopy(VEKANEX["VA"])
        change(raw)
        with pytest.raises(ConfigError):
            VekanexConfig.from_dict(raw)

    left = lambda r: r["layers"][1]["mixer"]["left"]
    broken(lambda r: r["layers"][0].update(type="retention"))
    broken(lambda r: left(r).update(kv_heads=3))
    broken(lambda r: left(r)["rot"].update(dims=7))
    broken(lambda r: left(r)["rot"].update(dims=18))
    broken(lambda r: left(r).pop("scale"))
    broken(lambda r: r["layers"][1]["mixer"]["right"].update(kv_heads=3))
    broken(lambda r: r["layers"][1]["mixer"]["right"].update(conv=0))
    broken(lambda r: r["layers"][1]["mixer"].pop("right"))
    broken(lambda r: r["layers"][0]["mixer"].update(tau=0.0))
    broken(lambda r: r["layers"][2]["mixer"].update(gate_cap=0.0))
    broken(lambda r: r["layers"][0]["mlp"]["router"].update(top=7))
    broken(lambda r: r["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda r: r["layers"][0]["mlp"]["shared"].update(ff=0))
    broken(lambda r: r["layers"][4]["mixer"].update(vdim=20))              # no longer the layer whose tensors it uses
    broken(lambda r: r["layers"][4].update(weights_of=4))
    broken(lambda r: r["layers"][4].update(weights_of=9))
    broken(lambda r: r.update(logit_softcap=-1.0))
    broken(lambda r: r.pop("norm"))
    broken(lambda r: r.update(layers=[]))


def test_ranks_come_from_the_checkpoint(tmp_path):
    folder = make_folder(tmp_path / "VA", VEKANEX["VA"], seed=1)
    arch, config = load_config(folder)
    assert config.layers[0].mixer.rank == 5 and (config.layers[3].mixer.right.decay_rank, config.layers[3].mixer.right.gate_rank) == (6, 9)
    import json
    bare = VekanexConfig.from_dict(json.loads((folder / "config.json").read_text()))
    assert bare.needs_tensor_shapes() and not config.needs_tensor_shapes()
    with pytest.raises(ValueError, match="rank"):
        vekanex_spec(bare)
    with pytest.raises(ConfigError, match="l0.mix.a1"):
        bare.with_tensor_shapes({})


def test_tensor_names_and_cache_entries():
    spec = vekanex_spec(VekanexConfig.from_dict(VEKANEX["VA"]))
    shapes = {name: tuple(request.shape) for name, request in expected_tensors(spec).items()}
    assert shapes["embed"] == shapes["head"] == (101, 64) and shapes["final.norm"] == (64,)
    assert shapes["l0.mix.q"] == (36, 64) and shapes["l0.mix.v"] == shapes["l0.mix.g"] == (60, 64) and shapes["l0.mix.norm"] == (20,)
    assert shapes["l0.mix.a1"] == (5, 64) and shapes["l0.mix.a2"] == (36, 5) and shapes["l0.mix.a2.b"] == (36,)
    assert shapes["l0.mlp.shared.gate"] == (40, 64) and shapes["l0.mlp.e5.down"] == (64, 24) and "l0.mlp.e6.up" not in shapes
    assert shapes["l1.mix.left.q.b"] == shapes["l1.mix.left.q.norm"] == (64,) and shapes["l1.mix.left.o"] == (64, 96)
    assert shapes["l1.mix.left.k.norm"] == (32,) and shapes["l1.mix.left.v.b"] == (48,) and shapes["l1.mix.left.o.b"] == (64,)
    assert shapes["l1.mix.right.q.conv"] == shapes["l1.mix.right.k.conv"] == (24, 4) and shapes["l1.mix.right.v.conv"] == (32, 4)
    assert shapes["l1.mix.right.b"] == (4, 64) and shapes["l1.mix.right.A_log"] == (4,) and shapes["l1.mix.right.dt_bias"] == (48,)
    assert shapes["l1.mix.right.a2"] == (48, 6) and shapes["l1.mix.right.g2"] == (32, 9) and shapes["l1.mix.right.norm"] == (8,)
    assert shapes["l2.mix.i"] == (2, 64) and shapes["l2.mix.f.b"] == (2,) and shapes["l2.mix.norm"] == (48,)
    assert "l2.norm2" not in shapes and "l2.norm2" in spec.ignorable
    assert not any(name.startswith(("l3.", "l4.")) for name in shapes)
    assert len(spec.layers) == 3 and [(e.layer, e.cache) for e in spec.schedule] == [(0, 0), (1, 1), (2, 2), (1, 3), (2, 4)]
    requests = cache_requests(spec)
    assert [r.kind for r in requests] == ["none", "kv", "none", "kv", "none"] and requests[1] == requests[3]
    # S twice; heads of at most 64 numbers cached 64 wide, S twice and the last four inputs; S and n twice, m twice
    assert requests[0].state_bytes == 4 * 2 * 3 * 12 * 20
    assert (requests[1].num_kv_heads, requests[1].head_dim) == (2, 64)
    assert requests[1].state_bytes == 4 * (2 * 4 * 12 * 8 + 4 * 80)
    assert requests[2].state_bytes == 4 * (2 * 2 * 16 * 25 + 4)
    vc, vd = (vekanex_spec(VekanexConfig.from_dict(VEKANEX[n])) for n in ("VC", "VD"))
    assert [r.head_dim for r in cache_requests(vc)] == [64, 0, 0, 128, 0] and default_head_dim(vc) == 64
    wide = cache_requests(vd)[0]
    assert (wide.head_dim, wide.v_head_dim) == (144, 136)              # wider than any compiled kernel: as they are


# ---- hand-worked numbers for the plain implementation ---------------------------------------------------------------

def test_exponential_gates_and_memory_by_hand():
    """One head, one number each: the maximum starts at 0, the floor counts, then the memory's own weight does."""
    v = lambda *x: torch.tensor(x, dtype=F64).view(-1, 1, 1)
    gates = lambda *x: torch.tensor(x, dtype=F64).view(-1, 1)
    i, f = gates(-2.0, 3.0), gates(-0.5, -1.0)
    o = plain.mlstm_memory(v(0.5, 2.0), v(3.0, 1.0), v(4.0, -6.0), i, f)
    m1 = -0.5                                                     # max(-0.5 + 0, -2): not -2, as from minus infinity
    s1, n1 = math.exp(-2 - m1) * 12.0, math.exp(-2 - m1) * 3.0
    near12(o[0, 0, 0], s1 * 0.5 / (max(abs(n1 * 0.5), math.exp(0.5)) + 1e-6))
    assert n1 * 0.5 < math.exp(0.5)
    m2 = 3.0
    s2, n2 = math.exp(-1 + m1 - m2) * s1 - 6.0, math.exp(-1 + m1 - m2) * n1 + 1.0
    near12(o[1, 0, 0], s2 * 2.0 / (max(abs(n2 * 2.0), math.exp(-3.0)) + 1e-6))
    P = {"x.i": torch.tensor([[2.0]], dtype=F64), "x.i.b": torch.tensor([1.0], dtype=F64),
         "x.f": torch.tensor([[-4.0]], dtype=F64), "x.f.b": torch.tensor([0.5], dtype=F64)}
    i, f = plain.mlstm_gates(torch.tensor([[3.0]], dtype=F64), P, "x.", {"gate_cap": 5.0})
    near12(i[0, 0], 5 * math.tanh(7 / 5))
    near12(f[0, 0], -math.log1p(math.exp(5 * math.tanh(11.5 / 5))))


def test_the_memory_does_not_depend_on_how_it_is_scaled():
    """Away from the 1e-6: o is sum_j w_j v_j / max(|sum_j w_j|, 1) with w_j = exp(i_j + f_(j+1) + .. + f_t) (k_j . q_t)."""
    torch.manual_seed(3)
    T, n = 7, 3
    q, k, v = (torch.randn(T, 1, n, dtype=F64) for _ in range(3))
    i, f = torch.randn(T, 1, dtype=F64) * 2, plain.log_sigmoid(torch.randn(T, 1, dtype=F64) + 1)
    o = plain.mlstm_memory(q, k, v, i, f)
    for t in range(T):
        w = torch.stack([torch.exp(i[j, 0] + f[j + 1:t + 1, 0].sum()) * (k[j, 0] @ q[t, 0]) for j in range(t + 1)])
        want = (w[:, None] * v[:t + 1, 0]).sum(dim=0) / max(abs(float(w.sum())), 1.0)
        np.testing.assert_allclose(o[t, 0].numpy(), want.numpy(), rtol=2e-5)


def test_channel_decays_by_hand():
    P = {"x.a1": torch.tensor([[2.0]], dtype=F64), "x.a2": torch.tensor([[1.0], [-3.0]], dtype=F64), "x.a2.b": torch.tensor([0.5, 0.0], dtype=F64)}
    l = plain.gla_log_decay(torch.tensor([[1.0]], dtype=F64), P, "x.", {"heads": 1, "dim": 2, "tau": 4.0})
    near12(torch.exp(l).flatten(), [(1 / (1 + math.exp(-2.5))) ** 0.25, (1 / (1 + math.exp(6.0))) ** 0.25])
    torch.manual_seed(1)
    q, k, l = torch.randn(5, 1, 3, dtype=F64), torch.randn(5, 1, 3, dtype=F64), -torch.rand(5, 1, 3, dtype=F64)
    v = torch.randn(5, 1, 2, dtype=F64)
    o = plain.channel_sums(q, k, v, l)
    for t in range(5):
        want = sum((q[t, 0] * k[j, 0] * torch.exp(l[j + 1:t + 1, 0].sum(dim=0))).sum() * v[j, 0] for j in range(t + 1))
        np.testing.assert_allclose(o[t, 0].numpy(), want.numpy(), rtol=1e-10)


def test_the_delta_rule_by_hand():
    one = lambda *x: torch.tensor(x, dtype=F64).view(-1, 1, 1)
    o = plain.delta_sums(one(2.0, 3.0), one(1.0, 0.5), one(4.0, 10.0), torch.tensor([[0.25], [0.5]], dtype=F64), one(math.log(0.5), math.log(0.8)))
    s1 = 0.25 * 4.0
    s2 = 0.8 * s1 + 0.5 * (0.5 * (10.0 - 0.5 * 0.8 * s1))
    near12(o.flatten(), [2.0 * s1, 3.0 * s2])
    # a key that is written again with beta one is overwritten, whatever was there
    k = torch.tensor([0.6, 0.8], dtype=F64).view(1, 1, 2).repeat(2, 1, 1)
    o = plain.delta_sums(k, k, one(4.0, -7.0), torch.ones(2, 1, dtype=F64), torch.zeros(2, 1, 2, dtype=F64))
    near12(o.flatten(), [4.0, -7.0])


def test_delta_inputs_by_hand():
    """Two value heads on one key head of one number: convolution, silu, unit length, step sizes."""
    m = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1}
    t = lambda *x: torch.tensor(x, dtype=F64)
    P = {"x.q": t([1.0]), "x.q.conv": t([0.5, 2.0]), "x.k": t([-1.0]), "x.k.conv": t([0.0, 1.0]), "x.v": t([1.0], [2.0]),
         "x.v.conv": t([0.0, 1.0], [1.0, 1.0]), "x.b": t([1.0], [0.0]), "x.a1": t([3.0]), "x.a2": t([1.0], [0.5]), "x.dt_bias": t(0.0, -1.0),
         "x.A_log": t(math.log(2.0), 0.0)}
    q, k, v, beta, l = plain.delta_inputs(t([1.0], [0.1]), P, "x.", m)
    silu = lambda u: u / (1 + math.exp(-u))
    unit = lambda u: u / math.sqrt(u * u + 1e-6)
    near12(q[:, 0, 0], [unit(silu(2.0)), unit(silu(0.5 + 0.2))])
    near12(k[:, 1, 0], [unit(silu(-1.0)), unit(silu(-0.1))])
    near12(v[:, 1, 0], [silu(2.0), silu(2.0 + 0.2)])
    near12(beta[0], [1 / (1 + math.exp(-1.0)), 0.5])
    near12(l[0, :, 0], [-2 * math.log1p(math.exp(3.0)), -math.log1p(math.exp(0.5))])


def test_rotation_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0, 6.0]]], dtype=F64).repeat(2, 1, 1)
    out = plain.rotate_halves(x, torch.tensor([0, 3]), {"dims": 4, "base": 100.0})
    assert torch.equal(out[0], x[0])
    a, b = 3.0, 3.0 * 100.0 ** -0.5
    near12(out[1, 0], [math.cos(a) - 3 * math.sin(a), 2 * math.cos(b) - 4 * math.sin(b), 3 * math.cos(a) + math.sin(a),
                       4 * math.cos(b) + 2 * math.sin(b), 5.0, 6.0])


def test_routing_and_experts_by_hand():
    logits = torch.tensor([[0.1, 2.0, -1.0, 0.5]], dtype=F64)
    chosen, weights = plain.route(logits, {"x.router": torch.eye(4, dtype=F64)}, "x.", {"experts": 4, "top": 2})
    assert chosen.tolist() == [[1, 3]]
    near12(weights, [[math.exp(2.0) / (math.exp(2.0) + math.exp(0.5)), math.exp(0.5) / (math.exp(2.0) + math.exp(0.5))]])
    P = {"m.router": torch.zeros(1, 1, dtype=F64)}
    for part, (g, u, d) in {"e0": (1.0, 2.0, 3.0), "shared": (-1.0, 1.0, 5.0)}.items():
        P.update({f"m.{part}.gate": torch.tensor([[g]], dtype=F64), f"m.{part}.up": torch.tensor([[u]], dtype=F64), f"m.{part}.down": torch.tensor([[d]], dtype=F64)})
    silu = lambda u: u / (1 + math.exp(-u))
    near12(plain.moe(torch.tensor([[2.0]], dtype=F64), P, "m.", {"router": {"experts": 1, "top": 1}, "shared": {"ff": 1}}),
           [[3 * silu(2.0) * 4.0 + 5 * silu(-2.0) * 2.0]])
    near12(plain.softcap(torch.tensor([3.0, -40.0], dtype=F64), 5.0), [5 * math.tanh(0.6), 5 * math.tanh(-8.0)])


# ---- a fault shows ---------------------------------------------------------------------------------------------------

def _set(name, value):
    return lambda cfg, P: P.update({name: torch.full_like(P[name], value)})


FAULTS = {
    "the factor on what joins the stream": lambda cfg, P: cfg.update(residual_mult=0.5),
    "the cap on the logits": lambda cfg, P: cfg.pop("logit_softcap"),
    "the first norm's weight": _set("l0.norm1", 1.0),
    "the second norm's weight": _set("l1.norm2", 1.0),
    "the channels' decay exponent": lambda cfg, P: cfg["layers"][0]["mixer"].update(tau=5.0),
    "the channels' decay bias": _set("l0.mix.a2.b", 0.0),
    "the linear attention's gate": _set("l0.mix.g", 0.1),
    "the gates' cap": lambda cfg, P: [cfg["layers"][i]["mixer"].update(gate_cap=2.0) for i in (2, 4)],
    "the input gates": _set("l2.mix.i", 0.0),
    "the forget gates' bias": _set("l2.mix.f.b", 0.0),
    "the memory's norm": _set("l2.mix.norm", 1.0),
    "the query projection's bias": _set("l1.mix.left.q.b", 0.0),
    "the value projection's bias": _set("l1.mix.left.v.b", 0.0),
    "the output projection's bias": _set("l1.mix.left.o.b", 0.0),
    "the query norm's weight": _set("l1.mix.left.q.norm", 1.0),
    "the key norm's weight": _set("l1.mix.left.k.norm", 1.0),
    "the rotated part, two numbers off": lambda cfg, P: [cfg["layers"][i]["mixer"]["left"]["rot"].update(dims=10) for i in (1, 3)],
    "the score's scale": lambda cfg, P: [cfg["layers"][i]["mixer"]["left"].update(scale=0.3) for i in (1, 3)],
    "the convolution's oldest tap": lambda cfg, P: P["l1.mix.right.v.conv"].__setitem__((slice(None), 0), 0.0),
    "the step sizes' bias": _set("l1.mix.right.dt_bias", 0.0),
    "the heads' rates": _set("l1.mix.right.A_log", 0.0),
    "beta": _set("l1.mix.right.b", 0.0),
    "the delta rule's norm": _set("l1.mix.right.norm", 1.0),
    "the low-rank gate": _set("l1.mix.right.g1", 0.0),
    "the right side's share": lambda cfg, P: [cfg["layers"][i]["mixer"].update(right_scale=0.6) for i in (1, 3)],
    "the shared expert": lambda cfg, P: cfg["layers"][0]["mlp"].pop("shared"),
    "one expert fewer": lambda cfg, P: cfg["layers"][0]["mlp"]["router"].update(top=1),
}


@pytest.fixture(scope="module")
def model_va(tmp_path_factory):
    cfg, P = plain.load_folder(make_folder(tmp_path_factory.mktemp("va"), VEKANEX["VA"], seed=2))
    tokens = random_tokens(101, 48, seed=5)
    return cfg, P, tokens, plain.logits_of(cfg, P, tokens)


def moves(moved, ref, fault):
    per_position = np.sqrt(((moved - ref) ** 2).mean(axis=-1)) / ref.std()
    assert per_position.max() > 0.1, f"{fault}: the logits move by {per_position.max():.3f} of their spread only"


@pytest.mark.parametrize("fault", list(FAULTS))
def test_a_fault_moves_the_plain_logits_far_more_than_rounding(model_va, fault):
    cfg, P, tokens, ref = model_va
    cfg, P = copy.deepcopy(cfg), {k: v.clone() for k, v in P.items()}
    FAULTS[fault](cfg, P)
    moves(plain.logits_of(cfg, P, tokens), ref, fault)


def _read_first(q, k, v, beta, log_decay):
    """A token reads the state before it has written its own share."""
    T, H, n = k.shape
    S = torch.zeros(H, n, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = torch.exp(log_decay[t])[:, :, None] * S
        o[t] = torch.einsum("hn,hnd->hd", q[t], S)
        S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - torch.einsum("hn,hnd->hd", k[t], S)))[:, None, :]
    return o


def _decay_last(q, k, v, beta, log_decay):
    """What the state says about the key is taken before the decay."""
    T, H, n = k.shape
    S = torch.zeros(H, n, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        u = beta[t][:, None] * (v[t] - torch.einsum("hn,hnd->hd", k[t], S))
        S = torch.exp(log_decay[t])[:, :, None] * S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hn,hnd->hd", q[t], S)
    return o


def _norm_per_head(h, P, p, m, eps, positions=None):
    T = h.shape[0]
    project = lambda name, heads, width: (h @ P[p + name].T + P[p + name + ".b"]).view(T, heads, width)
    q = plain.unit_rms(project("q", m["heads"], m["dim"]), eps) * P[p + "q.norm"].view(m["heads"], -1)
    k = plain.unit_rms(project("k", m["kv_heads"], m["dim"]), eps) * P[p + "k.norm"].view(m["kv_heads"], -1)
    at = torch.arange(T)
    return plain.rotate_halves(q, at, m["rot"]), plain.rotate_halves(k, at, m["rot"]), project("v", m["kv_heads"], m["vdim"])


def _all_experts(h, P, p, router, proposed=None, plain_route=plain.route):
    """Shares out of a softmax over all experts."""
    chosen, _ = plain_route(h, P, p, router, proposed)
    return chosen, torch.softmax(h @ P[p + "router"].T, dim=-1).gather(1, chosen)


def _norm_in_front(x, cfg, P, i, proposed=None):
    spec, p = cfg["layers"][i], f"l{plain.owner(cfg, i)}."
    eps, share = cfg["norm"]["eps"], cfg["residual_mult"]
    x = x + share * plain.MIXERS[spec["type"]](plain.rms_norm(x, P[p + "norm1"], eps), P, p + "mix.", spec["mixer"], eps)
    return x + share * plain.moe(plain.rms_norm(x, P[p + "norm2"], eps), P, p + "mlp.", spec["mlp"]) if spec.get("mlp") else x


# (the denominator of an exponential-gate memory hardly shows in the logits, since every head is divided by its root mean
# square right behind it: its numbers are held by hand above and on the kernels in test_vekanex_kernels_gpu.py)
DESIGN_FAULTS = {"the write before the read": ("delta_sums", _read_first),
                 "the decay before the delta": ("delta_sums", _decay_last), "one norm over all heads": ("attention_inputs", _norm_per_head),
                 "shares among the chosen": ("route", _all_experts), "norms behind the sublayers": ("layer", _norm_in_front),
                 "unit vectors": ("unit_vectors", lambda x: x)}


@pytest.mark.parametrize("fault", list(DESIGN_FAULTS))
def test_a_fault_of_the_design_itself_moves_the_plain_logits(model_va, fault, monkeypatch):
    cfg, P, tokens, ref = model_va
    monkeypatch.setattr(plain, *DESIGN_FAULTS[fault])
    moves(plain.logits_of(cfg, P, tokens), ref, fault)


# ---- the engine's bookkeeping, with stand-ins for the kernels ---------------------------------------------------------

def cpu_engine(folder, max_tokens=512, block_size=16, max_batch=0):
    arch, config = load_config(folder)
    spec = arch.build_spec(config)
    tensors = load_checkpoint(folder, {n: r.shape for n, r in expected_tensors(spec).items()}, spec.ignorable)
    return Engine(spec, tensors, EngineConfig(max_tokens=max_tokens, dtype="float32", device="cpu", block_size=block_size,
                                              max_batch=max_batch), kernel_loader=double_loader())


def near(got, want):
    np.testing.assert_allclose(got, want, rtol=3e-4, atol=3e-4)


@pytest.mark.parametrize("name", list(VEKANEX))
def test_bookkeeping_portions_batches_and_slots_used_again(tmp_path, name):
    folder = make_folder(tmp_path / name, VEKANEX[name], seed=3)
    cfg, P = plain.load_folder(folder)
    engine = cpu_engine(folder, max_tokens=16 * 14, max_batch=3)
    vocab = VEKANEX[name]["vocab"]
    for turn in range(2):                     # the second turn takes the slots, pages and states of the first
        prompts = [random_tokens(vocab, n, seed=10 * turn + n) for n in (5, 40, 18)]
        refs = [plain.logits_of(cfg, P, p) for p in prompts]
        slots = [engine.open_sequence() for _ in prompts]
        cut = [1, 20, 17]
        got = engine.step([StepEntry(s, p[:c], list(range(c))) for s, p, c in zip(slots, prompts, cut)])
        near(got.numpy(), np.concatenate([r[:c] for r, c in zip(refs, cut)]))
        got = engine.step([StepEntry(slots[0], prompts[0][1:], [3]), StepEntry(slots[1], prompts[1][20:22], [0, 1]),
                           StepEntry(slots[2], prompts[2][17:], [0])])
        near(got.numpy(), np.stack([refs[0][4], refs[1][20], refs[1][21], refs[2][17]]))
        engine.close_sequence(slots[0]); engine.close_sequence(slots[2])
        for position in range(22, 40):
            near(engine.step([StepEntry(slots[1], [prompts[1][position]], [0])]).numpy()[0], refs[1][position])
        engine.close_sequence(slots[1])
        assert engine.cache.all_free()


@pytest.mark.parametrize("name", ["VA", "VB"])
def test_a_step_that_runs_twice_leaves_the_states_as_one_run_does(tmp_path, name):
    """A decode graph's warm-up and its first replay run the same one-token step twice: no state a step reads (matrices, key
    sums, maxima, the convolution's last inputs) is one that it writes."""
    folder = make_folder(tmp_path / name, VEKANEX[name], seed=4)
    cfg, P = plain.load_folder(folder)
    engine = cpu_engine(folder)
    tokens = random_tokens(VEKANEX[name]["vocab"], 14, seed=1)
    ref = plain.logits_of(cfg, P, tokens)
    slot = engine.open_sequence()
    engine.step([StepEntry(slot, tokens[:6], [])])
    rows = torch.tensor([0], dtype=torch.int32)
    for position in range(6, 14):
        step, _, _ = engine.prepare([StepEntry(slot, [tokens[position]], [0])])
        first = engine.model.forward(step, rows, 1).clone()
        second = engine.model.forward(step, rows, 1).clone()
        engine.cache.advance(slot, position + 1)
        near(first.numpy()[0], ref[position])
        np.testing.assert_allclose(second.numpy(), first.numpy(), rtol=0, atol=0)
    engine.close_sequence(slot)


def test_a_normed_attention_alone_adds_its_output_bias(tmp_path):
    """The pair adds the left side's output bias with its weight where it does not take the result straight into the stream
    (VB's first parallel layer has a left weight of one, its second has not)."""
    folder = make_folder(tmp_path / "VB", VEKANEX["VB"], seed=6)
    engine = cpu_engine(folder)
    sides = [layer.mixer.left for layer in engine.model.layers if hasattr(layer.mixer, "left")]
    assert [side.leaves_output_bias for side in sides] == [False, True]


def test_a_missing_tensor_of_the_shared_expert_is_named(tmp_path):
    from stratakv_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
    folder = make_folder(tmp_path / "VA", VEKANEX["VA"], seed=2)
    handle = SafetensorsFile(folder / "model.safetensors")
    tensors = {n: handle.tensor(n).clone() for n in handle.names() if n != "l1.mlp.shared.gate"}
    write_safetensors(folder / "model.safetensors", tensors)
    with pytest.raises(ValueError, match="l1.mlp.shared.gate"):
        cpu_engine(folder)
