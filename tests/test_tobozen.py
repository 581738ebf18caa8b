"""The Tobozen decoder on the CPU: its configuration and refusals, tensor names and cache entries, hand-worked numbers for
the mechanisms of the plain implementation (tests/plain_tobozen.py), that a fault in any mechanism moves the plain logits
by far more than rounding, and the engine's bookkeeping (portions, batches, slots, pages and states used again, steps
that run twice) with torch stand-ins for the kernels (tests/ops_double.py)."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_tobozen as plain
from helpers import random_tokens
from ops_double import double_loader
from stratakv_b200 import Engine, EngineConfig, StepEntry
from stratakv_b200.config import ConfigError, TobozenConfig, load_config
from stratakv_b200.engine.model import cache_requests, default_head_dim, expected_tensors
from stratakv_b200.models.tobozen import tobozen_spec
from stratakv_b200.weights.loader import load_checkpoint
from tobozen_models import TOBOZEN, make_folder

F64 = torch.float64


def test_configuration_round_trip_and_refusals():
    for raw in TOBOZEN.values():
        typed = TobozenConfig.from_dict(raw)
        assert TobozenConfig.from_dict(typed.to_dict()) == typed
    ta = TobozenConfig.from_dict(TOBOZEN["TA"])
    assert (ta.vocab, ta.width, ta.norm_eps, ta.norm_groups) == (101, 64, 1e-5, 4)
    assert ta.layers[0].mixer.v_mix and ta.layers[0].mixer.rot_dims == 12 and ta.layers[0].mlp.limit == 0.7
    assert ta.layers[1].mixer.taps == 4 and ta.layers[1].mixer.norm_groups == 3 and ta.layers[2].mlp is None
    assert ta.layers[3].mixer.decay == (0.5, 0.93, 0.998)
    plain_norm = copy.deepcopy(TOBOZEN["TA"])
    del plain_norm["norm"]["groups"]
    assert TobozenConfig.from_dict(plain_norm).norm_groups == 1

    def broken(change):
        raw = copy.deepcopy(TOBOZEN["TA"])
        change(raw)
        with pytest.raises(ConfigError):
            TobozenConfig.from_dict(raw)

    broken(lambda r: r["layers"][0].update(type="retention"))
    broken(lambda r: r["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda r: r["layers"][0]["mixer"]["rot"].update(dims=7))
    broken(lambda r: r["layers"][0]["mixer"]["rot"].update(dims=18))
    broken(lambda r: r["layers"][0]["mixer"].update(vdim=20))              # the mixing layers' values differ in number
    broken(lambda r: r["layers"][0]["mixer"].update(v_mix=1))
    broken(lambda r: r["layers"][0]["mixer"].update(scale=0.0))
    broken(lambda r: r["layers"][0]["mlp"]["router"].update(top=7))
    broken(lambda r: r["layers"][0]["mlp"]["expert"].update(limit=0.0))
    broken(lambda r: r["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda r: r["layers"][1]["mixer"].update(groups=3))
    broken(lambda r: r["layers"][1]["mixer"].update(norm_groups=5))
    broken(lambda r: r["layers"][1]["mixer"].update(conv=0))
    broken(lambda r: r["layers"][3]["mixer"].update(decay=[0.5, 0.9]))
    broken(lambda r: r["layers"][3]["mixer"].update(decay=[0.5, 0.9, 1.5]))
    broken(lambda r: r["norm"].update(groups=3))
    broken(lambda r: r.pop("norm"))
    broken(lambda r: r.update(layers=[]))


def test_tensor_names_and_cache_entries():
    spec = tobozen_spec(TobozenConfig.from_dict(TOBOZEN["TA"]))
    shapes = {name: tuple(request.shape) for name, request in expected_tensors(spec).items()}
    assert shapes["embed"] == (101, 64) and "head" not in shapes and shapes["final.norm"] == (64,)
    assert shapes["l0.mix.q"] == (64, 64) and shapes["l0.mix.k"] == (32, 64) and shapes["l0.mix.v"] == (48, 64)
    assert shapes["l0.mix.q.norm"] == (64,) and shapes["l0.mix.k.norm"] == (32,) and shapes["l0.mix.o"] == (64, 96)
    assert "l0.mix.vmix" not in shapes and "l0.mix.vmix" in spec.ignorable and shapes["l2.mix.vmix"] == ()
    assert shapes["l1.mix.in"] == (2 * 48 + 2 * 16 + 4, 64) and shapes["l1.mix.conv"] == (80, 4) and shapes["l1.mix.conv.b"] == (80,)
    assert shapes["l1.mix.dt_bias"] == shapes["l1.mix.A_log"] == shapes["l1.mix.D"] == (4,) and shapes["l1.mix.norm"] == (48,)
    assert "l2.norm2" not in shapes and "l2.mlp.router" not in shapes and "l2.norm2" in spec.ignorable
    assert shapes["l3.mix.q"] == (36, 64) and shapes["l3.mix.v"] == shapes["l3.mix.g"] == (60, 64) and shapes["l3.mix.norm"] == (60,)
    assert shapes["l3.mlp.e4.down"] == (64, 20) and "l3.mlp.e5.up" not in shapes and shapes["l3.mlp.router"] == (5, 64)
    requests = cache_requests(spec)
    assert [r.kind for r in requests] == ["kv", "none", "kv", "none"]
    # heads of at most 64 numbers are cached 64 wide; S twice and the last four inputs; S twice
    assert (requests[0].num_kv_heads, requests[0].head_dim, requests[0].v_head_dim) == (2, 64, 0)
    assert requests[1].state_bytes == 4 * (2 * 4 * 8 * 12 + 4 * 80) and requests[3].state_bytes == 4 * 2 * 3 * 12 * 20
    tc, td = (tobozen_spec(TobozenConfig.from_dict(TOBOZEN[n])) for n in ("TC", "TD"))
    assert [r.head_dim for r in cache_requests(tc)] == [64, 0, 0, 128, 128] and default_head_dim(tc) == 64
    wide = cache_requests(td)[1]
    assert (wide.head_dim, wide.v_head_dim) == (144, 136)              # wider than any compiled kernel: as they are
    # a layer that mixes values takes those of the first one that does, whatever lies between
    tb = tobozen_spec(TobozenConfig.from_dict(TOBOZEN["TB"]))
    assert [(l.mixer.keeps_values, l.mixer.value_mix) for l in tb.layers if l.mixer.kind == "normed_attention"] == \
        [(False, None), (True, None), (False, "l5.mix.vmix")]


# ---- hand-worked numbers for the plain implementation ---------------------------------------------------------------

def test_grouped_norm_by_hand():
    x = torch.tensor([[3.0, 4.0, 0.0, 2.0]], dtype=F64)
    y = plain.grouped_norm(x, torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=F64), 2, 0.5)
    a, b = math.sqrt(12.5 + 0.5), math.sqrt(2.0 + 0.5)
    np.testing.assert_allclose(y.numpy(), [[3 / a, 8 / a, 0.0, 1 / b]], rtol=1e-12)


def test_rotation_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0, 6.0]]], dtype=F64).repeat(2, 1, 1)
    out = plain.rotate_pairs(x, torch.tensor([0, 3]), {"dims": 4, "base": 100.0})
    assert torch.equal(out[0], x[0])
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    want = [math.cos(a0) - 2 * math.sin(a0), 2 * math.cos(a0) + math.sin(a0),
            3 * math.cos(a1) - 4 * math.sin(a1), 4 * math.cos(a1) + 3 * math.sin(a1), 5.0, 6.0]
    np.testing.assert_allclose(out[1, 0].numpy(), want, rtol=1e-12)


def test_softmax_with_one_more_by_hand():
    weights = plain.softmax_plus_one(torch.tensor([[0.0, math.log(2.0), -math.inf], [-900.0, -900.0, -900.0]], dtype=F64))
    np.testing.assert_allclose(weights[0].numpy(), [1 / 4, 2 / 4, 0.0], rtol=1e-12)
    assert float(weights[1].sum()) == pytest.approx(0.0, abs=1e-300)        # nothing worth looking at: next to no weight


def test_values_are_mixed_by_hand():
    P = {"x.vmix": torch.tensor(0.25, dtype=F64)}
    v, first = torch.tensor([[4.0, 8.0]], dtype=F64), torch.tensor([[0.0, 16.0]], dtype=F64)
    assert plain.mixed_values(v, P, "x.", first).tolist() == [[3.0, 10.0]]
    assert plain.mixed_values(v, P, "x.", None).tolist() == [[4.0, 8.0]]


def test_decayed_sums_as_an_explicit_sum():
    torch.manual_seed(1)
    q, k, v = torch.randn(6, 2, 3, dtype=F64), torch.randn(6, 2, 3, dtype=F64), torch.randn(6, 2, 4, dtype=F64)
    d = torch.rand(6, 2, dtype=F64)
    o = plain.decayed_sums(q, k, v, d)
    for t in (0, 2, 5):
        for head in range(2):
            want = sum((q[t, head] @ k[s, head]) * d[s + 1:t + 1, head].prod() * v[s, head] for s in range(t + 1))
            np.testing.assert_allclose(o[t, head].numpy(), want.numpy(), rtol=1e-9, atol=1e-12)


def test_mamba2_inputs_by_hand():
    """One head, one number each: the layout of the input projection, the convolution with bias and silu, the step size."""
    m = {"heads": 1, "vdim": 1, "state": 1, "groups": 1, "conv": 2, "norm_groups": 1}
    P = {"x.in": torch.tensor([[1.0], [2.0], [3.0], [4.0], [5.0]], dtype=F64), "x.conv.b": torch.tensor([0.5, 0.0, -1.0], dtype=F64),
         "x.conv": torch.tensor([[10.0, 1.0], [0.0, 1.0], [1.0, 1.0]], dtype=F64), "x.dt_bias": torch.tensor([-2.0], dtype=F64)}
    z, x, B, C, dt = plain.mamba2_inputs(torch.tensor([[1.0], [0.1]], dtype=F64), P, "x.", m)
    silu = lambda u: u / (1.0 + math.exp(-u))
    np.testing.assert_allclose(z[:, 0].numpy(), [1.0, 0.1])
    np.testing.assert_allclose(x[:, 0, 0].numpy(), [silu(0.5 + 2.0), silu(0.5 + 20.0 + 0.2)])
    np.testing.assert_allclose(B[:, 0, 0].numpy(), [silu(3.0), silu(0.3)])
    np.testing.assert_allclose(C[:, 0, 0].numpy(), [silu(-1.0 + 4.0), silu(-1.0 + 4.0 + 0.4)])
    np.testing.assert_allclose(dt[:, 0].numpy(), [math.log1p(math.exp(3.0)), math.log1p(math.exp(0.5 - 2.0))])
    P.update({"x.A_log": torch.tensor([math.log(2.0)], dtype=F64), "x.D": torch.tensor([3.0], dtype=F64)})
    y = plain.mamba2_sums(x, B, C, dt, P, "x.")
    s0 = dt[0, 0] * B[0, 0, 0] * x[0, 0, 0]
    s1 = torch.exp(-2.0 * dt[1, 0]) * s0 + dt[1, 0] * B[1, 0, 0] * x[1, 0, 0]
    np.testing.assert_allclose(y[:, 0, 0].numpy(), [float(s0 * C[0, 0, 0] + 3 * x[0, 0, 0]), float(s1 * C[1, 0, 0] + 3 * x[1, 0, 0])])


def test_an_expert_and_its_weight_by_hand():
    P = {"x.gate": torch.tensor([[1.0], [1.0]], dtype=F64), "x.up": torch.tensor([[1.0], [-1.0]], dtype=F64),
         "x.down": torch.eye(2, dtype=F64)}
    g = 2.0 / (1.0 + math.exp(-1.702 * 2.0))
    np.testing.assert_allclose(plain.expert(torch.tensor([[3.0]], dtype=F64), P, "x.", 2.0).numpy(), [[g * 3.0, g * -1.0]], rtol=1e-12)
    # the weight goes into the expert: with a score of one half its input is halved, which its output is not
    Q = {"m.router": torch.zeros(1, 1, dtype=F64), **{"m.e0." + n[2:]: t for n, t in P.items()}}
    Q["m.e0.down"] = torch.tensor([[1.0, 0.0]], dtype=F64)
    mlp = {"expert": {"limit": 2.0}, "router": {"experts": 1, "top": 1}}
    g = 1.5 / (1.0 + math.exp(-1.702 * 1.5))
    np.testing.assert_allclose(plain.moe(torch.tensor([[3.0]], dtype=F64), Q, "m.", mlp).numpy(), [[g * 2.5]], rtol=1e-12)


def test_routing_by_hand():
    logits = torch.tensor([[0.1, 2.0, -1.0, 0.5]], dtype=F64)
    chosen, weights = plain.route(logits, {"x.router": torch.eye(4, dtype=F64)}, "x.", {"experts": 4, "top": 2})
    assert chosen.tolist() == [[1, 3]]
    np.testing.assert_allclose(weights.numpy(), [[1 / (1 + math.exp(-2.0)), 1 / (1 + math.exp(-0.5))]], rtol=1e-12)


def _mixed_first(cfg, P):
    """A later layer mixes in nobody's values."""
    P["l2.mix.vmix"] = torch.zeros_like(P["l2.mix.vmix"])


FAULTS = {
    "the norm's groups": lambda cfg, P: cfg["norm"].update(groups=1),
    "the query norm's weight": lambda cfg, P: P.update({"l0.mix.q.norm": torch.ones_like(P["l0.mix.q.norm"])}),
    "the key norm's weight": lambda cfg, P: P.update({"l2.mix.k.norm": torch.ones_like(P["l2.mix.k.norm"])}),
    "the rotated part, two numbers off": lambda cfg, P: cfg["layers"][0]["mixer"]["rot"].update(dims=10),
    "the scale": lambda cfg, P: cfg["layers"][2]["mixer"].update(scale=0.3),
    "the mixed values": _mixed_first,
    "the convolution's oldest tap": lambda cfg, P: P["l1.mix.conv"].__setitem__((slice(None), 0), 0.0),
    "the convolution's bias": lambda cfg, P: P.update({"l1.mix.conv.b": torch.zeros_like(P["l1.mix.conv.b"])}),
    "the step sizes' bias": lambda cfg, P: P.update({"l1.mix.dt_bias": torch.zeros_like(P["l1.mix.dt_bias"])}),
    "the skip": lambda cfg, P: P.update({"l1.mix.D": torch.zeros_like(P["l1.mix.D"])}),
    "the gated norm's groups": lambda cfg, P: cfg["layers"][1]["mixer"].update(norm_groups=1),
    "a slow decay": lambda cfg, P: cfg["layers"][3]["mixer"]["decay"].__setitem__(2, 0.9),
    "the gate of the linear attention": lambda cfg, P: P.update({"l3.mix.g": torch.zeros_like(P["l3.mix.g"])}),
    "the experts' clamp": lambda cfg, P: cfg["layers"][0]["mlp"]["expert"].update(limit=2.0),
    "one expert fewer": lambda cfg, P: cfg["layers"][3]["mlp"]["router"].update(top=2),
}


@pytest.mark.parametrize("fault", list(FAULTS))
def test_a_fault_moves_the_plain_logits_far_more_than_rounding(tmp_path, fault):
    folder = make_folder(tmp_path / "TA", TOBOZEN["TA"], seed=2)
    cfg, P = plain.load_folder(folder)
    tokens = random_tokens(101, 48, seed=5)
    ref = plain.logits_of(cfg, P, tokens)
    cfg, P = copy.deepcopy(cfg), {k: v.clone() for k, v in P.items()}
    FAULTS[fault](cfg, P)
    moved = plain.logits_of(cfg, P, tokens)
    per_position = np.sqrt(((moved - ref) ** 2).mean(axis=-1)) / ref.std()
    assert per_position.max() > 0.1, f"{fault}: the logits move by {per_position.max():.3f} of their spread only"


@pytest.mark.parametrize("fault", ["the one in the denominator", "the weight on the input"])
def test_a_fault_of_the_design_itself_moves_the_plain_logits(tmp_path, fault, monkeypatch):
    folder = make_folder(tmp_path / "TA", TOBOZEN["TA"], seed=2)
    cfg, P = plain.load_folder(folder)
    tokens = random_tokens(101, 48, seed=5)
    ref = plain.logits_of(cfg, P, tokens)
    if fault == "the one in the denominator":
        monkeypatch.setattr(plain, "softmax_plus_one", lambda scores: torch.softmax(scores, dim=-1))
    else:
        def weighed_output(h, P, p, mlp, proposed=None):
            chosen, weights = plain.route(h, P, p, mlp["router"], proposed)
            y = torch.zeros_like(h)
            for t in range(h.shape[0]):
                for e, w in zip(chosen[t].tolist(), weights[t]):
                    y[t] += w * plain.expert(h[t:t + 1], P, f"{p}e{e}.", mlp["expert"]["limit"])[0]
            return y
        monkeypatch.setattr(plain, "moe", weighed_output)
    per_position = np.sqrt(((plain.logits_of(cfg, P, tokens) - ref) ** 2).mean(axis=-1)) / ref.std()
    assert per_position.max() > 0.1, f"{fault}: the logits move by {per_position.max():.3f} of their spread only"


# ---- the engine's bookkeeping, with stand-ins for the kernels ---------------------------------------------------------

def cpu_engine(folder, max_tokens=512, block_size=16, max_batch=0):
    arch, config = load_config(folder)
    spec = arch.build_spec(config)
    tensors = load_checkpoint(folder, {n: r.shape for n, r in expected_tensors(spec).items()}, spec.ignorable)
    return Engine(spec, tensors, EngineConfig(max_tokens=max_tokens, dtype="float32", device="cpu", block_size=block_size,
                                              max_batch=max_batch), kernel_loader=double_loader())


def near(got, want):
    np.testing.assert_allclose(got, want, rtol=2e-4, atol=2e-4)


@pytest.mark.parametrize("name", list(TOBOZEN))
def test_bookkeeping_portions_batches_and_slots_used_again(tmp_path, name):
    folder = make_folder(tmp_path / name, TOBOZEN[name], seed=3)
    cfg, P = plain.load_folder(folder)
    engine = cpu_engine(folder, max_tokens=16 * 14, max_batch=3)
    vocab = TOBOZEN[name]["vocab"]
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


@pytest.mark.parametrize("name", ["TA", "TB"])
def test_a_step_that_runs_twice_leaves_the_states_as_one_run_does(tmp_path, name):
    """A decode graph's warm-up and its first replay run the same one-token step twice: no state a step reads (the
    matrices, the convolution's last inputs) is one that it writes."""
    folder = make_folder(tmp_path / name, TOBOZEN[name], seed=4)
    cfg, P = plain.load_folder(folder)
    engine = cpu_engine(folder)
    tokens = random_tokens(TOBOZEN[name]["vocab"], 14, seed=1)
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


def test_a_checkpoint_without_the_share_nobody_reads_loads_as_well(tmp_path):
    from stratakv_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
    folder = make_folder(tmp_path / "TA", TOBOZEN["TA"], seed=2)
    handle = SafetensorsFile(folder / "model.safetensors")
    tensors = {n: handle.tensor(n).clone() for n in handle.names() if n != "l0.mix.vmix"}
    write_safetensors(folder / "model.safetensors", tensors)
    cpu_engine(folder)
    del tensors["l2.mix.vmix"]
    write_safetensors(folder / "model.safetensors", tensors)
    with pytest.raises(ValueError, match="l2.mix.vmix"):
        cpu_engine(folder)
