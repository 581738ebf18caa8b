"""A plain, slow restatement of the Tobozen decoder: whole sequences, no cache, float64, one function per mechanism.
It shares no code with the library; the GPU tests compare the engine with it.

Notation: a sequence of T tokens at positions 0..T-1, width W.  ``P`` maps tensor names to float64 tensors, ``cfg`` is
the dictionary of a ``config.json`` of this design, ``p`` a tensor prefix (``"l3.mix."``), ``m`` a mixer's section of
the configuration.
"""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch

F64 = torch.float64


def unit_rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def grouped_norm(x, weight, groups, eps):
    """The last axis in ``groups`` equal parts, each divided by its own root mean square; then the weight."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return unit_rms(parts, eps).reshape(x.shape) * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-torch.abs(z)))


# ---- the attention mixer ------------------------------------------------------------------------------------------

def rotate_pairs(x, positions, rot):
    """x [T, heads, n]: of the first rot.dims numbers of a head, 2i and 2i + 1 turn together."""
    dims = rot["dims"]
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    angle = positions.to(F64)[:, None] * f[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def softmax_plus_one(scores):
    """Rows of scores (-inf where unseen): exp(s_j) / (1 + sum_j exp(s_j))."""
    top = scores.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(-top))


def mixed_values(v, P, p, first):
    """The layer's values with those of the first mixing layer taken in; ``first`` None: this is that layer."""
    return v if first is None else (1.0 - P[p + "vmix"]) * v + P[p + "vmix"] * first


def attention_inputs(h, P, p, m, eps, first=None, positions=None):
    """Rotated queries [T, H, d], rotated keys [T, G, d], mixed values [T, G, dv], and the values before mixing."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    positions = torch.arange(T) if positions is None else positions
    q = grouped_norm(h @ P[p + "q"].T, P[p + "q.norm"], 1, eps).view(T, H, m["dim"])
    k = grouped_norm(h @ P[p + "k"].T, P[p + "k.norm"], 1, eps).view(T, G, m["dim"])
    own = h @ P[p + "v"].T
    v = mixed_values(own, P, p, first) if m.get("v_mix") else own
    return rotate_pairs(q, positions, m["rot"]), rotate_pairs(k, positions, m["rot"]), v.view(T, G, m["vdim"]), own


def attend(q, k, v, scale):
    """Causal grouped-query attention with one added to every denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for head in range(H):
        g = head // (H // G)
        scores = ((q[:, head] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        out[:, head] = softmax_plus_one(scores) @ v[:, g]
    return out


def attention_mixer(h, P, p, m, eps, shared):
    """``shared`` (a dict of one forward pass) holds the values of the first layer that mixes values."""
    first = shared.get("first") if m.get("v_mix") else None
    q, k, v, own = attention_inputs(h, P, p, m, eps, first)
    if m.get("v_mix") and first is None:
        shared["first"] = own
    return attend(q, k, v, m["scale"]).reshape(h.shape[0], -1) @ P[p + "o"].T


# ---- the recurrent mixers -------------------------------------------------------------------------------------------

def decayed_sums(q, k, v, decay):
    """S_t = decay_t S_(t-1) + k_t v_t^T from S = 0, o_t = S_t^T q_t.  q, k [T, H, n], v [T, H, dv], decay [T, H]."""
    T, H, n = k.shape
    S = torch.zeros(H, n, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = decay[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hi,hij->hj", q[t], S)
    return o


def causal_convolution(u, w, b):
    """u [T, C], w [C, taps], b [C]: y_t = b + sum_j w[:, j] u_(t - taps + 1 + j), zeros before the sequence."""
    T, taps = u.shape[0], w.shape[1]
    y = b.expand(T, -1).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def mamba2_inputs(h, P, p, m):
    """z [T, inner], x [T, H, dv], B and C [T, G, N], the step sizes [T, H]."""
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, gn = H * dv, G * N
    row = h @ P[p + "in"].T
    z, xbc, dt = row[:, :inner], row[:, inner:2 * inner + 2 * gn], row[:, 2 * inner + 2 * gn:]
    xbc = silu(causal_convolution(xbc, P[p + "conv"], P[p + "conv.b"]))
    return (z, xbc[:, :inner].view(T, H, dv), xbc[:, inner:inner + gn].view(T, G, N), xbc[:, inner + gn:].view(T, G, N),
            softplus(dt + P[p + "dt_bias"]))


def mamba2_sums(x, B, C, dt, P, p):
    """y [T, H, dv]: the recurrence and the skip."""
    per_group = x.shape[1] // B.shape[1]
    B, C = B.repeat_interleave(per_group, dim=1), C.repeat_interleave(per_group, dim=1)
    decay = torch.exp(-torch.exp(P[p + "A_log"]) * dt)
    return decayed_sums(C, dt[:, :, None] * B, x, decay) + P[p + "D"][:, None] * x


def mamba2_mixer(h, P, p, m, eps):
    z, x, B, C, dt = mamba2_inputs(h, P, p, m)
    y = mamba2_sums(x, B, C, dt, P, p).reshape(h.shape[0], -1) * silu(z)
    return grouped_norm(y, P[p + "norm"], m["norm_groups"], eps) @ P[p + "o"].T


def lightning_mixer(h, P, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = silu(h @ P[p + "q"].T).view(T, H, m["dim"])
    k = silu(h @ P[p + "k"].T).view(T, H, m["dim"])
    v = silu(h @ P[p + "v"].T).view(T, H, m["vdim"])
    o = decayed_sums(q, k, v, torch.tensor(m["decay"], dtype=F64).expand(T, H))
    o = grouped_norm(o.reshape(T, -1), P[p + "norm"], 1, eps) * sigmoid(h @ P[p + "g"].T)
    return o @ P[p + "o"].T


# ---- the feed-forward ---------------------------------------------------------------------------------------------

# Where the engine computes in bfloat16 its router sees a rounded input, and where two experts score nearly alike it may
# choose the other one: that is no fault.  ``proposed`` ([T, top] expert indices, -1 where unknown) is the engine's
# choice; it is followed where its experts' scores add up to at least CLOSE_CALL of what the plain choice's do, and
# counted in FAR_CALLS otherwise (DECISIONS counts all choices that were compared).  float32 runs follow nobody.
CLOSE_CALL = 0.85
FAR_CALLS, DECISIONS = [], [0]


def route(h, P, p, router, proposed=None):
    """Per token: the chosen experts and their weights (the scores as they are)."""
    s = sigmoid(h @ P[p + "router"].T)
    chosen = s.topk(router["top"], dim=-1).indices
    if proposed is not None:
        DECISIONS[0] += s.shape[0]
        for t in range(s.shape[0]):
            theirs = proposed[t]
            if int(theirs.min()) < 0 or set(theirs.tolist()) == set(chosen[t].tolist()):
                continue
            if float(s[t, theirs].sum()) >= CLOSE_CALL * float(s[t, chosen[t]].sum()):
                chosen[t] = theirs
            else:
                FAR_CALLS.append((p, t))
    return chosen, s.gather(1, chosen)


def expert(h, P, p, limit):
    g = torch.clamp(h @ P[p + "gate"].T, max=limit)
    u = torch.clamp(h @ P[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ P[p + "down"].T


def moe(h, P, p, mlp, proposed=None):
    """The chosen experts of the weighted input, added up."""
    chosen, weights = route(h, P, p, mlp["router"], proposed)
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, k = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            y.index_add_(0, t, expert(weights[t, k][:, None] * h[t], P, f"{p}e{e}.", mlp["expert"]["limit"]))
    return y


# ---- the model ------------------------------------------------------------------------------------------------------

def layer(x, cfg, P, i, shared, proposed=None):
    spec, p = cfg["layers"][i], f"l{i}."
    eps, groups = cfg["norm"]["eps"], cfg["norm"].get("groups", 1)
    h = grouped_norm(x, P[p + "norm1"], groups, eps)
    if spec["type"] == "attention":
        x = x + attention_mixer(h, P, p + "mix.", spec["mixer"], eps, shared)
    elif spec["type"] == "mamba2":
        x = x + mamba2_mixer(h, P, p + "mix.", spec["mixer"], eps)
    else:
        x = x + lightning_mixer(h, P, p + "mix.", spec["mixer"], eps)
    if spec.get("mlp"):
        x = x + moe(grouped_norm(x, P[p + "norm2"], groups, eps), P, p + "mlp.", spec["mlp"], proposed)
    return x


def forward(cfg, P, tokens, layer_outputs=None, proposed=None):
    """Logits [T, vocab] of one sequence; ``layer_outputs`` (a list) gets the stream after every layer; ``proposed``:
    layer -> the experts another implementation chose there (see ``route``)."""
    x = P["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    shared = {}
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, P, i, shared, proposed.get(i) if proposed else None)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return grouped_norm(x, P["final.norm"], cfg["norm"].get("groups", 1), cfg["norm"]["eps"]) @ P["embed"].T


def load_folder(folder):
    """``(cfg, P)`` of a model folder; floating tensors widened to float64."""
    import numpy as np
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    size = int.from_bytes(raw[:8], "little")
    header = json.loads(raw[8:8 + size])
    data = raw[8 + size:]
    P = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        chunk = np.frombuffer(data[lo:hi], dtype=np.uint8)
        if info["dtype"] == "BF16":
            value = torch.from_numpy((chunk.view(np.uint16).astype(np.uint32) << 16).view(np.float32).copy())
        elif info["dtype"] == "F32":
            value = torch.from_numpy(chunk.view(np.float32).copy())
        else:
            raise ValueError(f"{name}: dtype {info['dtype']}")
        P[name] = value.view(info["shape"]).to(F64)
    return cfg, P


def logits_of(cfg, P, tokens, proposed=None):
    return forward(cfg, P, tokens, proposed=proposed).to(torch.float32).numpy()
