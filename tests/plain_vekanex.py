"""A plain, slow restatement of the Vekanex decoder: whole sequences, no cache, float64, one function per mechanism.
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


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-torch.abs(z)))


def log_sigmoid(z):
    return -softplus(-z)


# ---- matrix memory with exponential gates and a running maximum ------------------------------------------------------

def mlstm_gates(h, P, p, m):
    """The logarithms of the input and forget gates, [T, H] each."""
    cap = m["gate_cap"]
    i = cap * torch.tanh((h @ P[p + "i"].T + P[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ P[p + "f"].T + P[p + "f.b"]) / cap))
    return i, f


def mlstm_memory(q, k, v, i, f):
    """o [T, H, dv]; q, k [T, H, n], v [T, H, dv], i, f [T, H]."""
    T, H, n = k.shape
    S, z, top = torch.zeros(H, n, v.shape[2], dtype=F64), torch.zeros(H, n, dtype=F64), torch.zeros(H, dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        new_top = torch.maximum(f[t] + top, i[t])
        keep, take = torch.exp(f[t] + top - new_top), torch.exp(i[t] - new_top)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z = keep[:, None] * z + take[:, None] * k[t]
        top = new_top
        weight = torch.maximum(torch.abs((z * q[t]).sum(dim=-1)), torch.exp(-top)) + 1e-6
        o[t] = torch.einsum("hn,hnd->hd", q[t], S) / weight[:, None]
    return o


def mlstm_mixer(h, P, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = (h @ P[p + "q"].T).view(T, H, m["dim"]) * m["dim"] ** -0.5
    k = (h @ P[p + "k"].T).view(T, H, m["dim"])
    v = (h @ P[p + "v"].T).view(T, H, m["vdim"])
    o = mlstm_memory(q, k, v, *mlstm_gates(h, P, p, m))
    o = unit_rms(o, eps).reshape(T, -1) * P[p + "norm"] * sigmoid(h @ P[p + "g"].T)
    return o @ P[p + "o"].T


# ---- gated linear attention -------------------------------------------------------------------------------------------

def gla_log_decay(h, P, p, m):
    """[T, H, n]: the logarithm of every key channel's decay."""
    z = (h @ P[p + "a1"].T) @ P[p + "a2"].T + P[p + "a2.b"]
    return (log_sigmoid(z) / m["tau"]).view(h.shape[0], m["heads"], m["dim"])


def channel_sums(q, k, v, log_decay):
    """S_t = diag(exp(l_t)) S_(t-1) + k_t v_t^T from S = 0, o_t = S_t^T q_t.  q, k, l [T, H, n], v [T, H, dv]."""
    T, H, n = k.shape
    S = torch.zeros(H, n, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = torch.exp(log_decay[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hn,hnd->hd", q[t], S)
    return o


def gla_mixer(h, P, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = (h @ P[p + "q"].T).view(T, H, m["dim"]) * m["dim"] ** -0.5
    k = (h @ P[p + "k"].T).view(T, H, m["dim"])
    v = (h @ P[p + "v"].T).view(T, H, m["vdim"])
    o = channel_sums(q, k, v, gla_log_decay(h, P, p, m))
    o = rms_norm(o, P[p + "norm"], eps).reshape(T, -1) * silu(h @ P[p + "g"].T)
    return o @ P[p + "o"].T


# ---- the parallel mixer, left: softmax attention ------------------------------------------------------------------------

def rotate_halves(x, positions, rot):
    """x [T, heads, d]: of the first rot.dims numbers of a head, i turns with i + dims/2."""
    dims = rot["dims"]
    half = dims // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    angle = positions.to(F64)[:, None] * f[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def attention_inputs(h, P, p, m, eps, positions=None):
    """Rotated queries [T, H, d], rotated keys [T, G, d] and values [T, G, dv]."""
    T = h.shape[0]
    positions = torch.arange(T) if positions is None else positions
    project = lambda name: h @ P[p + name].T + P[p + name + ".b"]
    q = rms_norm(project("q"), P[p + "q.norm"], eps).view(T, m["heads"], m["dim"])
    k = rms_norm(project("k"), P[p + "k.norm"], eps).view(T, m["kv_heads"], m["dim"])
    return (rotate_halves(q, positions, m["rot"]), rotate_halves(k, positions, m["rot"]),
            project("v").view(T, m["kv_heads"], m["vdim"]))


def attend(q, k, v, scale):
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for head in range(H):
        g = head // (H // G)
        scores = ((q[:, head] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        out[:, head] = torch.softmax(scores, dim=-1) @ v[:, g]
    return out


def attention_side(h, P, p, m, eps):
    q, k, v = attention_inputs(h, P, p, m, eps)
    return attend(q, k, v, m["scale"]).reshape(h.shape[0], -1) @ P[p + "o"].T + P[p + "o.b"]


# ---- the parallel mixer, right: the gated delta rule ----------------------------------------------------------------------

def causal_convolution(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the sequence."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_inputs(h, P, p, m):
    """q, k [T, H, n] (spread over the heads that share them), v [T, H, dv], beta [T, H], log decay [T, H, n]."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    conv = lambda name: silu(causal_convolution(h @ P[p + name].T, P[p + name + ".conv"]))
    spread = lambda x: x.repeat_interleave(H // G, dim=1)
    q = spread(unit_vectors(conv("q").view(T, G, m["dim"]))) * m["dim"] ** -0.5
    k = spread(unit_vectors(conv("k").view(T, G, m["dim"])))
    v = conv("v").view(T, H, m["vdim"])
    beta = sigmoid(h @ P[p + "b"].T)
    step = softplus((h @ P[p + "a1"].T) @ P[p + "a2"].T + P[p + "dt_bias"]).view(T, H, m["dim"])
    return q, k, v, beta, -torch.exp(P[p + "A_log"])[:, None] * step


def delta_sums(q, k, v, beta, log_decay):
    """The state decays, what it already says about the key is taken off the value, the rest is written, then read."""
    T, H, n = k.shape
    S = torch.zeros(H, n, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = torch.exp(log_decay[t])[:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hn,hnd->hd", k[t], S))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hn,hnd->hd", q[t], S)
    return o


def delta_side(h, P, p, m, eps):
    T = h.shape[0]
    o = rms_norm(delta_sums(*delta_inputs(h, P, p, m)), P[p + "norm"], eps).reshape(T, -1)
    return (o * sigmoid((h @ P[p + "g1"].T) @ P[p + "g2"].T)) @ P[p + "o"].T


def parallel_mixer(h, P, p, m, eps):
    return (m["left_scale"] * attention_side(h, P, p + "left.", m["left"], eps)
            + m["right_scale"] * delta_side(h, P, p + "right.", m["right"], eps))


MIXERS = {"mlstm": mlstm_mixer, "gla": gla_mixer, "parallel": parallel_mixer}


# ---- the feed-forward ---------------------------------------------------------------------------------------------

# Where the engine computes in bfloat16 its router sees a rounded input, and where two experts score nearly alike it may
# choose the other one: that is no fault.  ``proposed`` ([T, top] expert indices, -1 where unknown) is the engine's
# choice; it is followed where its experts' logits add up to at most CLOSE_CALL less than the plain choice's do, and
# counted in FAR_CALLS otherwise (DECISIONS counts all choices that were compared).  float32 runs follow nobody.
CLOSE_CALL = 0.15
FAR_CALLS, DECISIONS = [], [0]


def route(h, P, p, router, proposed=None):
    """Per token: the chosen experts and their weights, a softmax over the chosen ones' logits."""
    z = h @ P[p + "router"].T
    chosen = z.topk(router["top"], dim=-1).indices
    if proposed is not None:
        DECISIONS[0] += z.shape[0]
        for t in range(z.shape[0]):
            theirs = proposed[t]
            if int(theirs.min()) < 0 or set(theirs.tolist()) == set(chosen[t].tolist()):
                continue
            if float(z[t, chosen[t]].sum() - z[t, theirs].sum()) <= CLOSE_CALL:
                chosen[t] = theirs
            else:
                FAR_CALLS.append((p, t))
    return chosen, torch.softmax(z.gather(1, chosen), dim=-1)


def expert(h, P, p):
    return (silu(h @ P[p + "gate"].T) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def moe(h, P, p, mlp, proposed=None):
    chosen, weights = route(h, P, p, mlp["router"], proposed)
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, c = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            y.index_add_(0, t, weights[t, c][:, None] * expert(h[t], P, f"{p}e{e}."))
    return y + expert(h, P, p + "shared.") if mlp.get("shared") else y


# ---- the model ------------------------------------------------------------------------------------------------------

def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while "weights_of" in cfg["layers"][i]:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer(x, cfg, P, i, proposed=None):
    spec, p = cfg["layers"][i], f"l{owner(cfg, i)}."
    eps, share = cfg["norm"]["eps"], cfg["residual_mult"]
    x = x + share * rms_norm(MIXERS[spec["type"]](x, P, p + "mix.", spec["mixer"], eps), P[p + "norm1"], eps)
    if spec.get("mlp"):
        x = x + share * rms_norm(moe(x, P, p + "mlp.", spec["mlp"], proposed), P[p + "norm2"], eps)
    return x


def softcap(logits, cap):
    return cap * torch.tanh(logits / cap) if cap else logits


def forward(cfg, P, tokens, layer_outputs=None, proposed=None):
    """Logits [T, vocab] of one sequence; ``layer_outputs`` (a list) gets the stream after every layer; ``proposed``:
    layer -> the experts another implementation chose there (see ``route``)."""
    x = P["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, P, i, proposed.get(i) if proposed else None)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return softcap(rms_norm(x, P["final.norm"], cfg["norm"]["eps"]) @ P["head"].T, cfg.get("logit_softcap"))


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
