"""Small Tobozen configurations for the tests, and folders with random weights for them.

The weights are drawn so that a fault shows: attention scores a few units apart around zero (so that the one in the
softmax's denominator counts, and a key that is lost or taken from another page moves the logits by far more than rounding
does), values that differ between the layers that mix them, decays of the recurrent layers from "forgets in a few tokens"
to "keeps for hundreds", step sizes that move with the token, gates away from their middle, norms' weights between 0.4
and 1.6, experts that differ and router scores a few tenths apart.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch


def moe(ff, limit, experts, top):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def attention(heads, kv_heads, dim, vdim, scale, rot, v_mix, mlp):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
             "rot": {"dims": rot[0], "base": rot[1]}}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def mamba2(heads, vdim, state, groups, conv, norm_groups, mlp):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                                    "conv": conv, "norm_groups": norm_groups}}


def lightning(dim, vdim, decay, mlp):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def config(vocab, width, layers, groups, eps=1e-5):
    return {"architecture": "Tobozen", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
            "layers": layers}


# TA: values wider and narrower than keys in the two layers that mix them (48 numbers in both), a rotation over part of a
#     head and over all of it; two groups in the recurrence and three in its norm; a layer without a feed-forward.
TA = config(101, 64, [
    attention(4, 2, 16, 24, 0.5, (12, 100.0), True, moe(24, 0.7, 6, 2)),
    mamba2(4, 12, 8, 2, 4, 3, moe(40, 1.0, 4, 1)),
    attention(6, 3, 20, 16, 0.45, (20, 10000.0), True, None),
    lightning(12, 20, [0.5, 0.93, 0.998], moe(20, 1.5, 5, 3))], groups=4)
# TB: a recurrent layer first; one group everywhere (also in the norms: they run folded or plain as in other decoders); head
#     sizes that are multiples of two only; no convolution to speak of in one layer and ten taps in the other; attention
#     whose values nobody mixes, then two layers that do, with another between; every expert chosen.
TB = config(211, 72, [
    lightning(10, 14, [0.7, 0.99], moe(28, 2.0, 3, 3)),
    attention(3, 1, 40, 40, 0.3, (40, 500.0), False, moe(36, 0.5, 7, 1)),
    mamba2(6, 10, 14, 1, 1, 1, None),
    attention(2, 2, 24, 12, 0.4, (8, 1000.0), True, moe(20, 1.0, 4, 2)),
    mamba2(2, 18, 6, 2, 10, 2, moe(24, 1.2, 4, 2)),
    attention(4, 4, 12, 6, 0.6, (2, 50.0), True, moe(24, 0.9, 8, 3))], groups=1, eps=1e-6)
# TC: the head sizes at which the tensor-core attention serves in bfloat16: 64 as it is, 96 and 112 padded to 128; a
#     recurrence of 128 x 64 (two tiles of keys) and one of 72 x 100 (two tiles of values); eight taps, one of twelve experts.
TC = config(300, 128, [
    attention(4, 1, 64, 64, 0.25, (64, 10000.0), True, moe(72, 1.0, 12, 1)),
    mamba2(2, 64, 128, 1, 8, 2, moe(48, 0.8, 6, 2)),
    lightning(72, 100, [0.9, 0.9995], moe(64, 1.1, 5, 2)),
    attention(2, 1, 96, 112, 0.2, (32, 500000.0), False, moe(40, 1.0, 4, 2)),
    attention(3, 1, 80, 64, 0.22, (80, 2000.0), True, None)], groups=2)
# TD: sizes that are multiples of nothing (such a width is served in float32): heads wider than any compiled kernel takes,
#     odd head sizes, eleven groups in the norms, two taps, no feed-forward in the recurrent layers.
TD = config(83, 44, [
    mamba2(3, 7, 9, 3, 2, 7, None),
    attention(2, 1, 144, 136, 0.17, (50, 10000.0), True, moe(17, 1.0, 3, 2)),
    lightning(5, 9, [0.8, 0.97, 1.0], None),
    attention(3, 1, 10, 136, 0.6, (4, 30.0), True, moe(9, 2.5, 2, 1))], groups=11)
TOBOZEN = {"TA": TA, "TB": TB, "TC": TC, "TD": TD}


def make_folder(folder, raw_config, seed, dtype=torch.float32):
    """A model folder with random weights stored in ``dtype``."""
    from stratakv_b200.config import TobozenConfig
    from stratakv_b200.engine.model import expected_tensors
    from stratakv_b200.models.tobozen import tobozen_spec
    from stratakv_b200.weights.random_init import random_tensors
    from stratakv_b200.weights.safetensors_io import write_safetensors
    typed = TobozenConfig.from_dict(raw_config)
    tensors = random_tensors(expected_tensors(tobozen_spec(typed)), seed, std=0.05, dtype=torch.float32)
    wide = (64.0 / typed.width) ** 0.5                     # weights of unit gain need 1 / sqrt(width)
    first = next((i for i, l in enumerate(raw_config["layers"]) if l["type"] == "attention" and l["mixer"]["v_mix"]), None)
    if first is not None:
        tensors[f"l{first}.mix.vmix"] = torch.tensor(0.37)     # a checkpoint carries it; nobody reads it
    for name in tensors:
        t = tensors[name]
        if name == "embed":
            tensors[name] = t * 8.0
        elif name.endswith((".mix.q", ".mix.k", ".mix.v", ".mix.g", ".mix.o", ".mix.in")):
            tensors[name] = t * 2.5 * wide
        elif name.endswith((".q.norm", ".k.norm", ".norm1", ".norm2", ".mix.norm")) or name == "final.norm":
            tensors[name] = 1.0 + (t - 1.0) * 6.0          # from 0.4 to 1.6
        elif name.endswith(".mlp.router"):
            tensors[name] = t * 4.0 * wide
        elif ".mlp.e" in name:
            tensors[name] = t * 4.0 * wide
        elif name.endswith(".mix.conv"):
            tensors[name] = t * 1.5
        elif name.endswith(".mix.conv.b"):
            # positive, so that a token's own B . C hardly ever cancels the skip (a row that is small everywhere before its
            # norm would make noise of rounding)
            tensors[name] = t.abs() * 8.0 + 0.2
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(raw_config, indent=1))
    write_safetensors(folder / "model.safetensors", {n: t.to(dtype) for n, t in tensors.items()})
    return folder
