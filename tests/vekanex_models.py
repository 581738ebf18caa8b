"""Small Vekanex configurations for the tests, and folders with random weights for them.

The weights are drawn so that a fault shows: projections of unit gain, attention scores a few units apart, decays per channel
from "forgets in a few tokens" to "keeps for hundreds", forget gates from half open to nearly shut, input gates on both sides
of one (so that the floor of a memory's denominator counts for some tokens and not for others), low-rank gates away from
their middle, norms' weights between 0.4 and 1.6, biases that count, experts that differ and router logits a unit apart.
"""
from __future__ import annotations

import copy
import json
from pathlib import Path

import torch


def moe(ff, experts, top, shared=0):
    raw = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        raw["shared"] = {"ff": shared}
    return raw


def mlstm(heads, dim, vdim, gate_cap, mlp):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def gla(heads, dim, vdim, tau, rank, mlp):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}, "mlp": mlp}


def parallel(left, right, scales, mlp):
    """left (heads, kv_heads, dim, vdim, scale, (rotated numbers, base)), right (heads, kv_heads, dim, vdim, taps, ranks)."""
    H, G, d, dv, scale, rot = left
    h, g, n, nv, taps, ranks = right
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": scale, "rot": {"dims": rot[0], "base": rot[1]}},
        "right": {"heads": h, "kv_heads": g, "dim": n, "vdim": nv, "conv": taps, "decay_rank": ranks[0], "gate_rank": ranks[1]},
        "left_scale": scales[0], "right_scale": scales[1]}}


def same_as(layers, index):
    return {**copy.deepcopy(layers[index]), "weights_of": index}


def config(vocab, width, layers, residual_mult, softcap=None, eps=1e-5):
    raw = {"architecture": "Vekanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": residual_mult,
           "layers": layers}
    if softcap:
        raw["logit_softcap"] = softcap
    return raw


# VA: values wider and narrower than keys; four query heads on two key heads, the delta rule's keys shared by two heads; an
#     attention layer and a memory that run twice on one set of weights; a layer without a feed-forward.
_A = [gla(3, 12, 20, 4.0, 5, moe(24, 6, 2, 40)),
      parallel((4, 2, 16, 24, 0.4, (12, 100.0)), (4, 2, 12, 8, 4, (6, 9)), (0.7, 0.9), moe(24, 5, 3, 16)),
      mlstm(2, 16, 24, 8.0, None)]
VA = config(101, 64, _A + [same_as(_A, 1), same_as(_A, 2)], 0.6, softcap=6.0)
# VB: a memory first, no cap on the logits, no shared experts, every expert chosen, a factor above one on what joins the stream;
#     head sizes that are multiples of two only, no convolution to speak of, ten taps in another layer, a rank of one.
_B = [mlstm(3, 10, 14, 3.0, moe(28, 3, 3)),
      parallel((3, 1, 40, 40, 0.3, (40, 500.0)), (2, 2, 14, 10, 1, (3, 1)), (1.0, 0.5), moe(36, 7, 1, 20)),
      gla(2, 10, 6, 1.0, 1, None),
      parallel((2, 2, 24, 12, 0.35, (8, 1000.0)), (6, 3, 6, 18, 10, (4, 7)), (0.4, 1.0), moe(20, 4, 2))]
VB = config(211, 72, _B + [same_as(_B, 0)], 1.1, eps=1e-6)
# VC: the head sizes at which the tensor-core attention serves in bfloat16 (64 as it is, 96 and 112 padded to 128); memories of
#     128 x 64 and 64 x 128, one of 72 x 100; eight taps, one of twelve experts.
_C = [parallel((4, 1, 64, 64, 0.2, (32, 10000.0)), (2, 1, 64, 128, 8, (16, 24)), (0.8, 0.6), moe(72, 12, 1, 48)),
      mlstm(2, 128, 64, 12.0, moe(48, 6, 2)),
      gla(2, 72, 100, 16.0, 12, moe(64, 5, 2, 24)),
      parallel((2, 1, 96, 112, 0.15, (96, 500000.0)), (3, 3, 32, 40, 3, (8, 8)), (1.0, 1.0), None)]
VC = config(300, 128, _C + [same_as(_C, 2)], 0.8, softcap=20.0)
# VD: sizes that are multiples of nothing (such a width is served in float32): heads wider than any compiled kernel takes, key
#     sizes too wide for chunks of 32 tokens, odd head sizes.
_D = [parallel((2, 1, 144, 136, 0.15, (50, 10000.0)), (3, 1, 7, 9, 2, (3, 5)), (0.9, 1.2), moe(17, 3, 2, 9)),
      mlstm(3, 5, 7, 5.0, moe(9, 2, 1)),
      gla(1, 290, 37, 8.0, 7, None),
      parallel((3, 1, 10, 136, 0.5, (4, 30.0)), (1, 1, 300, 21, 5, (2, 3)), (0.5, 1.0), None)]
VD = config(83, 44, _D + [same_as(_D, 1)], 0.5, softcap=11.0)
VEKANEX = {"VA": VA, "VB": VB, "VC": VC, "VD": VD}


def make_folder(folder, raw_config, seed, dtype=torch.float32):
    """A model folder with random weights stored in ``dtype``; config.json leaves the ranks to the tensors' shapes."""
    from stratakv_b200.config import VekanexConfig
    from stratakv_b200.engine.model import expected_tensors
    from stratakv_b200.models.vekanex import vekanex_spec
    from stratakv_b200.weights.random_init import random_tensors
    from stratakv_b200.weights.safetensors_io import write_safetensors
    typed = VekanexConfig.from_dict(raw_config)
    tensors = random_tensors(expected_tensors(vekanex_spec(typed)), seed, std=0.05, dtype=torch.float32)
    unit = 20.0 / typed.width ** 0.5                       # rows of unit gain need 1 / sqrt(width)
    for name in tensors:
        t = tensors[name]
        if name == "embed":
            tensors[name] = t * 16.0
        elif name.endswith(("norm", "norm1", "norm2")):
            tensors[name] = 1.0 + (t - 1.0) * 6.0          # from 0.4 to 1.6
        elif name.endswith((".a2", ".g2")):
            tensors[name] = t * 30.0 / t.shape[1] ** 0.5
        elif name.endswith("a2.b"):
            tensors[name] = t * 3.0
        elif name.endswith(".f.b"):
            tensors[name] = t * 6.0
        elif name.endswith(".b") and t.dim() == 1:
            tensors[name] = t * 10.0
        elif name.endswith(".conv"):
            tensors[name] = t * 1.5
            tensors[name][:, -1] += 0.7
        elif name.endswith(".right.b"):
            tensors[name] = t * 0.4 * unit                 # (betas between 0.2 and 0.8)
        elif t.dim() == 2 and name != "head":
            tensors[name] = t * unit
        elif name == "head":
            tensors[name] = t * 2.0 * unit
    # Every head of a recurrent mixer is divided by its root mean square, so a head whose terms cancel would make noise of
    # rounding: keys lean towards the queries, and a token's own term (nearly) always counts.
    for name in list(tensors):
        if name.endswith((".mix.k", ".right.k", ".right.k.conv")):
            q = tensors[name.replace(".k", ".q")]
            tensors[name] = 0.8 * q + 0.6 * tensors[name]
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    shown = json.loads(json.dumps(raw_config))
    for layer in shown["layers"]:
        for section in (layer["mixer"], layer["mixer"].get("right", {})):
            for key in ("rank", "decay_rank", "gate_rank"):
                section.pop(key, None)
    (folder / "config.json").write_text(json.dumps(shown, indent=1))
    write_safetensors(folder / "model.safetensors", {n: t.to(dtype) for n, t in tensors.items()})
    return folder
