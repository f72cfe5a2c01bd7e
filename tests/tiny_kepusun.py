"""Small Kepusun configurations for the tests, as config.json dictionaries, and a writer of model folders with random
weights that the tests may tune.

U1 mixes everything: a matrix memory with keys and values of unequal sizes, differential attention whose values are not
twice as wide as a map's keys, a layer that reads an earlier layer's keys and values, a layer without feed-forward, and
routers with and without groups, over three streams.
U2 has sizes the tensor-core kernels take (maps of 64 over values of 128, maps of 32 over values of 64, matrix memories of
64 x 128 and 32 x 32), four streams.
U3 has values that are 1 or absent elsewhere: one stream, one head, one key head per query head, one expert, one chosen
expert, a weight factor of 1, as many groups as experts, all groups kept, keys and values whose size is not said.
U4 has sizes that are no multiple of 8 anywhere, five streams, a memory with more rows than columns, and two layers that
read the same layer's keys and values.
"""
import json
import os

import torch


def moe(experts, top, ff, scale, groups=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def memory(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def attention(heads, kv_heads, dim, vdim, scale, diff, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def model(vocab, width, streams, layers, eps=1e-5):
    return {"architecture": "Kepusun", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}


U1 = model(300, 96, 3, [memory(3, 20, 12, 11.0, moe(6, 2, 40, 1.7, (3, 2))),
                        attention(4, 2, 24, 40, 0.3, 0.35, moe(5, 3, 24, 0.8)),
                        attention(6, 2, 24, 40, 0.2, 0.6, None, kv_from=1),
                        memory(2, 12, 28, 6.0, moe(8, 3, 16, 1.2, (4, 2)))])

U2 = model(260, 128, 4, [memory(2, 64, 128, 15.0, moe(8, 2, 64, 2.0, (4, 3))),
                         attention(4, 2, 64, 128, 0.18, 0.3, moe(8, 2, 64, 1.5, (2, 1))),
                         memory(4, 32, 32, 9.0, None),
                         attention(2, 2, 64, 128, 0.15, 0.25, moe(8, 2, 64, 1.5), kv_from=1),
                         attention(6, 1, 32, 64, 0.3, 0.2, moe(8, 4, 32, 1.0, (4, 2)))], eps=1e-6)

U3 = model(200, 64, 1, [memory(1, 16, 16, 4.0, moe(4, 1, 32, 1.0)),
                        attention(1, 1, 16, 32, 0.4, 0.0, moe(6, 2, 16, 1.0, (6, 6))),
                        memory(1, 8, 8, 20.0, moe(1, 1, 24, 1.0)),
                        attention(3, 3, 8, 8, 0.5, 0.6, moe(4, 2, 16, 1.0, (1, 1)))], eps=1e-6)
del U3["layers"][2]["mixer"]["vdim"], U3["layers"][3]["mixer"]["vdim"], U3["layers"][3]["mixer"]["kv_heads"]

U4 = model(173, 76, 5, [attention(3, 1, 18, 11, 0.33, 0.25, moe(9, 4, 12, 1.1, (3, 2))),
                        memory(5, 9, 37, 7.0, moe(3, 3, 20, 0.9)),
                        attention(5, 1, 18, 11, 0.27, 0.5, moe(6, 2, 28, 1.3, (2, 1)), kv_from=0),
                        memory(1, 70, 5, 12.0, None),
                        attention(1, 1, 18, 11, 0.4, 0.1, moe(4, 2, 12, 1.0), kv_from=0),
                        attention(2, 1, 9, 18, 0.3, 0.3, None)])

# Standard deviations (by the last part of a tensor's slot) that make every mechanism matter in a random model without
# making it chaotic: matrices (relative to one over the root of what they sum over) whose results are of order one, gates
# that open and close, routers that choose firmly; a second map whose weight stays away from one (two maps that see the
# same key leave 1 - lambda of it).
RELATIVE = {"q": 0.9, "k": 0.9, "v": 1.0, "g": 1.3, "o": 0.6, "i": 1.2, "f": 2.5, "up": 0.9, "down": 0.5, "router": 4.5}
ABSOLUTE = {"weight": 0.5, "lq1": 0.2, "lk1": 0.2, "lq2": 0.2, "lk2": 0.2}


def tune(tensors, streams):
    """Values away from the neutral ones for everything that is not a matrix, so that each of them shows when it is left
    out: norms, mixing coefficients, gate biases (forget gates mostly open, so that memories last)."""
    for name, t in tensors.items():
        g = torch.Generator().manual_seed(sum(ord(c) * (i + 1) for i, c in enumerate(name)) + t.numel())
        r = torch.randn(t.shape, generator=g)
        leaf = name.split(".")[-1]
        parts = name.split(".")
        if leaf == "alpha":
            new = 0.45 + 0.1 * r
        elif leaf == "b" and parts[-2] in ("norm1", "norm2", "norm"):
            new = 0.15 * r
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            new = 1.4 + 0.3 * r
        elif leaf == "norm":
            new = 1.0 + 0.3 * r
        elif leaf == "b" and parts[-2] == "i":
            new = 0.8 * r
        elif leaf == "b" and parts[-2] == "f":
            new = 3.5 + 1.5 * r
        elif leaf == "in":
            new = 1.0 / streams + 0.15 * r
        elif leaf == "out":
            new = 1.1 + 0.4 * r
        elif leaf == "mix":
            new = 0.75 * torch.eye(streams) + 0.3 / streams ** 0.5 * r
        else:
            continue
        t.copy_(new.to(t.dtype))


def write_model(model_dir, raw, seed, more=None, dtype=torch.bfloat16):
    """config.json + model.safetensors with random weights (the package's own generator and writer); ``more(tensors)``
    may change them before they are written.  Returns {name: tensor}."""
    from nanoinfer_b200.config import config_from_dict
    from nanoinfer_b200.weights.plan import tensor_plan
    from nanoinfer_b200.weights.random_init import random_tensors
    from nanoinfer_b200.weights.safetensors_io import write_safetensors
    cfg = config_from_dict(raw)
    tensors = dict(random_tensors(cfg, seed, 1.0, torch.float32))
    for p in tensor_plan(cfg):
        leaf = p.slot.split(".")[-1]
        if leaf in RELATIVE:
            tensors[p.name] *= RELATIVE[leaf] / p.shape[-1] ** 0.5
        elif leaf in ABSOLUTE:
            tensors[p.name] *= ABSOLUTE[leaf]
    tensors = {name: t.to(dtype) for name, t in tensors.items()}
    tune(tensors, raw["streams"])
    if more is not None:
        more(tensors)
    os.makedirs(model_dir, exist_ok=True)
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(raw, f)
    write_safetensors(os.path.join(model_dir, "model.safetensors"), tensors.items())
    return tensors
