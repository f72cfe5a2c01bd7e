"""Small Lomopel configurations for the tests, as config.json dictionaries, and a writer of model folders with random
weights that the tests may tune.

L1 mixes everything: three attention layers that mix values (the first of them not the model's first layer) with another
between them that does not, values wider than keys, side-by-side layers (a window of 20 beside a delta rule whose query/key
heads are shared by three value heads), a layer without feed-forward, thin matrices of 13 and 5.
L2 has sizes the tensor-core attention kernels take (heads of 64 and 128, values of the keys' size), a window of whole pages,
a delta rule of 64 x 64 heads, thin matrices of 16 and 24.
L3 has values that are 1 or absent elsewhere: one head, one tap (no convolution history), thin matrices of 1, a window of one
token, no query temperature, a rotation of nothing, an embedding scale of 1, sides weighted 1, no mixing of values.
L4 has sizes that are no multiple of 8 anywhere, a window that is no multiple of the page, delta heads of 40 x 9.
"""
import json
import os

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def attention(heads, kv_heads, dim, vdim, scale, v_mix, coef=None, every=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def window(heads, kv_heads, dim, vdim, scale, size, dims, base):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
            "rot": {"dims": dims, "base": base}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def side_by_side(left, right, left_scale, right_scale, mlp):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def config(vocab, width, eps, scale, layers):
    return {"architecture": "Lomopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


L1 = config(300, 96, 1e-5, 6.0, [
    side_by_side(window(6, 3, 16, 24, 0.25, 20, 12, 50000.0), delta(6, 2, 20, 12, 4), 1.3, 0.7, dense(72)),
    attention(4, 2, 24, 40, 0.15, True, 0.3, 16, dense(136)),
    attention(6, 1, 20, 28, 0.2, False, 0.4, 10, None),
    side_by_side(window(4, 4, 18, 10, 0.3, 9, 18, 100.0), delta(3, 3, 12, 32, 3), 0.6, 1.2, None),
    attention(8, 2, 16, 40, 0.2, True, None, None, dense(64)),
    attention(2, 2, 8, 40, 0.35, True, 0.2, 7, dense(40))])
L2 = config(260, 128, 1e-6, 3.0, [
    attention(8, 2, 64, 64, 0.11, True, 0.25, 32, dense(192)),
    side_by_side(window(4, 1, 128, 128, 0.09, 48, 64, 10000.0), delta(4, 2, 64, 64, 4), 1.25, 0.85, dense(128)),
    attention(4, 1, 128, 128, 0.08, False, 0.5, 20, dense(128)),
    side_by_side(window(8, 4, 64, 64, 0.12, 32, 64, 500.0), delta(2, 2, 128, 128, 2), 0.75, 1.5, dense(96)),
    attention(6, 2, 64, 64, 0.12, True, 0.1, 50, dense(128))])
L3 = config(200, 64, 1e-6, 1.0, [
    attention(1, 1, 16, 16, 0.4, False, None, None, dense(32)),
    side_by_side(window(2, 2, 32, 16, 0.2, 1, 0, 10.0), delta(1, 1, 32, 16, 1), 1.0, 1.0, None),
    attention(2, 2, 16, 16, 0.5, True, 0.3, 1, dense(64))])
L4 = config(173, 76, 1e-5, 2.5, [
    attention(5, 5, 18, 11, 0.33, True, 0.6, 9, dense(52)),
    side_by_side(window(3, 1, 22, 36, 0.2, 19, 6, 123.0), delta(5, 5, 40, 9, 5), 0.6, 1.7, dense(20)),
    attention(10, 5, 14, 11, 0.27, True, 0.4, 25, dense(12))])

# Inner sizes of the thin matrices (decay, gate) by model and layer: no configuration key names them.
RANKS = {"L1": {0: (13, 5), 3: (4, 9)}, "L2": {1: (16, 24), 3: (8, 8)}, "L3": {1: (1, 1)}, "L4": {1: (7, 10)}}

# Standard deviations (by the last part of a tensor's slot) that make every mechanism matter in a random model.
LIVELY = {"weight": 0.5, "q": 0.12, "k": 0.12, "v": 0.12, "g": 0.15, "o": 0.1, "up": 0.12, "gate": 0.12, "down": 0.1,
          "conv": 0.6, "b": 0.3, "a1": 0.15, "a2": 0.5, "g1": 0.15, "g2": 0.5, "sink": 1.0, "A_log": 0.7, "dt_bias": 1.5}


def settle(tensors):
    """Weights that differ from their neutral value: norms around zero and around one, layer scales of either side of one,
    mixing weights well inside (0, 1), decays from fast to slow."""
    for name, t in tensors.items():
        leaf = name.split(".")[-1]
        g = torch.Generator().manual_seed(len(name) * 131 + t.numel() + sum(map(ord, name)))
        noise = torch.randn(t.shape, generator=g)
        if leaf in ("norm1", "norm2") or name == "final.norm":
            t.copy_((0.3 * noise).to(t.dtype))
        elif leaf in ("ls1", "ls2") or (leaf == "norm" and t.dim() == 1):
            t.copy_((1.0 + 0.3 * noise).to(t.dtype))
        elif leaf == "vmix":
            t.copy_((0.4 + 0.1 * noise).to(t.dtype))
        elif leaf == "dt_bias":
            t.copy_((-2.5 + 1.5 * noise).to(t.dtype))


def resize_thin(tensors, ranks, seed=0):
    """The thin matrices of the given layers with inner sizes {layer: (decay's, gate's)}."""
    for i, pair in ranks.items():
        for (one, two), rank in zip((("a1", "a2"), ("g1", "g2")), pair):
            for name, shape in ((one, lambda t: (rank, t.shape[1])), (two, lambda t: (t.shape[0], rank))):
                key = f"l{i}.mix.right.{name}"
                g = torch.Generator().manual_seed(seed * 1000 + 17 * i + rank + ord(name[0]) + ord(name[1]))
                old = tensors[key]
                tensors[key] = (torch.randn(shape(old), generator=g) * LIVELY[name]).to(old.dtype)


def write_model(model_dir, raw, seed, tune=None, dtype=torch.bfloat16, ranks=None):
    """config.json + model.safetensors with random weights (the package's own generator and writer);
    ``tune(tensors)`` may change them before they are written.  Returns {name: tensor}."""
    from nanoinfer_b200.config import config_from_dict
    from nanoinfer_b200.weights.plan import tensor_plan
    from nanoinfer_b200.weights.random_init import random_tensors
    from nanoinfer_b200.weights.safetensors_io import write_safetensors
    cfg = config_from_dict(raw)
    std = {p.slot: LIVELY[p.slot.split(".")[-1]] for p in tensor_plan(cfg) if p.slot.split(".")[-1] in LIVELY}
    tensors = dict(random_tensors(cfg, seed, 0.05, dtype, std))
    if ranks:
        resize_thin(tensors, ranks, seed)
    settle(tensors)
    if tune is not None:
        tune(tensors)
    os.makedirs(model_dir, exist_ok=True)
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(raw, f)
    write_safetensors(os.path.join(model_dir, "model.safetensors"), tensors.items())
    return tensors
