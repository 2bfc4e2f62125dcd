"""Small Gubidra configurations for the tests, and random weights for them under the checkpoint's names.

The cases differ from one another in every size and option: the number of residual streams (one, two, three, five: more than
the fast kernel takes), the order of the layer kinds (each kind first somewhere, two of a kind in a row), a loop over some
layers, over one layer three times, once, none at all; heads and kv heads (also equal, also one), key and value widths (unequal,
equal, not multiples of 8, wider than 128), the part of a head that is turned (a part, all, none), decays (also exactly 1), the
cap of the gates, windows (also of one key, also none), the rows of the distance bias (also odd, also two) and the distance it
ends at (inside and beyond the window), the number of experts, of groups (also one, also as many as experts) and of the groups
kept (also all), how many a token runs (one, some, all that are open), the clamp of the experts (tight enough to bite, and so
wide that it never does), a layer without a feed-forward, the embedding's factor, eps from 1e-3 to 1e-6.
"""
from __future__ import annotations

import copy
import os
from typing import Dict

import torch


def moe(experts, top, ff, limit, groups=None, scale=1.0):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}


def attention(heads, kv_heads, dim, vdim, rows, far, window, mlp, scale=None):
    """`rows`: rows of the bias table, which config.json does not hold (the weight file's shape gives it)."""
    return {"type": "attention", "mlp": mlp, "_rows": rows,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 3.0 * dim ** -0.5, "bias_max": far,
                      "mask": {"size": window} if window else None}}


def mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def retention(heads, dim, vdim, decay, mlp, rot=None):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": rot}}


def model(vocab, width, streams, eps, layers, scale=1.0, loop=None):
    raw = {"architecture": "Gubidra", "vocab": vocab, "width": width, "streams": streams, "embedding": {"scale": scale}, "norm": {"eps": eps},
           "layers": layers}
    if loop:
        raw["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return raw


CASES = {
    # every kind once, two of them looped twice; three streams; part of a head turned; unequal widths; a window that ends before the
    # bias does; a clamp that bites; no feed-forward in the middle
    "a": model(210, 64, 3, 1e-5, [retention(3, 16, 24, (0.5, 0.9, 0.99), moe(6, 2, 24, 0.5, (3, 2), 1.7), rot={"base": 5000.0, "dims": 12}),
                                  attention(4, 2, 16, 24, 10, 60, 24, None),
                                  mlstm(2, 20, 12, 6.0, moe(6, 2, 24, 0.5, (3, 2), 1.7))], scale=5.0, loop=(0, 2, 2)),
    # one stream; a matrix memory first; sizes that are not multiples of 8; one head; no rotation; a decay of exactly 1; no window; an
    # odd number of bias rows; groups of one expert each, all kept; every expert that is open runs; a clamp that never bites
    "b": model(333, 72, 1, 1e-3, [mlstm(1, 12, 20, 2.0, moe(3, 3, 36, 1e4, (3, 3), 0.5)),
                                  retention(1, 20, 10, (1.0,), moe(4, 1, 30, 1.0)),
                                  attention(3, 3, 12, 12, 7, 21.5, None, moe(3, 1, 36, 1.0, (3, 1), 2.0)),
                                  attention(3, 1, 20, 28, 2, 9, 5, None)]),
    # sizes the tensor-core kernels like (heads of 64); two streams; a window beyond the bias's end; all of a head turned; the last
    # layer looped three times
    "c": model(256, 128, 2, 2e-6, [attention(4, 2, 64, 64, 32, 100, 150, moe(8, 3, 64, 2.0, (4, 2), 1.2)),
                                   retention(2, 64, 64, (0.97, 0.999), moe(8, 4, 64, 2.0, (2, 1), 2.5), rot={"base": 2e5, "dims": 64}),
                                   mlstm(2, 64, 32, 15.0, None),
                                   attention(8, 1, 64, 64, 16, 300, 130, moe(8, 3, 64, 2.0, (4, 2), 1.2))], scale=11.3, loop=(3, 4, 3)),
    # wide heads and wide keys; five streams; a window of one key; two of a kind in a row; a loop of one pass
    "d": model(150, 48, 5, 1e-6, [mlstm(1, 136, 40, 9.0, moe(2, 1, 16, 1.5)),
                                  mlstm(2, 8, 136, 9.0, None),
                                  attention(2, 2, 40, 136, 9, 40, 1, moe(4, 2, 16, 0.8, (2, 1), 1.0)),
                                  attention(2, 1, 80, 16, 6, 12, 33, None),
                                  retention(1, 136, 24, (0.95,), None, rot={"base": 300.0, "dims": 100})], scale=0.7, loop=(1, 3, 1)),
}


def raw_config(key: str) -> dict:
    """The configuration as config.json holds it."""
    raw = copy.deepcopy(CASES[key])
    for layer in raw["layers"]:
        layer.pop("_rows", None)
    return raw


def complete(raw: dict, weights: Dict[str, torch.Tensor]) -> dict:
    """With the sizes that only the tensors' shapes give."""
    from microllm_rocm_b200.config.gubidra import sizes_from_tensors
    return sizes_from_tensors(raw, {n: tuple(t.shape) for n, t in weights.items()})


def random_weights(spec: dict, seed: int, bias: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random tensors under the checkpoint's names, values that bf16 holds exactly (so that only the arithmetic differs between
    the two formats); `bias`: how far the distance biases spread."""
    g = torch.Generator().manual_seed(seed)
    W, S = spec["width"], spec["streams"]
    normal = lambda *shape, std=1.0: torch.randn(*shape, generator=g) * std
    proj = lambda rows, cols=W: normal(rows, cols, std=cols ** -0.5)
    out = {"embed": normal(spec["vocab"], W), "final.norm": 1 + normal(W, std=0.1), "head": proj(spec["vocab"]) * 3.0}
    for i, layer in enumerate(spec["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer.get("mlp") else (1,):
            # every stream a different share, so that an index taken the wrong way round shows, but no mixture that nearly cancels
            # (its norm would blow rounding errors up)
            out[f"{p}hc{q}.in"] = (1 + normal(S, std=0.3)) / S
            out[f"{p}hc{q}.out"] = 1 + normal(S, std=0.3)
            out[f"{p}hc{q}.mix"] = torch.eye(S) * 0.6 + normal(S, S).abs() * 0.6 / S
            out[f"{p}norm{q}"] = 1 + normal(W, std=0.1)
        q, H, dk, dv = p + "mix.", m["heads"], m["dim"], m["vdim"]
        out[q + "o"] = proj(W, H * dv)
        if layer["type"] == "attention":
            G = m["kv_heads"]
            out[q + "q"], out[q + "k"], out[q + "v"], out[q + "g"] = proj(H * dk), proj(G * dk), proj(G * dv), proj(H) * 2.0
            out[q + "rel"] = normal(layer["_rows"], H, std=bias)
        else:
            out[q + "q"], out[q + "k"], out[q + "v"], out[q + "g"] = proj(H * dk), proj(H * dk), proj(H * dv), proj(H * dv)
            if layer["type"] == "mlstm":
                out[q + "i"], out[q + "f"] = proj(H) * 2.0, proj(H) * 2.0
                out[q + "i.b"], out[q + "f.b"] = normal(H), 3.0 + normal(H)
                out[q + "norm"] = 1 + normal(H * dv, std=0.2)
        mlp = layer.get("mlp")
        if not mlp:
            continue
        q, ff = p + "mlp.", mlp["expert"]["ff"]
        out[q + "router"] = proj(mlp["router"]["experts"]) * 2.0
        for e in range(mlp["router"]["experts"]):
            out[f"{q}e{e}.gate"], out[f"{q}e{e}.up"], out[f"{q}e{e}.down"] = proj(ff) * 1.5, proj(ff) * 1.5, proj(W, ff)
    return {n: t.to(torch.bfloat16).to(torch.float32) for n, t in out.items()}


def case(key: str, seed: int = 0, sharp: float = 1.0, bias: float = 1.0):
    """(raw config as config.json holds it, weights).  `sharp` multiplies the scale of every softmax, which makes it peaky:
    single keys, far back, at a page's border or at a window's edge, then carry a position's output."""
    raw = raw_config(key)
    for layer in raw["layers"]:
        if layer["type"] == "attention":
            layer["mixer"]["scale"] *= sharp
    return raw, random_weights(CASES[key], seed or (len(key) + ord(key[0])), bias)


def write_folder(folder: str, raw: dict, weights: Dict[str, torch.Tensor], storage: torch.dtype = torch.float32) -> str:
    import json

    from microllm_rocm_b200.weights.safetensors import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    save_file({n: t.to(storage).contiguous() for n, t in weights.items()}, os.path.join(folder, "model.safetensors"), metadata={"format": "pt"})
    return folder
