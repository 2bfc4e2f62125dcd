"""Small Naburax configurations for the tests, and random weights for them under the checkpoint's names.

The cases differ from one another in every size and option: the order of the layer kinds (each kind first somewhere, two of a
kind in a row), heads and kv heads (also equal, also one), key and value widths (unequal, equal, not multiples of 8, wider
than 128), windows (shorter and longer than a page, one key, none) and the first tokens they keep (none, a few, more than the
window, more than a page), the recurrence's heads, groups, state rows, columns and norm groups (also all of them one), taps
of the convolution (also one), ranks of both latents, rotated parts (also none, also a stretched table), how many experts a token runs
(one, some, all), layers without a feed-forward, the pair table, factors of one and others, eps from 1e-3 to 1e-6.
"""
from __future__ import annotations

import copy
import os
from typing import Dict

import torch


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, mlp, window=None, rot=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": scale or 3.0 * (dim + rot_dim) ** -0.5}
    if rot:
        m["rot"] = dict(rot, dims=rot_dim)
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def parallel(left, right, mlp, window=None, keep=None, left_scale=1.3, right_scale=0.7, scale=None):
    """left = (heads, kv_heads, dim, vdim); right = (heads, vdim, state, groups, conv, norm_groups)"""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim"), left), scale=scale or 3.0 * left[2] ** -0.5)
    if window:
        l["mask"] = {"size": window} if keep is None else {"size": window, "keep_first": keep}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": l, "right": dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right)),
                      "left_scale": left_scale, "right_scale": right_scale}}


def model(vocab, width, eps, layers, bigram, embed_scale, logit_scale):
    embedding = {"scale": embed_scale}
    if bigram:
        embedding["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Naburax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers, "embedding": embedding,
            "logit_scale": logit_scale}


CASES = {
    # every kind, a window shorter than two pages with a few kept tokens, unequal widths, a stretched rotation beside a plain one
    "a": model(210, 64, 1e-5, [parallel((4, 2, 16, 24), (4, 12, 20, 2, 3, 3), moe(5, 2, 24), window=20, keep=5),
                               latent(3, 16, 8, 24, 28, 20, moe(5, 2, 24), window=33,
                                      rot={"base": 5000.0, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}}),
                               latent(3, 16, 8, 24, 28, 20, None, rot={"base": 300.0})], (97, 13, 5), 1.7, 0.8),
    # latent attention first; sizes that are not multiples of 8; one head and one group everywhere; one tap; no rotation, no
    # pair table, factors of one; more kept tokens than the window holds, and than a page holds; every expert runs
    "b": model(333, 72, 1e-3, [latent(1, 20, 6, 28, 18, 30, moe(3, 3, 36)),
                               parallel((3, 3, 12, 12), (1, 10, 12, 1, 1, 1), moe(3, 1, 36), window=3, keep=21, left_scale=1.0, right_scale=1.0),
                               parallel((3, 1, 20, 28), (6, 7, 9, 3, 2, 6), None, window=1, keep=0)], None, 1.0, 1.0),
    # sizes the tensor-core kernels like; windows of more than a tile with kept tokens that end inside one; two latent layers in a row
    "c": model(256, 128, 2e-6, [latent(4, 64, 16, 64, 64, 64, moe(4, 2, 64), window=100, rot={"base": 2e5}),
                                parallel((4, 2, 64, 64), (4, 64, 64, 2, 4, 2), moe(4, 3, 64), window=130, keep=37, left_scale=0.8, right_scale=1.1),
                                latent(4, 64, 16, 64, 64, 64, moe(4, 2, 64), window=41,
                                       rot={"base": 1e4, "scaling": {"factor": 8.0, "original": 128, "fast": 16.0, "slow": 1.0}}),
                                latent(4, 64, 16, 64, 64, 64, moe(4, 1, 64), rot={"base": 2e5}),
                                parallel((8, 1, 64, 64), (2, 64, 64, 1, 4, 1), moe(4, 2, 64), window=64, keep=16)], (251, 17, 9), 3.2, 0.3),
    # wide heads beside wide values; a wide state; a window whose kept tokens are one; no window on the attention of the last layer
    "d": model(150, 48, 1e-6, [parallel((2, 2, 40, 136), (2, 20, 136, 1, 6, 4), moe(2, 1, 16), window=33, keep=1),
                               latent(2, 24, 32, 40, 40, 160, moe(4, 2, 16), window=5, rot={"base": 700.0}),
                               parallel((2, 1, 80, 16), (3, 40, 40, 3, 5, 1), None, left_scale=2.0, right_scale=0.25)], (11, 7, 3), 0.5, 2.0),
}


def raw_config(key: str) -> dict:
    return copy.deepcopy(CASES[key])


def random_weights(raw: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Random tensors under the checkpoint's names, values that bf16 holds exactly (so that only the arithmetic differs between
    the two formats).  Decays are slow enough that a state forgotten at a cut shows many tokens later."""
    g = torch.Generator().manual_seed(seed)
    W = raw["width"]
    normal = lambda *shape, std=1.0: torch.randn(*shape, generator=g) * std
    proj = lambda rows, cols=W: normal(rows, cols, std=cols ** -0.5)
    out = {"embed": normal(raw["vocab"], W), "final.norm": 1 + normal(W, std=0.1), "head": proj(raw["vocab"]) * 3.0}
    bg = (raw.get("embedding") or {}).get("bigram")
    if bg:
        out["bigram"] = normal(bg["buckets"] + 1, W)
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = 1 + normal(W, std=0.1)
        if layer["type"] == "latent_attention":
            q, H, R = p + "mix.", m["heads"], m["kv_rank"]
            out[q + "dq"], out[q + "uq"] = proj(m["q_rank"]), proj(H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            out[q + "dkv"], out[q + "uk"], out[q + "uv"] = proj(R + m["rot_dim"]), proj(H * m["dim"], R), proj(H * m["vdim"], R)
            out[q + "dq.norm"], out[q + "dkv.norm"] = 1 + normal(m["q_rank"], std=0.2), 1 + normal(R, std=0.2)
            out[q + "o"] = proj(W, H * m["vdim"])
        else:
            l, q = m["left"], p + "mix.left."
            H, G, dk, dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            out[q + "q"], out[q + "k"], out[q + "v"], out[q + "o"] = proj(H * dk), proj(G * dk), proj(G * dv), proj(W, H * dv)
            out[q + "q.norm"], out[q + "k.norm"] = 1 + normal(H * dk, std=0.2), 1 + normal(G * dk, std=0.2)
            r, q = m["right"], p + "mix.right."
            inner, channels = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
            out[q + "in"] = proj(inner + channels + r["heads"])
            out[q + "conv"], out[q + "conv.b"] = normal(channels, r["conv"], std=0.6), normal(channels, std=0.3)
            out[q + "dt_bias"], out[q + "A_log"], out[q + "D"] = normal(r["heads"]) - 1.0, normal(r["heads"], std=0.5) - 2.0, 1 + normal(r["heads"], std=0.5)
            out[q + "norm"], out[q + "o"] = 1 + normal(inner, std=0.2), proj(W, inner)
        mlp = layer.get("mlp")
        if not mlp:
            continue
        q, ff = p + "mlp.", mlp["expert"]["ff"]
        out[p + "norm2"] = 1 + normal(W, std=0.1)
        out[q + "router"] = proj(mlp["router"]["experts"]) * 0.7
        for e in range(mlp["router"]["experts"]):
            out[f"{q}e{e}.gate"], out[f"{q}e{e}.up"], out[f"{q}e{e}.down"] = proj(ff) * 1.5, proj(ff) * 1.5, proj(W, ff)
    return {n: t.to(torch.bfloat16).to(torch.float32) for n, t in out.items()}


def case(key: str, seed: int = 0, sharp: float = 1.0):
    """(raw config as config.json holds it, weights).  `sharp` multiplies the scale of every softmax, which makes it peaky:
    single keys, far back, at a page's border or at a window's edge, then carry a position's output."""
    raw = raw_config(key)
    for layer in raw["layers"]:
        m = layer["mixer"]
        (m["left"] if layer["type"] == "parallel" else m)["scale"] *= sharp
    return raw, random_weights(raw, seed or (len(key) + ord(key[0])))


def write_folder(folder: str, raw: dict, weights: Dict[str, torch.Tensor], storage: torch.dtype = torch.float32) -> str:
    import json

    from microllm_rocm_b200.weights.safetensors import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    save_file({n: t.to(storage).contiguous() for n, t in weights.items()}, os.path.join(folder, "model.safetensors"), metadata={"format": "pt"})
    return folder
