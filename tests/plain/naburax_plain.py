"""Plain, slow restatement of the Naburax decoder: one function per mechanism, whole sequences at once, float64 on the
CPU.  It shares no code with the package: it reads a raw configuration (the keys of config.json) and a dict of tensors
under the checkpoint's names.

  stream        x_t = c E[tok_t] + B[(tok_(t-1) * a + tok_t * b) mod n]   (row n of B for a sequence's first token)
                per layer  x += n_1(mixer(x));  x += n_2(ff(x))      (the second only with a feed-forward)
                logits = s * W_head n_f(x);   every n:  y = x / sqrt(mean(x^2) + eps) * w
  parallel      a_l * left(x) + a_r * right(x)
     left       q and k each divided by the root mean square of their WHOLE row, times a weight of that length; no
                rotation; softmax over the keys i - W < j <= i and, of those further back, the first `keep_first`
     right      [z | u | dt] = W_in x, u = [x | B | C]; u through a causal convolution per channel with a bias, then silu;
                dt = softplus(dt + b);  per head S = exp(-exp(A) dt) S + dt B x^T,  y = S^T C + D x;  y * silu(z), divided
                by the root mean square of each of `norm_groups` equal parts, times a weight; W_o
  latent        c_q = n(W_dq x), q = W_uq c_q (per head `dim` plain, `rot_dim` rotated);  [c | r] = W_dkv x, c = n(c);
                k_h = W_uk c, v_h = W_uv c, r rotated and shared by the heads; score = (q.k_h + q_r.r) * scale; a window
  feed-forward  s = sigmoid(W_r x); the `top` largest s_e run: sum_e expert_e(s_e x),
                expert_e(h) = Wd_e (silu(Wg_e h) * (Wu_e h))
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w.to(F)


def project(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return h @ w.to(F).T


# ---------------------------------------------------------------------------------------- embedding
def pair_rows(tokens: List[int], buckets: int, mul_prev: int, mul_cur: int) -> List[int]:
    return [buckets] + [(p * mul_prev + c * mul_cur) % buckets for p, c in zip(tokens, tokens[1:])]


def embed(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    e = cfg.get("embedding") or {}
    x = w["embed"].to(F)[torch.tensor(tokens)] * float(e.get("scale", 1.0))
    b = e.get("bigram")
    if b:
        x = x + w["bigram"].to(F)[torch.tensor(pair_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


# ---------------------------------------------------------------------------------------- rotation
def rotation_table(dims: int, base: float, scaling: Optional[dict]):
    """(angle per position of each pair, factor on cosines and sines)"""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freq, 1.0
    turn = lambda t: dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turn(scaling["fast"])), 0), min(math.ceil(turn(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x: torch.Tensor, freq: List[float], magnitude: float) -> torch.Tensor:
    """x [T, heads, 2 * pairs]: elements (2i, 2i + 1) of the row of position t are turned by t * freq[i]."""
    a = torch.arange(x.shape[0], dtype=F)[:, None] * torch.tensor(freq, dtype=F)[None, :]
    cos, sin = torch.cos(a)[:, None, :] * magnitude, torch.sin(a)[:, None, :] * magnitude
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)


# ---------------------------------------------------------------------------------------- softmax attention
def visible(i: int, window: Optional[int], keep_first: int = 0) -> List[int]:
    return [j for j in range(i + 1) if window is None or i - j < window or j < keep_first]


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: Optional[int], keep_first: int = 0) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv]; query head h reads key/value head h // (H / G).  [T, H, dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros((T, H, v.shape[-1]), dtype=F)
    of_head = [h // (H // G) for h in range(H)]
    k, v = k[:, of_head], v[:, of_head]                                          # [T, H, .]: every query head's own copy
    for i in range(T):
        seen = visible(i, window, keep_first)
        p = torch.softmax((k[seen] * q[i]).sum(-1) * scale, 0)                  # [seen, H]
        out[i] = (p[:, :, None] * v[seen]).sum(0)
    return out


def mask_of(m: dict):
    mask = m.get("mask") or {}
    return mask.get("size"), int(mask.get("keep_first") or 0)


def left_attention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(project(h, w[p + "q"]), w[p + "q.norm"], eps).view(T, H, dk)        # over the whole row
    k = rms_norm(project(h, w[p + "k"]), w[p + "k.norm"], eps).view(T, G, dk)
    v = project(h, w[p + "v"]).view(T, G, dv)
    window, keep = mask_of(m)
    return project(softmax_attention(q, k, v, m["scale"], window, keep).reshape(T, -1), w[p + "o"])


# ---------------------------------------------------------------------------------------- selective state space
def causal_conv(u: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """u [T, C], taps [C, n]: out_t = bias + sum_j taps[:, n - 1 - j] u_(t-j), where u_i = 0 for i < 0."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros((n - 1, u.shape[1]), dtype=F), u], 0)
    out = torch.zeros_like(u) + bias.to(F)
    for j in range(n):
        out = out + padded[j:j + u.shape[0]] * taps[:, j].to(F)
    return out


def selective_state(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, a_log: torch.Tensor, D: torch.Tensor) -> torch.Tensor:
    """x [T, H, P], B, C [T, groups, N], dt [T, H] (already positive); y [T, H, P]."""
    T, H, P = x.shape
    groups, N = B.shape[1:]
    y = torch.zeros_like(x)
    for h in range(H):
        g = h // (H // groups)
        S = torch.zeros((N, P), dtype=F)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h].to(F)) * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + D[h].to(F) * x[t, h]
    return y


def right_mamba(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, u, dt = torch.split(project(h, w[p + "in"]), [inner, inner + 2 * G * N, H], -1)
    u = silu(causal_conv(u, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(u, [inner, G * N, G * N], -1)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"].to(F), threshold=60.0)
    y = selective_state(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), dt, w[p + "A_log"], w[p + "D"]).reshape(T, inner)
    y = (y * silu(z)).view(T, m["norm_groups"], -1)                               # the gate comes first
    y = rms_norm(y, None, eps).reshape(T, inner) * w[p + "norm"].to(F)
    return project(y, w[p + "o"])


def mixer_parallel(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    return (m["left_scale"] * left_attention(m["left"], w, p + "left.", h, eps)
            + m["right_scale"] * right_mamba(m["right"], w, p + "right.", h, eps))


# ---------------------------------------------------------------------------------------- latent attention
def mixer_latent(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = project(rms_norm(project(h, w[p + "dq"]), w[p + "dq.norm"], eps), w[p + "uq"]).view(T, H, d + r)
    both = project(h, w[p + "dkv"])
    c, kr = rms_norm(both[:, :R], w[p + "dkv.norm"], eps), both[:, R:]
    qr, kr = q[..., d:], kr[:, None, :]
    rot = m.get("rot")
    if rot:
        freq, magnitude = rotation_table(rot["dims"], rot["base"], rot.get("scaling"))
        qr, kr = rotate_pairs(qr, freq, magnitude), rotate_pairs(kr, freq, magnitude)
    q = torch.cat([q[..., :d], qr], -1)
    k = torch.cat([project(c, w[p + "uk"]).view(T, H, d), kr.expand(T, H, r)], -1)
    v = project(c, w[p + "uv"]).view(T, H, dv)
    window, keep = mask_of(m)
    return project(softmax_attention(q, k, v, m["scale"], window, keep).reshape(T, -1), w[p + "o"])


# ---------------------------------------------------------------------------------------- feed-forward
def route(z: torch.Tensor, top: int):
    """z [T, E] -> (chosen [T, top], their weights): sigmoid scores as they are.  The sigmoid grows with z, so the largest z are the
    largest scores, also where a score can no longer be told from 1 (ties: the smaller index)."""
    s = torch.sigmoid(z)
    chosen = torch.tensor([sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[:top] for t in range(z.shape[0])])
    return chosen, torch.gather(s, 1, chosen)


def expert(w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    return project(silu(project(h, w[p + "gate"])) * project(h, w[p + "up"]), w[p + "down"])


def routed_ff(mlp: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    chosen, weights = route(project(h, w[p + "router"]), mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weights[t]):
            out[t] += expert(w, f"{p}e{e}.", s * h[t])                              # the weight goes in, not on the result
    return out


# ---------------------------------------------------------------------------------------- the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], streams: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from position 0; `streams` (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = embed(cfg, w, tokens)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mixers = {"parallel": mixer_parallel, "latent_attention": mixer_latent}
        x = x + rms_norm(mixers[layer["type"]](m, w, p + "mix.", x, eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(routed_ff(layer["mlp"], w, p + "mlp.", x), w[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.clone())
    return project(rms_norm(x, w["final.norm"], eps), w["head"]) * float(cfg.get("logit_scale", 1.0))
