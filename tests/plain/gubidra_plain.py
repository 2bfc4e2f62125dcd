"""Plain, slow restatement of the Gubidra decoder: one function per mechanism, whole sequences at once, float64 on the CPU.
It shares no code with the package: it reads a raw configuration (the keys of config.json) and a dict of tensors under the
checkpoint's names.

  streams       X_1 .. X_s, all E[tok] * c at first.  Per sublayer with vectors a, b and a matrix M of its own:
                u = sum_i a_i X_i;  y = sublayer(n(u));  X_j <- sum_i M[i, j] X_i + b_j y      (from the old streams)
                logits = W_head n_f(sum_i X_i);   every n: (x - mean) / sqrt(mean((x - mean)^2) + eps) * w
  order         the layers in turn; layers start..stop-1 run `times` times, each pass with a state of its own
  attention     no rotation; s_ij = (q_i . k_j) * scale + R[bucket(i - j), head], keys 0 <= i - j < window; softmax; each head's
                output times sigmoid(Wg h)_head; Wo
  mlstm         i = c tanh((Wi h + bi) / c), f = log sigmoid(c tanh((Wf h + bf) / c)) per head;  m_t = max(f + m_(t-1), i), m_0 = 0;
                S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T, n_t likewise with k;  q times dk^-1/2;
                o = S^T q / (max(|n . q|, e^-m) + 1e-6);  o / rms(o) per head * weight * sigmoid(Wg h); Wo
  retention     rotation of the first `dims` elements of q and k (element i with i + dims/2), k times dk^-1/2;
                S_t = d_head S_(t-1) + k v^T, o = S^T q;  o / rms(o) per head * silu(Wg h); Wo
  feed-forward  s = sigmoid(Wr h); a group of neighbours scores the sum of its two largest s; the `top` largest s within the
                `keep` best groups run; weights s / (sum of the chosen + 1e-20) * scale;
                expert: g = min(Wg h, L), u = clamp(Wu h, -L, L), Wd (g sigmoid(1.702 g) (u + 1))
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w.to(F)


def rms_quotient(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------------------------------- streams
def read_streams(x: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """x [streams, T, width], a [streams]: what a sublayer reads."""
    return sum(a[i] * x[i] for i in range(x.shape[0]))


def write_streams(x: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """The streams after a sublayer that gave y; mix is indexed [from, to]."""
    s = x.shape[0]
    return torch.stack([sum(mix[i, j] * x[i] for i in range(s)) + b[j] * y for j in range(s)])


def run_order(cfg: dict) -> List[int]:
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


# ---------------------------------------------------------------------------------------- softmax attention with a distance bias
def bucket(n: int, buckets: int, far: int) -> int:
    """Distances below buckets/2 have a row each; from there on the rows widen logarithmically up to `far`."""
    near = buckets // 2
    if n < near:
        return n
    return min(buckets - 1, near + int(math.floor(math.log(n / near) / math.log(far / near) * (buckets - near))))


def biased_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, rel: torch.Tensor, far: int,
                     window: Optional[int]) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv], rel [buckets, H]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    rows = torch.tensor([bucket(n, rel.shape[0], far) for n in range(T)])
    out = torch.zeros((T, H, v.shape[-1]), dtype=F)
    for h in range(H):
        g = h // (H // G)
        for t in range(T):
            lo = max(0, t - window + 1) if window else 0
            s = (k[lo: t + 1, g] @ q[t, h]) * scale + rel[rows[t - torch.arange(lo, t + 1)], h]
            out[t, h] = torch.softmax(s, 0) @ v[lo: t + 1, g]
    return out


def mixer_attention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].to(F).T).view(T, H, m["dim"])
    k = (h @ w[p + "k"].to(F).T).view(T, G, m["dim"])
    v = (h @ w[p + "v"].to(F).T).view(T, G, m["vdim"])
    o = biased_attention(q, k, v, m["scale"], w[p + "rel"].to(F), m["bias_max"], (m.get("mask") or {}).get("size"))
    o = o * torch.sigmoid(h @ w[p + "g"].to(F).T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].to(F).T


# ---------------------------------------------------------------------------------------- matrix memory with exponential gates
def log_gates(h: torch.Tensor, wi, bi, wf, bf, cap: float):
    """(log input gate, log forget gate) [T, H]."""
    i = cap * torch.tanh((h @ wi.to(F).T + bi.to(F)) / cap)
    f = cap * torch.tanh((h @ wf.to(F).T + bf.to(F)) / cap)
    return i, torch.nn.functional.logsigmoid(f)


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor) -> torch.Tensor:
    """q, k [T, H, dk], v [T, H, dv], gates [T, H]; returns o [T, H, dv]."""
    T, H, dk = q.shape
    out = torch.zeros((T, H, v.shape[-1]), dtype=F)
    for h in range(H):
        S, n, m = torch.zeros((dk, v.shape[-1]), dtype=F), torch.zeros(dk, dtype=F), torch.zeros((), dtype=F)
        for t in range(T):
            m_new = torch.maximum(f[t, h] + m, i[t, h])
            keep, take = torch.exp(f[t, h] + m - m_new), torch.exp(i[t, h] - m_new)
            S = keep * S + take * torch.outer(k[t, h], v[t, h])
            n = keep * n + take * k[t, h]
            m = m_new
            out[t, h] = (S.T @ q[t, h]) / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def mixer_mlstm(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H = h.shape[0], m["heads"]
    q = (h @ w[p + "q"].to(F).T).view(T, H, m["dim"]) * m["dim"] ** -0.5
    k = (h @ w[p + "k"].to(F).T).view(T, H, m["dim"])
    v = (h @ w[p + "v"].to(F).T).view(T, H, m["vdim"])
    i, f = log_gates(h, w[p + "i"], w[p + "i.b"], w[p + "f"], w[p + "f.b"], m["gate_cap"])
    o = rms_quotient(matrix_memory(q, k, v, i, f), eps).reshape(T, -1) * w[p + "norm"].to(F)
    return (o * torch.sigmoid(h @ w[p + "g"].to(F).T)) @ w[p + "o"].to(F).T


# ---------------------------------------------------------------------------------------- retention
def rotate_halves(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, n]: element i is turned with element i + dims/2 by t * base^(-2i/dims), i < dims/2; the rest pass."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    a = torch.arange(x.shape[0], dtype=F)[:, None, None] * freq
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], -1)


def retain(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: List[float]) -> torch.Tensor:
    """S_t = d S_(t-1) + k v^T, o = S^T q per head, token by token."""
    T, H, dk = q.shape
    out = torch.zeros((T, H, v.shape[-1]), dtype=F)
    for h in range(H):
        S = torch.zeros((dk, v.shape[-1]), dtype=F)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def mixer_retention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H = h.shape[0], m["heads"]
    q = (h @ w[p + "q"].to(F).T).view(T, H, m["dim"])
    k = (h @ w[p + "k"].to(F).T).view(T, H, m["dim"])
    v = (h @ w[p + "v"].to(F).T).view(T, H, m["vdim"])
    rot = m.get("rot")
    if rot:
        q, k = rotate_halves(q, rot["dims"], rot["base"]), rotate_halves(k, rot["dims"], rot["base"])
    o = rms_quotient(retain(q, k * m["dim"] ** -0.5, v, m["decay"]), eps).reshape(T, -1)
    return (o * silu(h @ w[p + "g"].to(F).T)) @ w[p + "o"].to(F).T


MIXERS = {"attention": mixer_attention, "mlstm": mixer_mlstm, "retention": mixer_retention}


# ---------------------------------------------------------------------------------------- routed feed-forward
def route(z: torch.Tensor, top: int, groups: int, keep: int, scale: float):
    """z [T, experts] -> (chosen [T, top], best first; weights [T, top])."""
    s = torch.sigmoid(z)
    T, E = s.shape
    size = E // groups
    chosen, weights = [], []
    for t in range(T):
        score = [sum(sorted(s[t, g * size:(g + 1) * size].tolist(), reverse=True)[:2]) for g in range(groups)]
        best = sorted(range(groups), key=lambda g: (-score[g], g))[:keep]
        open_to = [e for e in range(E) if e // size in best]
        picked = sorted(open_to, key=lambda e: (-float(s[t, e]), e))[:top]
        w = s[t, picked]
        chosen.append(picked)
        weights.append(w / (w.sum() + 1e-20) * scale)
    return torch.tensor(chosen), torch.stack(weights)


def expert(w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, limit: float) -> torch.Tensor:
    g = (h @ w[p + "gate"].to(F).T).clamp(max=limit)
    u = (h @ w[p + "up"].to(F).T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].to(F).T


def routed_ff(mlp: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    chosen, weights = route(h @ w[p + "router"].to(F).T, r["top"], groups["count"], groups["keep"], r["scale"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        at = (chosen == e)
        rows = at.any(1)
        if rows.any():
            out[rows] += (weights * at).sum(1)[rows][:, None] * expert(w, f"{p}e{e}.", h[rows], mlp["expert"]["limit"])
    return out


# ---------------------------------------------------------------------------------------- the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab]; `layers_out` collects the sum of the streams after every layer run."""
    eps, s = cfg["norm"]["eps"], cfg["streams"]
    x = (w["embed"].to(F)[torch.tensor(tokens)] * cfg["embedding"]["scale"]).expand(s, -1, -1).clone()
    for i in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        steps = [(1, lambda h: MIXERS[layer["type"]](layer["mixer"], w, p + "mix.", h, eps))]
        if layer.get("mlp"):
            steps.append((2, lambda h: routed_ff(layer["mlp"], w, p + "mlp.", h)))
        for q, sublayer in steps:
            hc = {n: w[f"{p}hc{q}.{n}"].to(F) for n in ("in", "mix", "out")}
            y = sublayer(layer_norm(read_streams(x, hc["in"]), w[f"{p}norm{q}"], eps))
            x = write_streams(x, y, hc["mix"], hc["out"])
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return layer_norm(x.sum(0), w["final.norm"], eps) @ w["head"].to(F).T
