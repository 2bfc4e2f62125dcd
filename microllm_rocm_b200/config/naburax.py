"""Typed configuration of the Naburax decoder, read from its own config.json keys.

  architecture          "Naburax"
  vocab, width          vocabulary and residual width
  norm.eps              eps of every norm of the model
  embedding             {scale, bigram}: the factor on the token's row (absent: 1); bigram {buckets, mul_prev, mul_cur} | absent: a
                        second table whose row is chosen by the token and the one before it
  logit_scale           the factor on the logits (absent: 1)
  layers[i]             type ("parallel" | "latent_attention"), mixer (its sizes), mlp (moe, or null for none)
  max_positions         optional: the longest sequence the engine admits (no table depends on it)

Mixer "parallel": left {heads, kv_heads, dim, vdim, scale, mask}, right {heads, vdim, state, groups, conv, norm_groups}, left_scale,
right_scale.  mask: {size, keep_first} | absent (every earlier token is visible).
Mixer "latent_attention": heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask {size} | absent,
rot {base, dims (= rot_dim), scaling {factor, original, fast, slow} | absent} | absent.
mlp "moe": router {experts, top}, expert {ff}.
Every size and constant comes from here or from a tensor's shape; nothing in the engine carries one.
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .lozepel import _heads, _mapping
from .matidra import _number, _positive_int
from .qwen2 import ConfigError

ARCHITECTURE = "Naburax"
MIXER_KINDS = ("parallel", "latent_attention")
DEFAULT_MAX_POSITIONS = 1 << 20


def _mask(m: Mapping[str, Any], where: str, keeps: bool) -> None:
    mask = m.get("mask")
    if mask is None:
        return
    _positive_int(_mapping(mask, f"{where}.mask").get("size"), f"{where}.mask.size")
    keep = mask.get("keep_first", 0)
    if not isinstance(keep, int) or isinstance(keep, bool) or keep < 0 or (keep and not keeps):
        raise ConfigError(f"{where}.mask.keep_first must be a non-negative integer, and only attention with keys per head has it")


def _rot(m: Mapping[str, Any], where: str) -> None:
    rot = m.get("rot")
    if rot is None:
        return
    base = _mapping(rot, f"{where}.rot").get("base")
    _number(base, f"{where}.rot.base", positive=True)
    dims = rot.get("dims", m["rot_dim"])
    if not isinstance(dims, int) or isinstance(dims, bool) or dims <= 0 or dims % 2 or dims > m["rot_dim"]:
        raise ConfigError(f"{where}.rot.dims must be even, positive and at most rot_dim")
    scaling = rot.get("scaling")
    if scaling is None:
        return
    for key in ("factor", "original", "fast", "slow"):
        _number(_mapping(scaling, f"{where}.rot.scaling").get(key), f"{where}.rot.scaling.{key}", positive=True)
    if base == 1:
        raise ConfigError(f"{where}.rot.base must not be 1 when frequencies are stretched")


@dataclass(frozen=True)
class NaburaxConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[Dict[str, Any], ...]
    embedding_scale: float = 1.0
    bigram: Optional[Dict[str, int]] = None
    logit_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    torch_dtype: str = "bfloat16"

    # ---- what the engine asks of any configuration ------------------------------------
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    eos_token_id = None

    # ---- validation ----------------------------------------------------------------
    def validate(self) -> None:
        _positive_int(self.vocab, "vocab"); _positive_int(self.width, "width"); _positive_int(self.max_positions, "max_positions")
        _number(self.norm_eps, "norm.eps", positive=True)
        _number(self.embedding_scale, "embedding.scale"); _number(self.logit_scale, "logit_scale")
        if self.bigram is not None:
            for key in ("buckets", "mul_prev", "mul_cur"):
                _positive_int(_mapping(self.bigram, "embedding.bigram").get(key), f"embedding.bigram.{key}")
        if not self.layers:
            raise ConfigError("layers must list at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = layer.get("type")
            if kind not in MIXER_KINDS:
                raise ConfigError(f"{where}.type {kind!r} is not one of {', '.join(MIXER_KINDS)}")
            m = _mapping(layer.get("mixer"), f"{where}.mixer")
            if kind == "latent_attention":
                for key in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"):
                    _positive_int(m.get(key), f"{where}.mixer.{key}")
                _number(m.get("scale"), f"{where}.mixer.scale", positive=True)
                _mask(m, f"{where}.mixer", keeps=False); _rot(m, f"{where}.mixer")
            else:
                left, right = _mapping(m.get("left"), f"{where}.mixer.left"), _mapping(m.get("right"), f"{where}.mixer.right")
                _heads(left, f"{where}.mixer.left"); _mask(left, f"{where}.mixer.left", keeps=True)
                for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
                    _positive_int(right.get(key), f"{where}.mixer.right.{key}")
                if right["heads"] % right["groups"] or right["heads"] * right["vdim"] % right["norm_groups"]:
                    raise ConfigError(f"{where}.mixer.right: groups must divide heads, and norm_groups heads * vdim")
                _number(m.get("left_scale"), f"{where}.mixer.left_scale"); _number(m.get("right_scale"), f"{where}.mixer.right_scale")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if _mapping(mlp, f"{where}.mlp").get("kind") != "moe":
                raise ConfigError(f"{where}.mlp.kind {mlp.get('kind')!r} is not 'moe'")
            router = _mapping(mlp.get("router"), f"{where}.mlp.router")
            _positive_int(router.get("experts"), f"{where}.mlp.router.experts"); _positive_int(router.get("top"), f"{where}.mlp.router.top")
            if router["top"] > router["experts"]:
                raise ConfigError(f"{where}.mlp.router.top must be at most experts")
            _positive_int(_mapping(mlp.get("expert"), f"{where}.mlp.expert").get("ff"), f"{where}.mlp.expert.ff")

    # ---- (de)serialisation -----------------------------------------------------------
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "NaburaxConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if k not in raw]
        if missing:
            raise ConfigError("config.json is missing " + ", ".join(missing))
        if not isinstance(raw["layers"], list):
            raise ConfigError("layers must be a list")
        embedding = raw.get("embedding") or {}
        bigram = embedding.get("bigram")
        cfg = cls(vocab=raw["vocab"], width=raw["width"], norm_eps=(raw["norm"] or {}).get("eps"),
                  layers=tuple(copy.deepcopy(l) for l in raw["layers"]), embedding_scale=embedding.get("scale", 1.0),
                  bigram=dict(bigram) if bigram else None, logit_scale=raw.get("logit_scale", 1.0),
                  max_positions=raw.get("max_positions", DEFAULT_MAX_POSITIONS), torch_dtype=raw.get("torch_dtype", "bfloat16"))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "NaburaxConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path, "r", encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> Dict[str, Any]:
        embedding: Dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram:
            embedding["bigram"] = dict(self.bigram)
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": embedding, "layers": [copy.deepcopy(l) for l in self.layers], "logit_scale": self.logit_scale,
                "max_positions": self.max_positions, "torch_dtype": self.torch_dtype}

    def __hash__(self):
        return hash(json.dumps(self.to_dict(), sort_keys=True))


# ---- presets: a tiny one for smoke runs, and two whose layers have the sizes of real models' layers ---------------
def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, mlp, window=None, base=10000.0, scaling=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim, **({"scaling": scaling} if scaling else {})}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def parallel_layer(left, right, mlp, window=None, keep_first=0, left_scale=1.0, right_scale=1.0, scale=None):
    """left = (heads, kv_heads, dim, vdim); right = (heads, vdim, state, groups, conv, norm_groups)"""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim"), left), scale=scale or left[2] ** -0.5)
    if window:
        l["mask"] = {"size": window, "keep_first": keep_first}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": l, "right": dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right)),
                      "left_scale": left_scale, "right_scale": right_scale}}


def _preset(vocab, width, layers, buckets):
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "layers": layers,
            "embedding": {"scale": 2.0, "bigram": {"buckets": buckets, "mul_prev": 36313, "mul_cur": 27191}}, "logit_scale": 0.5}


YARN = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}
PRESETS: Dict[str, Dict[str, Any]] = {
    "naburax-tiny": _preset(320, 96, [parallel_layer((4, 2, 16, 24), (4, 16, 24, 2, 3, 2), moe(4, 2, 48), window=24, keep_first=5, right_scale=0.7),
                                      latent_layer(3, 16, 8, 24, 40, 32, moe(4, 2, 48), window=40, scaling=YARN),
                                      latent_layer(3, 16, 8, 24, 40, 32, None)], buckets=211),
    "naburax-small": _preset(32000, 1024, [parallel_layer((16, 4, 64, 64), (16, 64, 64, 1, 4, 1), moe(16, 4, 704), window=1024, keep_first=64),
                                           latent_layer(16, 64, 32, 64, 384, 256, moe(16, 4, 704), window=1024, scaling=YARN),
                                           latent_layer(16, 64, 32, 64, 384, 256, moe(16, 4, 704), scaling=YARN),
                                           latent_layer(16, 64, 32, 64, 384, 256, moe(16, 4, 704), scaling=YARN)], buckets=32749),
    "naburax-3b-layers": _preset(102400, 2048, [parallel_layer((16, 4, 128, 128), (32, 64, 128, 2, 4, 2), moe(32, 4, 704), window=1024, keep_first=128),
                                                latent_layer(16, 128, 64, 128, 768, 512, moe(32, 4, 704), window=1024, scaling=YARN),
                                                latent_layer(16, 128, 64, 128, 768, 512, moe(32, 4, 704), scaling=YARN),
                                                latent_layer(16, 128, 64, 128, 768, 512, moe(32, 4, 704), scaling=YARN)], buckets=65521),
}
