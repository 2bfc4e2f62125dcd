"""Typed configuration of the Gubidra decoder, read from its own config.json keys.

  architecture          "Gubidra"
  vocab, width          vocabulary and width of a residual stream
  streams               how many residual streams the blocks mix
  embedding.scale       factor on the embedding rows
  norm.eps              eps of every norm of the model
  layers[i]             type ("attention" | "mlstm" | "retention"), mixer (its sizes), mlp (moe, or null for none)
  loop                  {start, stop, times}: layers start..stop-1 run `times` times in a row, each pass with a state of its
                        own; absent or null: every layer runs once
  max_positions         optional: the longest sequence the engine admits (no table depends on it)

Mixer "attention": heads, kv_heads, dim, vdim, scale, bias_max (the distance from which the distance bias takes its last row),
mask {size} | null (keys a query sees, itself included), bias_rows (rows of the bias table; may be absent from config.json: it is
then read from the shape of `<layer>.mix.rel` in the weight file, `sizes_from_tensors`).
Mixer "mlstm": heads, dim, vdim, gate_cap.
Mixer "retention": heads, dim, vdim, decay [one per head], rot {base, dims} | null.
mlp: kind "moe", router {experts, top, scale, groups {count, keep} | null}, expert {ff, limit}.
Every size and constant comes from here or from a tensor's shape; nothing in the engine carries one.
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Sequence, Tuple

from .lozepel import _mapping, _rot
from .matidra import _heads, _number, _positive_int
from .qwen2 import ConfigError

ARCHITECTURE = "Gubidra"
MIXER_KINDS = ("attention", "mlstm", "retention")
DEFAULT_MAX_POSITIONS = 1 << 20
MAX_STREAMS = 16


@dataclass(frozen=True)
class GubidraConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[Dict[str, Any], ...]
    embedding_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None          # (start, stop, times)
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

    def run_order(self) -> List[int]:
        """Layer indices in execution order."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    # ---- validation ----------------------------------------------------------------
    def validate(self) -> None:
        _positive_int(self.vocab, "vocab"); _positive_int(self.width, "width"); _positive_int(self.max_positions, "max_positions")
        if _positive_int(self.streams, "streams") > MAX_STREAMS:
            raise ConfigError(f"streams must be at most {MAX_STREAMS}")
        _number(self.embedding_scale, "embedding.scale"); _number(self.norm_eps, "norm.eps", positive=True)
        if not self.layers:
            raise ConfigError("layers must list at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = layer.get("type")
            if kind not in MIXER_KINDS:
                raise ConfigError(f"{where}.type {kind!r} is not one of {', '.join(MIXER_KINDS)}")
            m = _mapping(layer.get("mixer"), f"{where}.mixer")
            if kind == "attention":
                _heads(m, f"{where}.mixer")
                _number(m.get("scale"), f"{where}.mixer.scale", positive=True)
                rows = m.get("bias_rows")
                if not isinstance(rows, int) or isinstance(rows, bool) or rows < 2:
                    raise ConfigError(f"{where}.mixer.bias_rows must be an integer of 2 or more (read from the weight file when config.json has none)")
                if _number(m.get("bias_max"), f"{where}.mixer.bias_max", positive=True) <= rows // 2:
                    raise ConfigError(f"{where}.mixer.bias_max must lie beyond half of the bias table's {rows} rows")
                if m.get("mask") is not None:
                    _positive_int(_mapping(m["mask"], f"{where}.mixer.mask").get("size"), f"{where}.mixer.mask.size")
            else:
                for key in ("heads", "dim", "vdim"):
                    _positive_int(m.get(key), f"{where}.mixer.{key}")
                if kind == "mlstm":
                    _number(m.get("gate_cap"), f"{where}.mixer.gate_cap", positive=True)
                else:
                    _rot(m, f"{where}.mixer")
                    decay = m.get("decay")
                    if not isinstance(decay, (list, tuple)) or len(decay) != m["heads"]:
                        raise ConfigError(f"{where}.mixer.decay must list one number per head")
                    for d in decay:
                        _number(d, f"{where}.mixer.decay")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if _mapping(mlp, f"{where}.mlp").get("kind") != "moe":
                raise ConfigError(f"{where}.mlp.kind {mlp.get('kind')!r} is not 'moe'")
            router = _mapping(mlp.get("router"), f"{where}.mlp.router")
            experts = _positive_int(router.get("experts"), f"{where}.mlp.router.experts")
            top = _positive_int(router.get("top"), f"{where}.mlp.router.top")
            _number(router.get("scale"), f"{where}.mlp.router.scale")
            count, keep = 1, 1
            if router.get("groups") is not None:
                groups = _mapping(router["groups"], f"{where}.mlp.router.groups")
                count = _positive_int(groups.get("count"), f"{where}.mlp.router.groups.count")
                keep = _positive_int(groups.get("keep"), f"{where}.mlp.router.groups.keep")
                if experts % count or keep > count:
                    raise ConfigError(f"{where}.mlp.router.groups: {keep} of {count} groups do not fit {experts} experts")
            if top > keep * (experts // count):
                raise ConfigError(f"{where}.mlp.router.top must be at most the experts that can be chosen")
            expert = _mapping(mlp.get("expert"), f"{where}.mlp.expert")
            _positive_int(expert.get("ff"), f"{where}.mlp.expert.ff"); _number(expert.get("limit"), f"{where}.mlp.expert.limit", positive=True)
        if self.loop is not None:
            start, stop, times = self.loop
            if not (0 <= start < stop <= len(self.layers)) or times < 1:
                raise ConfigError(f"loop {{start {start}, stop {stop}, times {times}}} does not fit {len(self.layers)} layers")

    # ---- (de)serialisation -----------------------------------------------------------
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "GubidraConfig":
        missing = [k for k in ("vocab", "width", "streams", "layers", "norm") if k not in raw]
        if missing:
            raise ConfigError("config.json is missing " + ", ".join(missing))
        if not isinstance(raw["layers"], list):
            raise ConfigError("layers must be a list")
        loop = raw.get("loop")
        if loop is not None:
            for k in ("start", "stop", "times"):
                if not isinstance(loop.get(k), int) or isinstance(loop.get(k), bool):
                    raise ConfigError(f"loop.{k} must be an integer")
            loop = (loop["start"], loop["stop"], loop["times"])
        cfg = cls(vocab=raw["vocab"], width=raw["width"], streams=raw["streams"], norm_eps=(raw["norm"] or {}).get("eps"),
                  layers=tuple(copy.deepcopy(l) for l in raw["layers"]), embedding_scale=(raw.get("embedding") or {}).get("scale", 1.0),
                  loop=loop, max_positions=raw.get("max_positions", DEFAULT_MAX_POSITIONS), torch_dtype=raw.get("torch_dtype", "bfloat16"))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "GubidraConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path, "r", encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "streams": self.streams,
               "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
               "layers": [copy.deepcopy(l) for l in self.layers], "max_positions": self.max_positions, "torch_dtype": self.torch_dtype}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return out

    def __hash__(self):
        return hash(json.dumps(self.to_dict(), sort_keys=True))


def sizes_from_tensors(raw: Dict[str, Any], shapes: Mapping[str, Sequence[int]]) -> Dict[str, Any]:
    """config.json completed with the rows of the distance-bias tables, which only the weight file knows (tensor name -> shape)."""
    raw = copy.deepcopy(raw)
    for i, layer in enumerate(raw.get("layers") or []):
        if not isinstance(layer, dict) or layer.get("type") != "attention" or not isinstance(layer.get("mixer"), dict):
            continue
        tensor = f"l{i}.mix.rel"
        if "bias_rows" not in layer["mixer"] and tensor in shapes and len(shapes[tensor]) == 2:
            layer["mixer"]["bias_rows"] = int(shapes[tensor][0])
    return raw


# ---- presets: a tiny one for smoke runs, and two whose layers have the sizes of real models' layers ---------------
def moe(experts, top, ff, groups=1, keep=1, scale=1.5, limit=7.0):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale},
            "expert": {"ff": ff, "limit": limit}}


def attention_layer(heads, kv_heads, dim, vdim, window, mlp, bias_rows=32, bias_max=128, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "bias_max": bias_max,
                      "bias_rows": bias_rows, "mask": {"size": window} if window else None}}


def mlstm_layer(heads, dim, vdim, mlp, gate_cap=15.0):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def retention_layer(heads, dim, vdim, mlp, rot_dims=None, base=10000.0, decay=None):
    decay = decay or [1.0 - 2.0 ** (-(5 + 4.0 * h / max(1, heads - 1))) for h in range(heads)]
    return {"type": "retention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot_dims} if rot_dims else None}}


def _preset(vocab, width, streams, layers, loop=None):
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "streams": streams, "embedding": {"scale": width ** 0.5},
            "norm": {"eps": 1e-5}, "layers": layers, "loop": loop}


PRESETS: Dict[str, Dict[str, Any]] = {
    "gubidra-tiny": _preset(320, 96, 3, [mlstm_layer(3, 16, 24, moe(6, 2, 48, groups=3, keep=2, limit=2.0), gate_cap=10.0),
                                         attention_layer(4, 2, 32, 16, 40, moe(6, 2, 48, groups=3, keep=2, limit=2.0), bias_rows=12, bias_max=50),
                                         retention_layer(2, 24, 40, None, rot_dims=16)], loop={"start": 1, "stop": 3, "times": 2}),
    "gubidra-small": _preset(32000, 1024, 2, [retention_layer(8, 64, 128, moe(16, 4, 704, groups=4, keep=2), rot_dims=64),
                                              attention_layer(16, 4, 64, 64, 1024, moe(16, 4, 704, groups=4, keep=2)),
                                              mlstm_layer(4, 128, 256, moe(16, 4, 704, groups=4, keep=2)),
                                              attention_layer(16, 4, 64, 64, 1024, moe(16, 4, 704, groups=4, keep=2))]),
    "gubidra-3b-layers": _preset(102400, 2048, 2, [retention_layer(16, 64, 128, moe(32, 4, 704, groups=4, keep=2), rot_dims=64),
                                                   attention_layer(16, 4, 128, 128, 1024, moe(32, 4, 704, groups=4, keep=2)),
                                                   mlstm_layer(8, 128, 256, moe(32, 4, 704, groups=4, keep=2)),
                                                   attention_layer(16, 4, 128, 128, 1024, moe(32, 4, 704, groups=4, keep=2))]),
}
