"""The Gubidra decoder as data: which parts, with which sizes, in which order.

token embedding times a constant, copied into several residual streams -> layers of two pre-norm sublayers (layer norms with a
weight and no bias), each of which reads a learned mixture of the streams and is written back through another -> sum of the
streams -> layer norm -> head.  A range of layers may run several times in a row with the same weights and a cache or state
per pass.  A layer's mixer is one of: grouped-query softmax attention without rotation, with a learned bias by distance and
head, an optional sliding window and one sigmoid gate per head; the matrix memory with capped exponential gates, a norm per
head and a sigmoid gate; retention (rotated q and k, one fixed decay per head, a norm per head without a weight, a silu gate).
The feed-forward is routed experts with a clamped activation (sigmoid scores, a choice limited to the best groups of
experts, renormalised weights times a constant), or none.

Tensor names: `embed`, `final.norm`, `head`; layer i: `l<i>.norm1`, `.norm2`, `l<i>.hc1.{in,out,mix}`, `l<i>.hc2.{in,out,mix}`;
`l<i>.mix.{q,k,v,g,o}` with `.rel` (attention) or `.i`, `.i.b`, `.f`, `.f.b`, `.norm` (matrix memory);
`l<i>.mlp.{router,e<j>.gate,e<j>.up,e<j>.down}`.

This file only describes; the parts it names live in `parts/` and know nothing of it.
"""
from __future__ import annotations

from ..config.gubidra import ARCHITECTURE, PRESETS, GubidraConfig, sizes_from_tensors
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunSpec

NAMES = dict(q="q", k="k", v="v", o="o", gate="g")


def _mixer(cfg: GubidraConfig, layer: dict) -> PartSpec:
    m = layer["mixer"]
    params = dict(prefix="mix.", hidden_size=cfg.width, num_heads=m["heads"], dim=m["dim"], vdim=m["vdim"], eps=float(cfg.norm_eps))
    if layer["type"] == "attention":
        return PartSpec("normed_attention", dict(
            params, num_kv_heads=m["kv_heads"], scale=float(m["scale"]), values="projected", qk_norm=False, gate="head",
            window=(m.get("mask") or {}).get("size"), distance_bias=dict(buckets=m["bias_rows"], far=m["bias_max"]),
            names=dict(NAMES, distance="rel")))
    if layer["type"] == "mlstm":
        return PartSpec("mlstm", dict(params, gate_cap=float(m["gate_cap"]),
                                      names=dict(NAMES, i="i", f="f", i_bias="i.b", f_bias="f.b", norm="norm")))
    params.update(decay=tuple(float(d) for d in m["decay"]), names=NAMES)
    rot = m.get("rot")
    if rot:
        params["position"] = PartSpec("rotary", dict(head_dim=m["dim"], rotary_dim=int(rot["dims"]), theta=float(rot["base"]),
                                                     layout="split_half"))
    return PartSpec("retention", params)


def _feed_forward(cfg: GubidraConfig, mlp) -> PartSpec:
    if mlp is None:
        return PartSpec("none")
    router, groups = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}
    return PartSpec("routed_experts", dict(
        prefix="mlp.", hidden_size=cfg.width, experts=router["experts"], top=router["top"], expert_size=mlp["expert"]["ff"],
        expert_names=("e{}.gate", "e{}.up", "e{}.down"), router_name="router", scoring="sigmoid_groups", groups=groups["count"],
        keep=groups["keep"], weight_scale=float(router["scale"]), activation="clamped_swish", limit=float(mlp["expert"]["limit"])))


def build_spec(cfg: GubidraConfig) -> ModelSpec:
    cfg.validate()
    w, eps = cfg.width, float(cfg.norm_eps)
    norm = lambda name, **more: PartSpec("layernorm", dict(prefix="", name=name, size=w, eps=eps, bias=False, **more))
    layers, tolerated = [], []
    for i, layer in enumerate(cfg.layers):
        mlp = layer.get("mlp")
        layers.append(LayerSpec(prefix=f"l{i}.",
                                block=PartSpec("mixed_streams", dict(size=w, streams=cfg.streams, names=("hc1.", "hc2."))),
                                mixer_norm=norm("norm1"), mixer=_mixer(cfg, layer),
                                ffn_norm=norm("norm2", absent=mlp is None), feed_forward=_feed_forward(cfg, mlp)))
        if mlp is None:                          # a layer without a feed-forward: what would surround it may still be stored
            tolerated += [f"l{i}.norm2"] + [f"l{i}.hc2.{n}" for n in ("in", "out", "mix")]
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=w, vocab_size=cfg.vocab, max_position=cfg.max_positions,
        embedding=PartSpec("token_embedding", dict(name="embed", vocab_size=cfg.vocab, hidden_size=w, scale=float(cfg.embedding_scale),
                                                   streams=cfg.streams)),
        position=PartSpec("none"), layers=layers, order=[RunSpec(layer=i) for i in cfg.run_order()], final_norm=norm("final.norm"),
        head=PartSpec("lm_head", dict(name="head", vocab_size=cfg.vocab, hidden_size=w)),
        streams=cfg.streams, tolerated_tensors=tuple(tolerated))
    spec.validate()
    return spec


register_architecture(Architecture(name=ARCHITECTURE, config_class=GubidraConfig, build_spec=build_spec, presets=PRESETS,
                                   sizes_from_tensors=sizes_from_tensors), replace=True)
