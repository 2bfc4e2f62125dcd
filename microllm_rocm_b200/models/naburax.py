"""The Naburax decoder as data: which parts, with which sizes, in which order.

scaled token embedding plus a row of a second table chosen by the token and the one before it -> layers of
[x += norm(mixer(x)); x += norm(ff(x))], the sublayers reading the stream itself -> rms norm -> head, times a factor.  A layer's
mixer is one of: two mixers side by side added with fixed weights (grouped-query softmax attention without rotation, q and k
normalised over their whole rows, a window in front of which the first tokens stay visible; a selective state space with a
grouped norm behind its gate); latent attention whose queries have a latent of their own, with interleaved, possibly stretched
rotation and a window.  The feed-forward is routed experts (sigmoid scores used as they are, multiplied into the expert's
input), or none.

Tensor names: `embed`, `bigram`, `final.norm`, `head`; layer i: `l<i>.norm1`, `.norm2`;
`l<i>.mix.left.{q,k,v,q.norm,k.norm,o}` and `l<i>.mix.right.{in,conv,conv.b,dt_bias,A_log,D,norm,o}`;
`l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}`; `l<i>.mlp.{router,e<j>.gate,e<j>.up,e<j>.down}`.

This file only describes; the parts it names live in `parts/` and know nothing of it.
"""
from __future__ import annotations

from ..config.naburax import ARCHITECTURE, PRESETS, NaburaxConfig
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunSpec

LEFT_NAMES = dict(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm")
RIGHT_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "a_log": "A_log", "d": "D", "norm": "norm", "o": "o"}
LATENT_NAMES = dict(dq="dq", dq_norm="dq.norm", uq="uq", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", o="o")


def _rotation(m: dict):
    rot = m.get("rot")
    if not rot:
        return PartSpec("none")
    params = dict(head_dim=m["rot_dim"], rotary_dim=int(rot.get("dims", m["rot_dim"])), theta=float(rot["base"]), layout="interleaved")
    if rot.get("scaling"):
        params["stretch"] = {k: float(rot["scaling"][k]) for k in ("factor", "original", "fast", "slow")}
    return PartSpec("rotary", params)


def _mixer(cfg: NaburaxConfig, layer: dict) -> PartSpec:
    m, eps = layer["mixer"], float(cfg.norm_eps)
    if layer["type"] == "latent_attention":
        return PartSpec("latent_attention", dict(
            prefix="mix.", hidden_size=cfg.width, num_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"],
            kv_rank=m["kv_rank"], scale=float(m["scale"]), eps=eps, window=(m.get("mask") or {}).get("size"), names=LATENT_NAMES,
            position=_rotation(m)))
    left, right = m["left"], m["right"]
    mask = left.get("mask") or {}
    attention = PartSpec("normed_attention", dict(
        prefix="left.", hidden_size=cfg.width, num_heads=left["heads"], num_kv_heads=left["kv_heads"], dim=left["dim"], vdim=left["vdim"],
        scale=float(left["scale"]), eps=eps, values="projected", conv=1, qk_norm="row", gate=False, window=mask.get("size"),
        keep_first=int(mask.get("keep_first") or 0), names=LEFT_NAMES))
    state_space = PartSpec("selective_state_space", dict(
        prefix="right.", hidden_size=cfg.width, num_heads=right["heads"], vdim=right["vdim"], state=right["state"], groups=right["groups"],
        conv=right["conv"], norm_groups=right["norm_groups"], eps=eps, names=RIGHT_NAMES))
    return PartSpec("parallel", dict(prefix="mix.", hidden_size=cfg.width, branches=(
        ("left", float(m["left_scale"]), attention), ("right", float(m["right_scale"]), state_space))))


def _feed_forward(cfg: NaburaxConfig, mlp) -> PartSpec:
    if mlp is None:
        return PartSpec("none")
    router = mlp["router"]
    return PartSpec("routed_experts", dict(prefix="mlp.", hidden_size=cfg.width, experts=router["experts"], top=router["top"],
                                           expert_size=mlp["expert"]["ff"], expert_names=("e{}.gate", "e{}.up", "e{}.down"),
                                           router_name="router", scoring="sigmoid", weight_on="input"))


def build_spec(cfg: NaburaxConfig) -> ModelSpec:
    cfg.validate()
    w, eps = cfg.width, float(cfg.norm_eps)
    norm = lambda name, **more: PartSpec("rmsnorm", dict(prefix="", name=name, size=w, eps=eps, **more))
    layers, tolerated = [], []
    for i, layer in enumerate(cfg.layers):
        mlp = layer.get("mlp")
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("output_norm_residual"), mixer_norm=norm("norm1"), mixer=_mixer(cfg, layer),
                                ffn_norm=norm("norm2", absent=mlp is None), feed_forward=_feed_forward(cfg, mlp)))
        if mlp is None:
            tolerated.append(f"l{i}.norm2")
    embedding = dict(name="embed", vocab_size=cfg.vocab, hidden_size=w, scale=float(cfg.embedding_scale))
    if cfg.bigram:
        embedding["bigram"] = dict(name="bigram", **{k: int(cfg.bigram[k]) for k in ("buckets", "mul_prev", "mul_cur")})
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=w, vocab_size=cfg.vocab, max_position=cfg.max_positions,
        embedding=PartSpec("token_embedding", embedding), position=PartSpec("none"), layers=layers,
        order=[RunSpec(layer=i) for i in range(len(layers))],
        # the factor on the logits is a factor on the rows in front of the head
        final_norm=norm("final.norm", scale=float(cfg.logit_scale)),
        head=PartSpec("lm_head", dict(name="head", vocab_size=cfg.vocab, hidden_size=w)), tolerated_tensors=tuple(tolerated))
    spec.validate()
    return spec


register_architecture(Architecture(name=ARCHITECTURE, config_class=NaburaxConfig, build_spec=build_spec, presets=PRESETS), replace=True)
