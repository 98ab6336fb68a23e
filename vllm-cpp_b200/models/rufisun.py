"""Rufisun: a pre-norm decoder whose norm is a tanh with a learned slope (no statistics), whose layers mix tokens by attention
with a distance bias over a window and the sequence's first tokens, by latent attention with queries through a latent and one
stretched rotation, or by two mixers side by side (attention with capped scores and growing queries, a state space in its dual
form), all softmaxes with a learned number per head in the denominator; dense feed-forwards with the square of relu or experts
whose weight multiplies what they read, beside a shared expert; typed configuration and its description as parts.

config.json names the design in ``architecture`` and gives every size and constant:

    vocab, width, norm.eps,
    layers[i] = {type: "attention",        mixer: {heads, kv_heads, dim, vdim, scale, bias_max, mask: {size, keep_first}},
                 type: "latent_attention", mixer: {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale,
                                                   rot: {base, dims, scaling: {factor, original, fast, slow}}},
                 type: "parallel",         mixer: {left: {heads, kv_heads, dim, vdim, scale, softcap, q_temp: {coef, every}},
                                                   right: {heads, vdim, state, groups, conv, norm_groups}, left_scale, right_scale},
                 mlp: null | {kind: "dense", ff}
                           | {kind: "moe", expert: {ff}, router: {experts, top}, shared: null | {ff}}}

Layer i's tensors are ``l<i>.*``: ``norm1`` before the mixer ``mix.*`` (``mix.left.*`` and ``mix.right.*`` in a parallel layer),
``norm2`` before the feed-forward ``mlp.*``; a norm's slope and shift are its name plus ``.alpha`` and ``.b``; outside the layers
``embed`` (also the output matrix) and ``final.norm``.  The number of rows of a distance-bias table comes from the tensor alone.
What the design fixes (relu squared, gelu by its definition, sigmoid scores that are not renormalised, interleaved pairs) is named
here or in the parts.  The reference has no model of this kind (src/core/engine.cpp:26-28).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

from ..config.engine_config import ConfigError
from ..config.model_spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..config.registry import register_architecture

MAX_POSITIONS = 1 << 22              # no position table bounds a request; the cache does first
MIXERS = ("attention", "latent_attention", "parallel")
NAMES = ("up", "down")               # the two matrices of a feed-forward or an expert


@dataclass
class RufisunLayer:
    kind: str
    mixer: dict                      # the layer's "mixer" object, checked
    mlp: Optional[dict] = None


@dataclass
class RufisunConfig:
    vocab: int
    width: int
    eps: float
    layers: List[RufisunLayer] = field(default_factory=list)

    @classmethod
    def from_dict(cls, cfg: dict) -> "RufisunConfig":
        problems: List[str] = []

        def number(d, key, where, integer=False, positive=True):
            v = d.get(key) if isinstance(d, dict) else None
            if v is None:
                problems.append(f"missing {where}'{key}'")
                return 1
            ok = isinstance(v, int) or (isinstance(v, float) and (not integer or v.is_integer()))
            if isinstance(v, bool) or not ok:
                problems.append(f"{where}'{key}' must be {'an integer' if integer else 'a number'}, got {v!r}")
                return 1
            if positive and not v > 0:
                problems.append(f"{where}'{key}' must be positive, got {v!r}")
                return 1
            return int(v) if integer else float(v)

        def integers(d, where, keys):
            return {k: number(d, k, where, integer=True) for k in keys}

        def heads(m, where):
            out = integers(m, where, ("heads", "dim", "vdim"))
            out["kv_heads"] = out["heads"] if m.get("kv_heads") is None else number(m, "kv_heads", where, integer=True)
            if out["heads"] % out["kv_heads"]:
                problems.append(f"{where}heads {out['heads']} is no multiple of kv_heads {out['kv_heads']}")
            out["scale"] = number(m, "scale", where, positive=False)
            return out

        def attention(m, where):
            out = heads(m, where)
            out["bias_max"] = number(m, "bias_max", where)
            mask = m.get("mask")
            # no mask: every token is seen
            out["window"] = 0 if mask is None else number(mask, "size", where + "mask.", integer=True)
            out["keep_first"] = 0
            if isinstance(mask, dict) and mask.get("keep_first") is not None:
                out["keep_first"] = number(mask, "keep_first", where + "mask.", integer=True, positive=False)
                if out["keep_first"] < 0:
                    problems.append(f"{where}mask.'keep_first' must not be negative, got {out['keep_first']}")
            return out

        def latent(m, where):
            out = integers(m, where, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            out["scale"] = number(m, "scale", where, positive=False)
            rot, rw = m.get("rot"), where + "rot."
            out["rot"] = {"base": number(rot, "base", rw), "dims": number(rot, "dims", rw, integer=True), "scaling": None}
            if out["rot"]["dims"] != out["rot_dim"] or out["rot_dim"] % 2:
                problems.append(f"{rw}dims {out['rot']['dims']} must be rot_dim {out['rot_dim']}, an even number")
            if isinstance(rot, dict) and rot.get("scaling") is not None:
                out["rot"]["scaling"] = {k: number(rot["scaling"], k, rw + "scaling.") for k in ("factor", "original", "fast", "slow")}
            return out

        def pair(m, where):
            left, right = m.get("left"), m.get("right")
            if not isinstance(left, dict) or not isinstance(right, dict):
                problems.append(f"{where}'left' and {where}'right' must be objects")
                return None
            lw, rw = where + "left.", where + "right."
            l = heads(left, lw)
            l["softcap"] = 0.0 if left.get("softcap") is None else number(left, "softcap", lw)
            temp = left.get("q_temp")
            l["q_temp"] = None if temp is None else (number(temp, "coef", lw + "q_temp.", positive=False), number(temp, "every", lw + "q_temp.", integer=True))
            r = integers(right, rw, ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
            if r["heads"] % r["groups"]:
                problems.append(f"{rw}heads {r['heads']} is no multiple of groups {r['groups']}")
            if (r["heads"] * r["vdim"]) % r["norm_groups"]:
                problems.append(f"{rw}heads * vdim {r['heads'] * r['vdim']} is no multiple of norm_groups {r['norm_groups']}")
            return {"left": l, "right": r, "left_scale": number(m, "left_scale", where, positive=False),
                    "right_scale": number(m, "right_scale", where, positive=False)}

        readers = {"attention": attention, "latent_attention": latent, "parallel": pair}
        vocab = number(cfg, "vocab", "", integer=True)
        width = number(cfg, "width", "", integer=True)
        eps = number(cfg.get("norm"), "eps", "norm.")
        raw_layers = cfg.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            problems.append("'layers' must be a non-empty list")
            raw_layers = []
        layers: List[RufisunLayer] = []
        for i, entry in enumerate(raw_layers):
            where = f"layers[{i}]."
            if not isinstance(entry, dict) or not isinstance(entry.get("mixer"), dict):
                problems.append(f"layers[{i}] must be an object with a 'mixer'")
                continue
            kind = entry.get("type")
            if kind not in readers:
                problems.append(f"{where}type {kind!r} is not a mixer of this design (known: {MIXERS})")
                continue
            mixer = readers[kind](entry["mixer"], where + "mixer.")
            mlp, checked = entry.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
                    problems.append(f"{where}mlp.kind {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not a "
                                    "feed-forward of this design (known: 'dense', 'moe')")
                elif mlp["kind"] == "dense":
                    checked = {"kind": "dense", "ff": number(mlp, "ff", where + "mlp.", integer=True)}
                else:
                    ro, rw = mlp.get("router"), where + "mlp.router."
                    checked = {"kind": "moe", "ff": number(mlp.get("expert"), "ff", where + "mlp.expert.", integer=True),
                               "experts": number(ro, "experts", rw, integer=True), "top": number(ro, "top", rw, integer=True),
                               "shared": None if mlp.get("shared") is None else number(mlp["shared"], "ff", where + "mlp.shared.", integer=True)}
                    if checked["top"] > checked["experts"]:
                        problems.append(f"{rw}top {checked['top']} exceeds the {checked['experts']} experts")
            layers.append(RufisunLayer(kind, mixer, checked))
        if problems:
            raise ConfigError("Rufisun config.json: " + "; ".join(problems))
        return cls(vocab=vocab, width=width, eps=eps, layers=layers)


def rufisun_model_spec(c: RufisunConfig) -> ModelSpec:
    layers, order, absent = [], [], []
    norm = lambda: PartSpec("tanh", {"size": c.width, "tensor_name": ""})
    two_layer = lambda ff, act: PartSpec("two_layer_mlp", {"hidden_size": c.width, "intermediate_size": ff, "activation": act, "tensor_names": NAMES})

    def softmax_attention(m, **more):
        return PartSpec("biased_window_attention", dict({
            "hidden_size": c.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
            "scale": m["scale"], "softcap": 0.0, "window": 0, "bias_reach": None, "eps": c.eps, "qk_norm": False, "output_gate": False,
            "sink": True, "precise_weights": True}, **more))

    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer.mixer
        if layer.kind == "attention":
            mixer = softmax_attention(m, window=m["window"], keep_first=m["keep_first"], bias_reach=m["bias_max"], output_gate=True)
        elif layer.kind == "latent_attention":
            rot = m["rot"]
            mixer = PartSpec("rotary_latent_attention", {
                "hidden_size": c.width, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_head_dim": m["vdim"],
                "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": m["scale"], "eps": c.eps, "gate": "none", "sink": True,
                "position": PartSpec("scaled_rope", {"theta": rot["base"], "rotary_dim": rot["dims"], "pairing": "interleaved",
                                                     "scaling": rot["scaling"]})})
        else:
            l, r = m["left"], m["right"]
            mixer = PartSpec("parallel", {
                "hidden_size": c.width, "left_scale": m["left_scale"], "right_scale": m["right_scale"],
                "left": softmax_attention(l, softcap=l["softcap"], temperature=l["q_temp"]),
                "right": PartSpec("state_dual", {"hidden_size": c.width, "num_heads": r["heads"], "v_head_dim": r["vdim"], "state": r["state"],
                                                 "groups": r["groups"], "taps": r["conv"], "norm_groups": r["norm_groups"], "eps": c.eps})})
        mlp = layer.mlp
        if mlp is None:
            ff = PartSpec("none")
            absent += [p + "norm2", p + "norm2.alpha", p + "norm2.b"]           # a file may still hold them
        elif mlp["kind"] == "dense":
            ff = two_layer(mlp["ff"], "relu_squared")
        else:
            ff = PartSpec("routed_experts", {"hidden_size": c.width, "expert_size": mlp["ff"], "num_experts": mlp["experts"], "num_identity": 0,
                                             "top": mlp["top"], "limit": 1.0, "activation": "gelu", "score": "sigmoid", "correction": False,
                                             "normalize": False, "weight_input": True,
                                             "shared": None if mlp["shared"] is None else two_layer(mlp["shared"], "gelu")})
        layers.append(LayerSpec(
            mixer=mixer, feed_forward=ff, mixer_norm=norm(), feed_forward_norm=norm() if mlp is not None else PartSpec("none"), block="prenorm",
            names={"mixer": p + "mix.", "feed_forward": p + "mlp.", "mixer_norm": p + "norm1", "feed_forward_norm": p + "norm2"},
        ))
        order.append(LayerCall(layer=i, cache=i))
    return ModelSpec(
        architecture="Rufisun",
        hidden_size=c.width,
        vocab_size=c.vocab,
        layers=layers,
        run_order=order,
        final_norm=norm(),
        tie_word_embeddings=True,
        max_position_embeddings=MAX_POSITIONS,
        embed_name="embed",
        final_norm_prefix="final.norm",
        ignored_tensors=absent,
        init_std=0.05,
        init_gain_std=0.05,
    )


@register_architecture("Rufisun", "rufisun")
def build_rufisun(config: dict):
    typed = RufisunConfig.from_dict(config)
    return typed, rufisun_model_spec(typed)
