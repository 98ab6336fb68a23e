"""Kasuvik: a decoder with a norm before and after every sublayer whose layers mix tokens either by a generalised delta
rule (a matrix per head that decays per key channel, forgets along the token's key and adds the token's key and value) or
by two mixers side by side: a windowed softmax attention that sees what lies before its window through mean keys and
values of blocks of tokens, and a selective state space; typed configuration and its description as parts.

config.json names the design in ``architecture`` and gives every size and constant:

    vocab, width, embedding.scale, norm.eps,
    layers[i] = {type: "general_delta", mixer: {heads, dim},
                 type: "parallel",      mixer: {left: {heads, kv_heads, dim, vdim, conv, scale, rot: {base, dims},
                                                       mask: {size, pool}},
                                                right: {inner, state, dt_rank, conv}},
                 mlp: null | {kind: "dense", ff}}

Layer i's tensors are ``l<i>.*``: ``norm1`` / ``norm1b`` around the mixer ``mix.*`` (``mix.left.*`` and ``mix.right.*`` in a
parallel layer), ``norm2`` / ``norm2b`` around the feed-forward ``mlp.*``; outside the layers ``embed``, ``final.norm`` and
``head``.  The inner width of the delta mixer's decay product (``w1`` / ``w2``) comes from the tensors alone.  What the
design fixes (the decay's rate exp(-1/2), 1e-6 in the unit keys, relu in the feed-forward, half the sum of the two
mixers, the interleaved rotation) is named here or in the parts.  The reference has no model of this kind
(src/core/engine.cpp:26-28).
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import List, Optional

from ..config.engine_config import ConfigError
from ..config.model_spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..config.registry import register_architecture

MAX_POSITIONS = 1 << 22              # no position table bounds a request; the cache does first
DELTA_DECAY_RATE = math.exp(-0.5)    # decay = exp(-rate * sigmoid(.))
MIX_SCALE = 0.5                      # half the sum of the two mixers' normed results


@dataclass
class KasuvikLayer:
    kind: str                        # "general_delta" or "parallel"
    mixer: dict                      # the layer's "mixer" object, checked
    ff: Optional[int] = None         # width of the feed-forward; None: no feed-forward


@dataclass
class KasuvikConfig:
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    layers: List[KasuvikLayer] = field(default_factory=list)

    @classmethod
    def from_dict(cls, cfg: dict) -> "KasuvikConfig":
        problems: List[str] = []

        def number(d, key, where, integer=False, positive=True):
            v = d.get(key) if isinstance(d, dict) else None
            if v is None:
                problems.append(f"missing {where}'{key}'")
                return 1
            ok = isinstance(v, int) if integer else isinstance(v, (int, float))
            if isinstance(v, bool) or not ok:
                problems.append(f"{where}'{key}' must be {'an integer' if integer else 'a number'}, got {v!r}")
                return 1
            if positive and not v > 0:
                problems.append(f"{where}'{key}' must be positive, got {v!r}")
                return 1
            return v

        def integers(d, where, keys):
            return {k: number(d, k, where, integer=True) for k in keys}

        def attention(m, where):
            out = integers(m, where, ("heads", "dim", "vdim", "conv"))
            out["kv_heads"] = out["heads"] if m.get("kv_heads") is None else number(m, "kv_heads", where, integer=True)
            if out["heads"] % out["kv_heads"]:
                problems.append(f"{where}heads {out['heads']} is no multiple of kv_heads {out['kv_heads']}")
            out["scale"] = float(number(m, "scale", where, positive=False))
            rot, mask = m.get("rot"), m.get("mask")
            out["rot"] = None
            if rot is not None:
                out["rot"] = {"base": float(number(rot, "base", where + "rot.")), "dims": number(rot, "dims", where + "rot.", integer=True)}
                if out["rot"]["dims"] % 2 or out["rot"]["dims"] > out["dim"]:
                    problems.append(f"{where}rot.dims {out['rot']['dims']} must be even and at most dim {out['dim']}")
            # no mask: every token is seen; a mask without pool: a plain sliding window
            out["window"] = 0 if mask is None else number(mask, "size", where + "mask.", integer=True)
            out["pool"] = 0 if mask is None or mask.get("pool") is None else number(mask, "pool", where + "mask.", integer=True)
            return out

        vocab = number(cfg, "vocab", "", integer=True)
        width = number(cfg, "width", "", integer=True)
        emb_scale = number(cfg.get("embedding"), "scale", "embedding.", positive=False)
        eps = number(cfg.get("norm"), "eps", "norm.")
        raw_layers = cfg.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            problems.append("'layers' must be a non-empty list")
            raw_layers = []
        layers: List[KasuvikLayer] = []
        for i, entry in enumerate(raw_layers):
            where = f"layers[{i}]."
            if not isinstance(entry, dict) or not isinstance(entry.get("mixer"), dict):
                problems.append(f"layers[{i}] must be an object with a 'mixer'")
                continue
            kind, m, mw = entry.get("type"), entry["mixer"], where + "mixer."
            if kind == "general_delta":
                mixer = integers(m, mw, ("heads", "dim"))
            elif kind == "parallel":
                left, right = m.get("left"), m.get("right")
                if not isinstance(left, dict) or not isinstance(right, dict):
                    problems.append(f"{mw}'left' and {mw}'right' must be objects")
                    continue
                mixer = {"left": attention(left, mw + "left."),
                         "right": integers(right, mw + "right.", ("inner", "state", "dt_rank", "conv"))}
            else:
                problems.append(f"{where}type {kind!r} is not a mixer of this design (known: 'general_delta', 'parallel')")
                continue
            mlp, ff = entry.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    problems.append(f"{where}mlp.kind {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not a "
                                    "feed-forward of this design (known: 'dense')")
                else:
                    ff = number(mlp, "ff", where + "mlp.", integer=True)
            layers.append(KasuvikLayer(kind, mixer, ff))
        if problems:
            raise ConfigError("Kasuvik config.json: " + "; ".join(problems))
        return cls(vocab=vocab, width=width, embedding_scale=float(emb_scale), eps=float(eps), layers=layers)


def kasuvik_model_spec(c: KasuvikConfig) -> ModelSpec:
    layers, order, absent = [], [], []
    norm = lambda: PartSpec("rmsnorm", {"size": c.width, "eps": c.eps, "tensor_name": ""})
    none = lambda: PartSpec("none")
    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer.mixer
        if layer.kind == "general_delta":
            mixer = PartSpec("general_delta", {"hidden_size": c.width, "num_heads": m["heads"], "head_dim": m["dim"],
                                               "v_head_dim": m["dim"], "decay_rate": DELTA_DECAY_RATE, "eps": c.eps})
        else:
            l, r = m["left"], m["right"]
            position = none() if l["rot"] is None else PartSpec("scaled_rope", {"theta": l["rot"]["base"], "rotary_dim": l["rot"]["dims"],
                                                                                "pairing": "interleaved", "scaling": None})
            mixer = PartSpec("parallel", {
                "hidden_size": c.width, "left_scale": MIX_SCALE, "right_scale": MIX_SCALE, "result_eps": c.eps,
                "left": PartSpec("pooled_window_attention", {
                    "hidden_size": c.width, "num_heads": l["heads"], "num_kv_heads": l["kv_heads"], "head_dim": l["dim"],
                    "v_head_dim": l["vdim"], "taps": l["conv"], "scale": l["scale"], "window": l["window"], "pool": l["pool"],
                    "position": position, "qkv_bias": True, "temperature": True}),
                "right": PartSpec("selective_state", {
                    "hidden_size": c.width, "inner": r["inner"], "state": r["state"], "dt_rank": r["dt_rank"], "taps": r["conv"]})})
        has_ff = layer.ff is not None
        if has_ff:
            ff = PartSpec("gated_mlp", {"hidden_size": c.width, "intermediate_size": layer.ff, "activation": "relu",
                                        "tensor_names": ("gate", "up", "down")})
        else:
            ff = none()
            absent += [p + "norm2", p + "norm2b"]                 # a file may still hold them
        layers.append(LayerSpec(
            mixer=mixer, feed_forward=ff, mixer_norm=norm(), mixer_post_norm=norm(), mixer_scale=none(),
            feed_forward_norm=norm() if has_ff else none(), feed_forward_post_norm=norm() if has_ff else none(),
            feed_forward_scale=none(), block="sandwich_norm",
            names={"mixer": p + "mix.", "feed_forward": p + "mlp.", "mixer_norm": p + "norm1", "mixer_post_norm": p + "norm1b",
                   "mixer_scale": p + "ls1", "feed_forward_norm": p + "norm2", "feed_forward_post_norm": p + "norm2b",
                   "feed_forward_scale": p + "ls2"},
        ))
        order.append(LayerCall(layer=i, cache=i))
    return ModelSpec(
        architecture="Kasuvik",
        hidden_size=c.width,
        vocab_size=c.vocab,
        layers=layers,
        run_order=order,
        final_norm=norm(),
        tie_word_embeddings=False,
        max_position_embeddings=MAX_POSITIONS,
        embed_name="embed",
        final_norm_prefix="final.norm",
        lm_head_name="head",
        ignored_tensors=absent,
        init_std=0.05,
        init_gain_std=0.05,
        model_class="scaled_embedding_decoder",
        model_params={"embedding_scale": c.embedding_scale},
    )


@register_architecture("Kasuvik", "kasuvik")
def build_kasuvik(config: dict):
    typed = KasuvikConfig.from_dict(config)
    return typed, kasuvik_model_spec(typed)
