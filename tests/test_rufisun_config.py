"""The Rufisun design without a GPU: its configuration reader, its description as parts, the tensors it declares, the caches its
mixers ask for (a window whose pages of the first tokens stay), the stretched frequencies, the distance buckets, and the plain
implementation's own consistency."""
import copy
import math
import random

import numpy as np
import pytest
import torch

import plain_rufisun as plain


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": None if shared is None else {"ff": shared}}


def att(heads, kv_heads, dim, vdim, scale=0.3, bias_max=40, mask=(20, 3), mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
         "mask": {"size": mask[0], "keep_first": mask[1]}}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def lat(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale=0.25, base=500.0, scaling=(4.0, 64, 8.0, 0.5), mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                  "scale": scale, "rot": rot}, "mlp": mlp}


def cap(heads, kv_heads, dim, vdim, scale=0.3, softcap=6.0, q_temp=(0.4, 11)):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
            "q_temp": {"coef": q_temp[0], "every": q_temp[1]}}


def ssd(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def par(left, right, scales=(0.7, 1.2), mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def config(layers, width=48, vocab=150, eps=1e-5):
    return {"architecture": "Rufisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


SAMPLE = config([att(6, 2, 12, 20, mlp=dense(40)), lat(3, 10, 6, 14, 20, 24, mlp=moe(16, 5, 2, shared=24)),
                 par(cap(4, 4, 16, 16), ssd(6, 8, 12, groups=3, norm_groups=2), mlp=moe(20, 4, 1)),
                 att(2, 1, 8, 8, bias_max=33.5, mask=(9, 0)), par(cap(2, 1, 8, 12), ssd(2, 10, 5, conv=1))])


def test_config_is_read_and_described_as_parts():
    from vllm_cpp_b200.config.registry import resolve_architecture
    typed, spec = resolve_architecture(SAMPLE)
    assert (typed.width, typed.vocab, typed.eps) == (48, 150, 1e-5)
    assert [l.kind for l in typed.layers] == ["attention", "latent_attention", "parallel", "attention", "parallel"]
    assert spec.tie_word_embeddings and spec.model_class == "decoder" and all(l.block == "prenorm" for l in spec.layers)
    a = spec.layers[0].mixer
    assert a.kind == "biased_window_attention"
    assert {k: a.params[k] for k in ("window", "keep_first", "bias_reach", "softcap", "scale", "sink", "output_gate", "qk_norm", "precise_weights")} == \
        {"window": 20, "keep_first": 3, "bias_reach": 40.0, "softcap": 0.0, "scale": 0.3, "sink": True, "output_gate": True, "qk_norm": False,
         "precise_weights": True}
    l = spec.layers[1].mixer
    assert l.kind == "rotary_latent_attention" and l.params["sink"] and l.params["gate"] == "none" and l.params["q_rank"] == 24
    assert l.params["position"].params == {"theta": 500.0, "rotary_dim": 6, "pairing": "interleaved",
                                           "scaling": {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 0.5}}
    p = spec.layers[2].mixer
    assert p.kind == "parallel" and (p.params["left_scale"], p.params["right_scale"]) == (0.7, 1.2) and "result_eps" not in p.params
    left, right = p.params["left"], p.params["right"]
    assert left.kind == "biased_window_attention" and left.params["bias_reach"] is None and left.params["temperature"] == (0.4, 11)
    assert left.params["softcap"] == 6.0 and not left.params["output_gate"] and left.params["window"] == 0
    assert right.kind == "state_dual" and right.params["groups"] == 3 and right.params["norm_groups"] == 2
    ffs = [l.feed_forward for l in spec.layers]
    assert ffs[0].params["activation"] == "relu_squared" and ffs[1].params["shared"].params["activation"] == "gelu"
    assert ffs[1].params["weight_input"] and ffs[1].params["score"] == "sigmoid" and not ffs[1].params["normalize"]
    assert ffs[2].params["shared"] is None and ffs[3].kind == ffs[4].kind == "none"
    assert all(l.mixer_norm.kind == "tanh" for l in spec.layers) and spec.final_norm.kind == "tanh"
    assert resolve_architecture(SAMPLE, "rufisun")[1].architecture == "Rufisun"
    # what may be absent: kv_heads (one for every query head), the cap, the growing queries, the stretching, the mask
    cfg = copy.deepcopy(SAMPLE)
    del cfg["layers"][0]["mixer"]["kv_heads"], cfg["layers"][0]["mixer"]["mask"]
    del cfg["layers"][1]["mixer"]["rot"]["scaling"], cfg["layers"][2]["mixer"]["left"]["softcap"], cfg["layers"][2]["mixer"]["left"]["q_temp"]
    typed, spec = resolve_architecture(cfg)
    assert typed.layers[0].mixer["kv_heads"] == 6 and spec.layers[0].mixer.params["window"] == 0
    assert spec.layers[1].mixer.params["position"].params["scaling"] is None
    assert spec.layers[2].mixer.params["left"].params["softcap"] == 0.0 and spec.layers[2].mixer.params["left"].params["temperature"] is None


def test_tensors_declared_are_the_design_s():
    from vllm_cpp_b200.config.registry import resolve_architecture
    from vllm_cpp_b200.parts.model import build_model
    _, spec = resolve_architecture(SAMPLE)
    declared = {k: tuple(v.shape) for k, v in build_model(spec, torch.float32, "meta").param_specs().items()}
    assert declared == plain.tensor_shapes(SAMPLE, bias_rows=-1)


def test_cache_layers():
    from vllm_cpp_b200.config.registry import resolve_architecture
    from vllm_cpp_b200.parts.base import CompositeSpec, PagedKVSpec, StateSpec
    from vllm_cpp_b200.parts.model import build_model
    _, spec = resolve_architecture(SAMPLE)
    specs = build_model(spec, torch.bfloat16, "meta").cache_specs()
    assert specs[0] == PagedKVSpec(2, 20, 20, keep_first=3)
    assert specs[1] == PagedKVSpec(1, 26, 0, planes=1)
    left, right = specs[2].parts
    assert left == PagedKVSpec(4, 16, 0) and right == CompositeSpec((StateSpec((6, 12, 8)), StateSpec((3, 48 + 2 * 3 * 12))))
    assert specs[3] == PagedKVSpec(1, 8, 9)
    assert specs[4].parts[1] == CompositeSpec((StateSpec((2, 5, 10)), StateSpec((1, 20 + 2 * 5))))       # one tap keeps nothing


@pytest.mark.parametrize("change,message", [
    (lambda c: c["norm"].pop("eps"), "norm.'eps'"),
    (lambda c: c.pop("vocab"), "'vocab'"),
    (lambda c: c["layers"][0].update(type="conv"), "not a mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("bias_max"), "'bias_max'"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "no multiple"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "mask.'size'"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "not a"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=5), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "'slow'"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "exceeds"),
    (lambda c: c["layers"][2]["mixer"].pop("right"), "'right'"),
    (lambda c: c["layers"][2]["mixer"].pop("left_scale"), "'left_scale'"),
    (lambda c: c["layers"][2]["mixer"]["right"].update(groups=4), "no multiple of groups"),
    (lambda c: c["layers"][2]["mixer"]["right"].update(norm_groups=5), "no multiple of norm_groups"),
    (lambda c: c["layers"][2]["mixer"]["left"]["q_temp"].update(every=0), "'every'"),
    (lambda c: c["layers"][2]["mixer"]["right"].update(state=True), "state"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_what_the_reader_refuses(change, message):
    from vllm_cpp_b200.config.engine_config import ConfigError
    from vllm_cpp_b200.models.rufisun import RufisunConfig
    cfg = copy.deepcopy(SAMPLE)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        RufisunConfig.from_dict(cfg)


# ------------------------------------------------------------------ a window whose first tokens stay
@pytest.mark.parametrize("window,keep,page", [(20, 3, 8), (5, 8, 8), (5, 9, 8), (1, 1, 4), (30, 70, 16), (7, 0, 8), (64, 16, 16)])
def test_pages_of_the_first_tokens_stay(window, keep, page):
    """Every token that a later query sees is still in a page, whatever the steps; the others go back and are handed out again."""
    from vllm_cpp_b200.cache.manager import CacheManager
    from vllm_cpp_b200.parts.base import PagedKVSpec
    for seed in range(6):
        rng = random.Random(seed)
        m = CacheManager([PagedKVSpec(1, 4, window, keep_first=keep)], page, 60, 2)
        m.add_request("a")
        n = 0
        while n < 230:
            step = min(rng.choice([1, 1, 2, 7, 30]), 230 - n)
            table = m.table("a", 0)
            seen = [j for j in range(n) if n - j < window or j < keep]
            assert all(table[j // page] >= 0 for j in seen)
            m.reserve("a", step)
            n += step
            m.commit("a", step)
            gone = [b for b, pg in enumerate(m.table("a", 0)) if pg < 0]
            assert gone == list(range(-(-keep // page), max(-(-keep // page), max(0, n - window + 1) // page)))
            rows = m.table_rows(0, 60)[m.slot("a")]
            assert all((rows[b] < 0) == (b in gone or b >= len(m.table("a", 0))) for b in range(60))
        held = len(m.table("a", 0)) - len(gone)
        assert m.num_free_pages() == 60 - held
        m.free_request("a")
        assert m.num_free_pages() == 60


def test_decode_splits_count_the_kept_tokens():
    """The work of a decode step over a window and kept tokens: one tile for each 64 keys of either, wherever they are."""
    from types import SimpleNamespace
    from vllm_cpp_b200.csrc import ops
    from vllm_cpp_b200.parts.biased_attention import BiasedWindowAttention
    a = BiasedWindowAttention(64, 4, 4, 64, 64, 0.1, 0.0, 128, 500.0, 1e-5, torch.bfloat16, "meta", qk_norm=False, keep_first=70, sink=True,
                              precise_weights=True)
    assert a.keep_first == 70 and a.cache_spec().keep_first == 70
    real, ops._sm_count = ops._sm_count, 148
    try:
        key = a._splits_key()
        assert key.endswith("_k70")
        host = SimpleNamespace(q_lens=[1], ctx_lens=[5000], shapes={}, page_size=16)
        per = int(a.step_arrays()[key](host)[0])
        # the window's 128 keys lie in three tiles, the kept 70 in two
        assert -(-5 // per) <= host.shapes[key] and per >= 1
    finally:
        ops._sm_count = real
    # without a window everything is seen anyway
    assert BiasedWindowAttention(64, 4, 4, 64, 64, 0.1, 0.0, 0, 500.0, 1e-5, torch.bfloat16, "meta", keep_first=5).keep_first == 0


# ------------------------------------------------------------------ frequencies, buckets
@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(16, 1e4, 8.0, 512, 16.0, 1.0), (8, 300.0, 2.0, 4096, 64.0, 2.0), (64, 1e6, 40.0, 4096, 32.0, 1.0),
                                                                 (2, 50.0, 3.0, 100, 4.0, 1.0), (6, 500.0, 4.0, 64, 8.0, 0.5), (12, 20.0, 5.0, 1000, 1.0, 1.0)])
def test_stretched_frequencies(dims, base, factor, original, fast, slow):
    from vllm_cpp_b200.parts.position import ScaledRotaryEmbedding
    enc = ScaledRotaryEmbedding(base, dims, "interleaved", {"factor": factor, "original": original, "fast": fast, "slow": slow}, device="cpu")
    want = plain.stretched_frequencies(dims, base, factor, original, fast, slow)
    assert np.allclose(enc.inv_freq.numpy(), want, rtol=1e-6) and abs(enc.magnitude - (0.1 * math.log(factor) + 1)) < 1e-12
    # a frequency is never raised, and never divided by more than the factor
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    assert (want <= f * (1 + 1e-12)).all() and (want >= f / factor * (1 - 1e-12)).all()
    assert ScaledRotaryEmbedding(base, dims, "interleaved", None, device="cpu").magnitude == 1.0


def test_mixers_without_a_factor_refuse_it():
    from vllm_cpp_b200.config.model_spec import PartSpec
    from vllm_cpp_b200.parts import model  # noqa: F401
    from vllm_cpp_b200.parts.sink_attention import SinkAttention
    pos = PartSpec("scaled_rope", {"theta": 100.0, "rotary_dim": 8, "pairing": "half", "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}})
    with pytest.raises(ValueError, match="factor"):
        SinkAttention(32, 2, 1, 16, 16, 0.1, 1e-5, pos, torch.float32, "cpu")


@pytest.mark.parametrize("rows,reach", [(24, 90), (8, 40), (64, 1000.0), (5, 7.5), (2, 9)])
def test_distance_buckets(rows, reach):
    from vllm_cpp_b200.parts.biased_attention import distance_buckets
    want = [plain.bias_bucket(n, rows, reach) for n in range(1200)]
    assert distance_buckets(rows, reach, 1200).tolist() == want
    assert want[0] == 0 and want[-1] == rows - 1 and all(a <= b for a, b in zip(want, want[1:]))
    # the table a kernel reads is constant from the reach on
    assert all(b == rows - 1 for b in want[int(math.ceil(reach)):])


# ------------------------------------------------------------------ the plain implementation itself
def test_plain_is_causal_and_continues():
    w = plain.random_weights(SAMPLE, 3)
    ids = np.random.default_rng(1).integers(0, 150, size=30).tolist()
    assert np.allclose(plain.forward(SAMPLE, w, ids)[:17], plain.forward(SAMPLE, w, ids[:17]))
    rng = np.random.default_rng(2)
    x, dt, B, C = rng.standard_normal((9, 4, 5)), rng.random((9, 4)), rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 3))
    A, D = -rng.random(4), rng.standard_normal(4)
    y, S = plain.decaying_outer_products(x, dt, A, B, C, D)
    y1, S1 = plain.decaying_outer_products(x[:4], dt[:4], A, B[:4], C[:4], D)
    y2, S2 = plain.decaying_outer_products(x[4:], dt[4:], A, B[4:], C[4:], D, S1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S2, S)


def test_plain_dual_form():
    """The recurrence is a masked attention: y_t = sum_(s <= t) (prod of decays s + 1 .. t) (C_t . B_s) dt_s x_s + D x_t."""
    rng = np.random.default_rng(4)
    n, H, G, N, P = 12, 4, 2, 3, 5
    x, dt, B, C = rng.standard_normal((n, H, P)), rng.random((n, H)), rng.standard_normal((n, G, N)), rng.standard_normal((n, G, N))
    A, D = -rng.random(H) * 2, rng.standard_normal(H)
    y, _ = plain.decaying_outer_products(x, dt, A, B, C, D)
    for h in range(H):
        total = np.cumsum(A[h] * dt[:, h])
        M = np.tril(np.exp(total[:, None] - total[None, :]) * (C[:, h // 2] @ B[:, h // 2].T) * dt[None, :, h])
        assert np.allclose(M @ x[:, h] + D[h] * x[:, h], y[:, h])


def test_plain_sink_and_weights_on_inputs():
    rng = np.random.default_rng(5)
    q, k, v = rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 2, 3))
    free = plain.attention_core(q, k, v, 0.5, np.full(2, -1e9))
    half = plain.attention_core(q[:1], k[:1], v[:1], 0.0, np.zeros(2))       # one key of score 0 beside a sink of 0
    assert np.allclose(free[0], v[0]) and np.allclose(half[0], v[0] / 2)
    h = rng.standard_normal((3, 8))
    w = {"up": rng.standard_normal((5, 8)), "down": rng.standard_normal((8, 5))}
    assert np.abs(plain.expert_ff(0.3 * h, w, "") - 0.3 * plain.expert_ff(h, w, "")).max() > 0.05      # it matters where the weight goes
