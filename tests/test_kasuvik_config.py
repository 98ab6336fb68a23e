"""The Kasuvik design without a GPU: its configuration reader, its description as parts, the tensors it declares, the
caches its mixers ask for (a window's pages that keep an unfinished block, pages of one row per block), and the plain
implementation's own consistency."""
import copy
import random

import numpy as np
import pytest
import torch

import plain_kasuvik as plain


def gdelta(heads, dim, ff=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def att(heads, kv_heads, dim, vdim, conv=3, scale=0.3, rot=(4, 100.0), mask=(20, 6)):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale}
    if rot is not None:
        out["rot"] = {"dims": rot[0], "base": rot[1]}
    if mask is not None:
        out["mask"] = {"size": mask[0], "pool": mask[1]} if mask[1] else {"size": mask[0]}
    return out


def sel(inner, state, dt_rank, conv=4):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def par(left, right, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=48, vocab=150, scale=0.7, eps=1e-5):
    return {"architecture": "Kasuvik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


SAMPLE = config([gdelta(3, 8, ff=40), par(att(6, 2, 12, 20), sel(36, 5, 7), ff=56), gdelta(2, 20),
                 par(att(4, 4, 16, 16, conv=1, rot=None, mask=(33, 0)), sel(24, 16, 3, conv=1)),
                 par(att(2, 1, 8, 8, mask=None), sel(20, 3, 2, conv=2), ff=32)])


def test_config_is_read_and_described_as_parts():
    from vllm_cpp_b200.config.registry import resolve_architecture
    typed, spec = resolve_architecture(SAMPLE)
    assert (typed.width, typed.vocab, typed.eps, typed.embedding_scale) == (48, 150, 1e-5, 0.7)
    assert [l.kind for l in typed.layers] == ["general_delta", "parallel", "general_delta", "parallel", "parallel"]
    assert [l.ff for l in typed.layers] == [40, 56, None, None, 32]
    lefts = [l.mixer["left"] for l in typed.layers if l.kind == "parallel"]
    assert [(l["window"], l["pool"]) for l in lefts] == [(20, 6), (33, 0), (0, 0)]
    assert spec.model_class == "scaled_embedding_decoder" and spec.model_params == {"embedding_scale": 0.7}
    assert not spec.tie_word_embeddings and spec.lm_head_name == "head"
    assert all(l.block == "sandwich_norm" for l in spec.layers)
    d = spec.layers[0].mixer
    assert d.kind == "general_delta" and abs(d.params["decay_rate"] - np.exp(-0.5)) < 1e-15 and d.params["v_head_dim"] == 8
    p = spec.layers[1].mixer
    assert p.kind == "parallel" and (p.params["left_scale"], p.params["right_scale"], p.params["result_eps"]) == (0.5, 0.5, 1e-5)
    assert p.params["left"].params["position"].params == {"theta": 100.0, "rotary_dim": 4, "pairing": "interleaved", "scaling": None}
    assert spec.layers[3].mixer.params["left"].params["position"].kind == "none"
    assert spec.layers[1].feed_forward.params["activation"] == "relu" and spec.layers[2].feed_forward.kind == "none"
    assert resolve_architecture(SAMPLE, "kasuvik")[1].architecture == "Kasuvik"
    # kv_heads absent: a key/value head for every query head
    cfg = copy.deepcopy(SAMPLE)
    del cfg["layers"][1]["mixer"]["left"]["kv_heads"]
    assert resolve_architecture(cfg)[0].layers[1].mixer["left"]["kv_heads"] == 6


def test_tensors_declared_are_the_design_s():
    from vllm_cpp_b200.config.registry import resolve_architecture
    from vllm_cpp_b200.parts.model import build_model
    _, spec = resolve_architecture(SAMPLE)
    declared = {k: tuple(v.shape) for k, v in build_model(spec, torch.float32, "meta").param_specs().items()}
    assert declared == plain.tensor_shapes(SAMPLE, rank=-1)


def test_cache_layers():
    from vllm_cpp_b200.cache.manager import CacheManager
    from vllm_cpp_b200.config.registry import resolve_architecture
    from vllm_cpp_b200.parts.base import CompositeSpec, PagedKVSpec, StateSpec
    from vllm_cpp_b200.parts.model import build_model
    _, spec = resolve_architecture(SAMPLE)
    specs = build_model(spec, torch.bfloat16, "meta").cache_specs()
    assert specs[0] == StateSpec((3, 8, 8)) and specs[2] == StateSpec((2, 20, 20))
    left, right = specs[1].parts
    assert left == CompositeSpec((PagedKVSpec(2, 20, 20, keep_block=6), PagedKVSpec(2, 20, stride=6), StateSpec((2, 6 * 12 + 2 * 32))))
    assert right == CompositeSpec((StateSpec((36, 5)), StateSpec((3, 36))))
    assert specs[3].parts[0] == CompositeSpec((PagedKVSpec(4, 16, 33), StateSpec((1, 4 * 48))))       # no blocks; one tap keeps nothing
    assert specs[4].parts[0].parts[0] == PagedKVSpec(1, 8, 0)
    page = 16
    assert CacheManager.bytes_per_page(specs, page, torch.bfloat16) == 2 * page * 2 * (2 * 20 + 4 * 16 + 8) + -(-2 * page * 2 * 2 * 20 // 6)
    assert CacheManager.fixed_bytes(specs, page, 3, torch.bfloat16) == 4 * 2 * page * 2 * 2 * 20


@pytest.mark.parametrize("change,message", [
    (lambda c: c["embedding"].pop("scale"), "embedding.'scale'"),
    (lambda c: c["norm"].pop("eps"), "norm.'eps'"),
    (lambda c: c["layers"][0].update(type="conv"), "not a mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "'dim'"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "'right'"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "no multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=14), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].pop("size"), "mask.'size'"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(pool=-2), "pool"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(state=True), "state"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "not a"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_what_the_reader_refuses(change, message):
    from vllm_cpp_b200.config.engine_config import ConfigError
    from vllm_cpp_b200.models.kasuvik import KasuvikConfig
    cfg = copy.deepcopy(SAMPLE)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        KasuvikConfig.from_dict(cfg)


# ------------------------------------------------------------------ pages of blocks, pages that keep a block
def manager(window, pool, pages=12, seqs=3, page=8):
    from vllm_cpp_b200.cache.manager import CacheManager
    from vllm_cpp_b200.parts.base import CompositeSpec, PagedKVSpec, StateSpec
    spec = CompositeSpec((PagedKVSpec(1, 4, window, keep_block=pool), PagedKVSpec(1, 4, stride=pool), StateSpec((2, 3))))
    return CacheManager([spec], page, pages, seqs)


def test_pages_of_blocks_follow_the_complete_blocks():
    m = manager(window=20, pool=6)
    assert m.paged[1].pool.num_blocks == 2 + 3                      # a sixth of the tokens' pages and one a request
    m.add_request("a")
    assert m.pages_needed("a", 5) == [1, 0] and m.pages_needed("a", 6) == [1, 1]
    assert m.pages_needed("a", 53) == [7, 1] and m.pages_needed("a", 54) == [7, 2]      # the ninth block starts a second page
    m.reserve("a", 5)
    m.commit("a", 5)
    assert m.table("a", 1) == []
    m.reserve("a", 49)
    m.commit("a", 49)
    assert len(m.table("a", 1)) == 2
    m.free_request("a")
    assert m.num_free_pages() == 12 and m.paged[1].pool.num_free == 5


@pytest.mark.parametrize("window,pool", [(20, 6), (3, 40), (8, 8), (1, 1), (5, 17)])
def test_tokens_of_an_unfinished_block_are_kept(window, pool):
    """Every token that a later query or a later block mean reads is still in a page, whatever the steps; pages of tokens
    that nothing reads again go back."""
    page = 8
    for seed in range(6):
        rng = random.Random(seed)
        m = manager(window, pool, pages=30, seqs=1, page=page)
        m.add_request("a")
        n = 0
        while n < 200:
            step = min(rng.choice([1, 1, 2, 7, 30]), 200 - n)
            table = m.table("a", 0)
            first_query, first_block = max(0, n - window + 1), n // pool * pool
            needed = {j // page for j in range(first_query, n)} | {j // page for j in range(first_block, n)}
            assert all(table[b] >= 0 for b in needed)
            m.reserve("a", step)
            n += step
            m.commit("a", step)
            dead = min(max(0, n - window + 1), n // pool * pool) // page
            assert [b for b, pg in enumerate(m.table("a", 0)) if pg < 0] == list(range(dead))
            assert len(m.table("a", 1)) == -(-(n // pool) // page)
        m.free_request("a")
        assert m.num_free_pages() == 30


def test_what_fits_the_tokens_pages_fits_the_blocks_pages():
    """Requests of any mixture whose tokens fit the pool (no window: none come back) never run out of pages of blocks."""
    from vllm_cpp_b200.cache.manager import CacheManager
    from vllm_cpp_b200.parts.base import PagedKVSpec
    for seed in range(20):
        rng = random.Random(seed)
        page, pages, seqs, pool = rng.choice([4, 8, 16]), rng.randrange(4, 40), rng.randrange(1, 6), rng.randrange(1, 30)
        m = CacheManager([PagedKVSpec(1, 4), PagedKVSpec(1, 4, stride=pool)], page, pages, seqs)
        live = []
        for step in range(200):
            if rng.random() < 0.2 and m.has_free_slot():
                m.add_request(step)
                live.append(step)
            elif live:
                r = rng.choice(live)
                if rng.random() < 0.1:
                    m.free_request(r)
                    live.remove(r)
                    continue
                room = m.paged[0].pool.num_free * page + (-m.num_tokens(r)) % page
                n = min(rng.choice([1, 3, 17, 60]), room)
                assert m.max_appendable(r) >= room
                if n:
                    m.reserve(r, n)
                    m.commit(r, n)


# ------------------------------------------------------------------ the plain implementation itself
def test_plain_visibility():
    for size, pool in ((5, 3), (1, 1), (7, 10), (4, 4)):
        for i in range(60):
            first, blocks = plain.pooled_visibility(i, size, pool)
            assert [j for j in range(i + 1) if 0 <= i - j < size] == list(range(first, i + 1))
            assert [b for b in range(60) if b * pool + pool - 1 <= i - size] == list(range(blocks))
    assert plain.pooled_visibility(9, None, None) == (0, 0) and plain.pooled_visibility(9, 4, None) == (6, 0)


def test_plain_delta_rule_forgets_along_the_unit_key():
    """With no decay and full removal, a token whose key was written before replaces what the key held."""
    rng = np.random.default_rng(0)
    k = rng.standard_normal(6)
    k /= np.linalg.norm(k)
    ks = np.stack([k, k * 3.0])[:, None]
    v = rng.standard_normal((2, 1, 4))
    one = np.ones((2, 1, 6))
    o, S = plain.general_delta_core(ks, ks, v, one, one)
    assert np.allclose(S[0], np.outer(k * 3.0, v[1, 0]), atol=1e-5) and np.allclose(o[1, 0], 9.0 * v[1, 0], atol=1e-4)


def test_plain_is_causal_and_continues():
    cfg = config([par(att(4, 2, 8, 6, mask=(5, 3)), sel(12, 4, 3), ff=16), gdelta(2, 4, ff=20)], width=16, vocab=30)
    w = plain.random_weights(cfg, 3)
    ids = np.random.default_rng(1).integers(0, 30, size=24).tolist()
    assert np.allclose(plain.forward(cfg, w, ids)[:17], plain.forward(cfg, w, ids[:17]))
    rng = np.random.default_rng(2)
    x, dt, B, C = rng.standard_normal((9, 5)), rng.random((9, 5)), rng.standard_normal((9, 3)), rng.standard_normal((9, 3))
    A, D = -rng.random((5, 3)), rng.standard_normal(5)
    y, S = plain.selective_scan_core(x, dt, A, B, C, D)
    y1, S1 = plain.selective_scan_core(x[:4], dt[:4], A, B[:4], C[:4], D)
    y2, S2 = plain.selective_scan_core(x[4:], dt[4:], A, B[4:], C[4:], D, S1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S2, S)
