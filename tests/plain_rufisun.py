"""A plain, slow implementation of the Rufisun design in numpy (float64), one function per mechanism, written from the
design's equations.  It shares no code with the engine: the tests compare the engine with it.

The design.  A pre-norm decoder: x += mixer(norm1(x)), then x += feed_forward(norm2(x)), where the norm is a tanh with a learned
slope and an affine map per coordinate and no statistics.  The embedding table is also the output matrix.  Mixers:

  "attention"         grouped-query softmax attention without rotation: a learned bias by bucket of distance and head joins the
                      scaled score; a query sees a sliding window and the first few tokens of the sequence; a learned number per
                      head joins the denominator; the concatenated heads pass a sigmoid gate before the output product.
  "latent_attention"  keys and values are projections of a normed low-rank row per token; queries pass a normed low-rank row
                      too; positions enter through a rotated part (interleaved pairs, frequencies rescaled between two
                      borders of wavelength, cosine and sine with a factor) that the heads' keys share; causal, with the
                      same number per head in the denominator.
  "parallel"          two mixers on the same input, joined with two constants.  Left: grouped-query attention whose queries grow
                      with the logarithm of the position's bucket, whose scores are capped by a tanh, with the number in the
                      denominator.  Right: a matrix per head that decays by one number per token and head and takes up an outer
                      product, behind a short convolution, its result gated and then normed in equal parts.

Feed-forwards: dense with the square of relu, or experts (the exact gelu between two matrices) chosen by sigmoid scores, the
score multiplying what the expert reads, beside a shared expert.
"""
import math

import numpy as np
from scipy.special import erf

from plain_kasuvik import perturbed, product, rms, rounded_like_bf16, short_conv, sigmoid, silu, softplus  # noqa: F401
from plain_gipinex import read_model_folder, read_safetensors, round_to_bf16, write_model_folder  # noqa: F401

BIAS_ROWS = 20          # rows of the distance-bias table that random_weights makes


# ------------------------------------------------------------- shapes and random weights
def kv_heads(m):
    return m.get("kv_heads") or m["heads"]


def tensor_shapes(cfg, bias_rows=BIAS_ROWS):
    """name -> shape of every tensor a model of this configuration has; ``bias_rows``: no configuration key gives it."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W)}

    def norm(name):
        out.update({name: (W,), name + ".alpha": (), name + ".b": (W,)})

    def expert(p, ff):
        out.update({p + "up": (ff, W), p + "down": (W, ff)})

    def heads(p, m):
        H, G = m["heads"], kv_heads(m)
        out.update({p + "q": (H * m["dim"], W), p + "k": (G * m["dim"], W), p + "v": (G * m["vdim"], W), p + "sink": (H,), p + "o": (W, H * m["vdim"])})

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        q = p + "mix."
        if layer["type"] == "attention":
            heads(q, m)
            out.update({q + "rel": (bias_rows, m["heads"]), q + "g": (m["heads"] * m["vdim"], W)})
        elif layer["type"] == "latent_attention":
            H = m["heads"]
            out.update({q + "dq": (m["q_rank"], W), q + "dq.norm": (m["q_rank"],), q + "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                        q + "dkv": (m["kv_rank"] + m["rot_dim"], W), q + "dkv.norm": (m["kv_rank"],), q + "uk": (H * m["dim"], m["kv_rank"]),
                        q + "uv": (H * m["vdim"], m["kv_rank"]), q + "sink": (H,), q + "o": (W, H * m["vdim"])})
        else:
            heads(q + "left.", m["left"])
            r = m["right"]
            I = r["heads"] * r["vdim"]
            C = I + 2 * r["groups"] * r["state"]
            q += "right."
            out.update({q + "in": (I + C + r["heads"], W), q + "conv": (C, r["conv"]), q + "conv.b": (C,), q + "dt_bias": (r["heads"],),
                        q + "A_log": (r["heads"],), q + "D": (r["heads"],), q + "norm": (I,), q + "o": (W, I)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        norm(p + "norm2")
        p += "mlp."
        if mlp["kind"] == "dense":
            expert(p, mlp["ff"])
            continue
        for e in range(mlp["router"]["experts"]):
            expert(f"{p}e{e}.", mlp["expert"]["ff"])
        out[p + "router"] = (mlp["router"]["experts"], W)
        if mlp.get("shared"):
            expert(p + "shared.", mlp["shared"]["ff"])
    return out


def random_weights(cfg, seed, sharp=1.0, bias_rows=BIAS_ROWS, decisive_routing=False):
    """Matrices of standard deviation fan_in^(-1/2); queries and keys times ``sharp`` (peaked scores, so that a wrong key shows);
    sinks and distance biases large enough to show; decays and step sizes spread over their ranges.  ``decisive_routing``: a few
    coordinates of the second norm's result are constants that the routers read above all, so that no rounding turns a choice."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, bias_rows).items():
        x = rng.standard_normal(shape)
        tail = name.split(".")[-1]
        if name == "embed":
            w = x
        elif tail == "alpha":
            w = 0.5 + 0.3 * rng.random()
        elif tail in ("norm", "norm1", "norm2", "D"):
            w = 1.0 + 0.2 * x
        elif tail == "rel":
            w = 1.5 * x
        elif tail == "sink":
            w = 1.0 + x
        elif tail == "conv":
            w = 0.4 * x
            w[:, -1] += 1.0
        elif tail == "A_log":
            w = np.log(np.linspace(0.3, 4.0, shape[0])) + 0.2 * x
        elif tail == "dt_bias":
            w = -1.5 + x
        elif tail == "b":
            w = 0.2 * x
        else:
            w = x / math.sqrt(shape[1])
            if tail in ("q", "k", "uq", "uk"):
                w = w * sharp
        out[name] = np.asarray(w, dtype=np.float64)
    if decisive_routing:
        for name, r in out.items():
            if name.endswith("mlp.router"):
                p, E = name.split("mlp.")[0], r.shape[0]
                r *= 0.05
                pick = min(6, cfg["width"])
                out[p + "norm2"][:pick] = 0.0
                out[p + "norm2.b"][:pick] = 1.0
                r[:, :pick] = (rng.permutation(E)[:, None] * 0.6 - 0.3 * E) / pick
    return out


# ------------------------------------------------------------- mechanisms
def tanh_norm(x, w, name):
    """tanh(slope x) * gain + shift, coordinate by coordinate."""
    return np.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def bias_bucket(n, rows, reach):
    """The row of the bias table for distance n: its own below rows / 2, then even in the logarithm up to ``reach``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(reach / half) * (rows - half))))


def visible(i, j, size, keep):
    """Does position i see position j?  ``size`` None: every j <= i."""
    return j <= i and (size is None or i - j < size or j < keep)


def attention_core(q, k, v, scale, sink, size=None, keep=0, rel=None, reach=None, cap=None):
    """q: [n, H, d]; k: [n, G, d]; v: [n, G, dv].  Returns [n, H, dv]."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.empty((n, H, v.shape[2]))
    buckets = None if rel is None else np.array([bias_bucket(t, rel.shape[0], reach) for t in range(n)])
    for i in range(n):
        js = np.array([j for j in range(i + 1) if visible(i, j, size, keep)])
        for h in range(H):
            g = h // (H // G)
            s = k[js, g] @ q[i, h] * scale
            if cap is not None:
                s = cap * np.tanh(s / cap)
            if rel is not None:
                s = s + rel[buckets[i - js], h]
            top = max(s.max(), sink[h])
            e = np.exp(s - top)
            out[i, h] = (e / (e.sum() + math.exp(sink[h] - top))) @ v[js, g]
    return out


def biased_attention(h, w, p, m, eps):
    n = h.shape[0]
    H, G = m["heads"], kv_heads(m)
    q, k, v = product(h, w[p + "q"]).reshape(n, H, -1), product(h, w[p + "k"]).reshape(n, G, -1), product(h, w[p + "v"]).reshape(n, G, -1)
    mask = m.get("mask") or {}
    o = attention_core(q, k, v, m["scale"], w[p + "sink"], mask.get("size"), mask.get("keep_first") or 0, w[p + "rel"], m["bias_max"])
    o = o.reshape(n, H * m["vdim"]) * sigmoid(product(h, w[p + "g"]))
    return product(o, w[p + "o"])


def stretched_frequencies(dims, base, factor, original, fast, slow):
    """Frequencies base^(-2i / dims), divided by ``factor`` where the ramp between the borders is 1."""
    border = lambda turns: dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(border(fast)), 0), min(math.ceil(border(slow)), dims - 1)
    i = np.arange(dims // 2)
    f = base ** (-2.0 * i / dims)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1 - ramp)


def turn_pairs(x, positions, freq, factor):
    """Pairs (2i, 2i + 1) of the last axis turned by position * freq[i], cosine and sine times ``factor``.  x: [n, ..., 2 len(freq)]."""
    ang = (positions[:, None] * freq).reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (len(freq),))
    c, s = factor * np.cos(ang), factor * np.sin(ang)
    out = np.empty_like(x)
    u, v = x[..., 0::2], x[..., 1::2]
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def latent_attention(h, w, p, m, eps):
    n, H, d, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    cq = perturbed(rms(product(h, w[p + "dq"]), eps) * w[p + "dq.norm"])
    q = product(cq, w[p + "uq"]).reshape(n, H, d + R)
    down = product(h, w[p + "dkv"])
    c = perturbed(rms(down[:, :m["kv_rank"]], eps) * w[p + "dkv.norm"])
    kr = down[:, m["kv_rank"]:]
    if R:
        rot, s = m["rot"], m["rot"].get("scaling")
        pos = np.arange(n, dtype=np.float64)
        if s:
            freq, mult = stretched_frequencies(R, rot["base"], s["factor"], s["original"], s["fast"], s["slow"]), 0.1 * math.log(s["factor"]) + 1
        else:
            freq, mult = rot["base"] ** (-2.0 * np.arange(R // 2) / R), 1.0
        q = np.concatenate([q[..., :d], turn_pairs(q[..., d:], pos, freq, mult)], axis=-1)
        kr = turn_pairs(kr, pos, freq, mult)
    k = np.concatenate([product(c, w[p + "uk"]).reshape(n, H, d), np.repeat(kr[:, None], H, axis=1)], axis=-1)
    v = product(c, w[p + "uv"]).reshape(n, H, m["vdim"])
    o = attention_core(perturbed(q), perturbed(k), v, m["scale"], w[p + "sink"])
    return product(o.reshape(n, -1), w[p + "o"])


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((positions + 1) / every) + 1)


def capped_attention(h, w, p, m, eps):
    """The left one of two mixers side by side."""
    n, H, G = h.shape[0], m["heads"], kv_heads(m)
    q, k, v = product(h, w[p + "q"]).reshape(n, H, -1), product(h, w[p + "k"]).reshape(n, G, -1), product(h, w[p + "v"]).reshape(n, G, -1)
    if m.get("q_temp"):
        q = perturbed(q * query_temperature(np.arange(n), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None])
    o = attention_core(q, k, v, m["scale"], w[p + "sink"], cap=m.get("softcap"))
    return product(o.reshape(n, -1), w[p + "o"])


def decaying_outer_products(x, dt, A, B, C, D, S=None):
    """x: [n, H, P]; dt: [n, H] (positive); A: [H] (negative); B, C: [n, G, N]; D: [H].  S: [H, N, P].  Returns (y [n, H, P], S)."""
    n, H, P = x.shape
    G = B.shape[1]
    S = np.zeros((H, B.shape[2], P)) if S is None else S.copy()
    y = np.empty_like(x)
    for t in range(n):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(A[h] * dt[t, h]) * S[h] + np.outer(B[t, g], dt[t, h] * x[t, h])
            y[t, h] = C[t, g] @ S[h] + D[h] * x[t, h]
    return y, S


def state_space_dual(h, w, p, m, eps):
    """The right one of two mixers side by side."""
    n, H, P, G, N = h.shape[0], m["heads"], m["vdim"], m["groups"], m["state"]
    I = H * P
    u = product(h, w[p + "in"])
    z, xbc, dt = u[:, :I], u[:, I:-H], u[:, -H:]
    xbc = perturbed(silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"])))
    x, B, C = xbc[:, :I].reshape(n, H, P), xbc[:, I:I + G * N].reshape(n, G, N), xbc[:, I + G * N:].reshape(n, G, N)
    y, _ = decaying_outer_products(x, softplus(dt + w[p + "dt_bias"]), -np.exp(w[p + "A_log"]), B, C, w[p + "D"])
    y = y.reshape(n, I) * silu(z)
    parts = m["norm_groups"]
    y = rms(y.reshape(n, parts, I // parts), eps).reshape(n, I) * w[p + "norm"]
    return product(y, w[p + "o"])


def parallel(h, w, p, m, eps):
    return m["left_scale"] * capped_attention(h, w, p + "left.", m["left"], eps) + m["right_scale"] * state_space_dual(h, w, p + "right.", m["right"], eps)


def gelu(z):
    return 0.5 * z * (1.0 + erf(z / math.sqrt(2.0)))


def dense_ff(h, w, p):
    return product(np.maximum(product(h, w[p + "up"]), 0.0) ** 2, w[p + "down"])


def expert_ff(h, w, p):
    return product(gelu(product(h, w[p + "up"])), w[p + "down"])


def route(h, w_router, top):
    """(ids [n, top], scores [n, top]): the outputs with the largest sigmoid scores."""
    s = sigmoid(h @ w_router.T)
    ids = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=-1)


def routed_ff(h, w, p, mlp):
    ids, scores = route(h, w[p + "router"], mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(ids[t], scores[t]):
            out[t] += expert_ff(s * h[t:t + 1], w, f"{p}e{int(e)}.")[0]
    return out + expert_ff(h, w, p + "shared.") if mlp.get("shared") else out


def feed_forward(h, w, p, mlp):
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else routed_ff(h, w, p, mlp)


MIXERS = {"attention": biased_attention, "latent_attention": latent_attention, "parallel": parallel}


def forward(cfg, w, ids, return_layers=False):
    """Logits [n, vocab] of one request's tokens, all at once."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(ids)].copy()
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](tanh_norm(x, w, p + "norm1"), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + feed_forward(tanh_norm(x, w, p + "norm2"), w, p + "mlp.", layer["mlp"])
        after.append(x.copy())
    logits = product(tanh_norm(x, w, "final.norm"), w["embed"])
    return (logits, np.stack(after)) if return_layers else logits


def routing_margin(cfg, w, ids):
    """The smallest gap between a chosen score and the best one left out, over all tokens and layers."""
    gaps = [np.inf]
    x = w["embed"][np.asarray(ids)].copy()
    for i, layer in enumerate(cfg["layers"]):
        p, eps = f"l{i}.", cfg["norm"]["eps"]
        x = x + MIXERS[layer["type"]](tanh_norm(x, w, p + "norm1"), w, p + "mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        h = tanh_norm(x, w, p + "norm2")
        if mlp["kind"] == "moe" and mlp["router"]["top"] < mlp["router"]["experts"]:
            s = -np.sort(-sigmoid(h @ w[p + "mlp.router"].T), axis=-1)
            gaps.append((s[:, mlp["router"]["top"] - 1] - s[:, mlp["router"]["top"]]).min())
        x = x + feed_forward(h, w, p + "mlp.", mlp)
    return min(gaps)


def rounding_error(cfg, w, ids, runs=4):
    """Per row of the logits, the largest error over all tokens that perturbations of bfloat16's size caused in ``runs`` tries."""
    want = forward(cfg, w, ids)
    worst = np.zeros(len(want))
    for seed in range(runs):
        with rounded_like_bf16(seed):
            worst = np.maximum(worst, np.abs(forward(cfg, w, ids) - want).max(axis=1))
    return worst


def greedy(logits):
    return int(np.argmax(logits))
