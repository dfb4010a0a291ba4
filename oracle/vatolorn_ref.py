"""Plain restatement of the Vatolorn decoder on the CPU -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, float64 throughout, whole sequences at once, no cache: every position is computed from the
sequence's first token on.  ``config`` is the parsed ``config.json`` dictionary, ``weights`` maps tensor names to arrays.
"""
from __future__ import annotations

import numpy as np

from oracle.hybrid_ref import rms_norm, sigmoid

UNIT_EPS = 1e-6   # under the root of a unit vector's squared length


def silu(z: np.ndarray) -> np.ndarray:
    return z * sigmoid(z)


def softplus(z: np.ndarray) -> np.ndarray:
    return np.logaddexp(0.0, z)


def unit(x: np.ndarray) -> np.ndarray:
    return x / np.sqrt((x ** 2).sum(axis=-1, keepdims=True) + UNIT_EPS)


def causal_convolution(u: np.ndarray, taps: np.ndarray) -> np.ndarray:
    """u [T, C], taps [C, n]: the last tap weighs the token itself, the one before it the token before, and so on."""
    out = np.zeros(u.shape)
    count = taps.shape[1]
    for j in range(count):
        back = count - 1 - j
        if back < len(u):
            out[back:] += taps[:, j] * u[: len(u) - back]
    return out


def yarn_frequencies(dims: int, base: float, scaling: dict | None):
    """Angular frequency of each pair of dimensions and the factor on cosines and sines."""
    index = np.arange(dims // 2, dtype=np.float64)
    plain = float(base) ** (-2.0 * index / dims)
    if scaling is None:
        return plain, 1.0
    pair_of = lambda turns: dims * np.log(scaling["original"] / (2.0 * np.pi * turns)) / (2.0 * np.log(base))
    low, high = max(np.floor(pair_of(scaling["fast"])), 0.0), min(np.ceil(pair_of(scaling["slow"])), dims - 1.0)
    ramp = np.clip((index - low) / max(high - low, 0.001), 0.0, 1.0)
    return plain / scaling["factor"] * ramp + plain * (1.0 - ramp), 0.1 * np.log(scaling["factor"]) + 1.0


def rotate_adjacent(x: np.ndarray, positions: np.ndarray, rot: dict) -> np.ndarray:
    """x [T, H, D]: dimensions 2i and 2i + 1 turn together, the first ``dims`` of every head."""
    frequency, factor = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    angle = positions[:, None, None] * frequency
    cosine, sine = np.cos(angle) * factor, np.sin(angle) * factor
    out = np.array(x, dtype=np.float64)
    even, odd = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = even * cosine - odd * sine
    out[..., 1:rot["dims"]:2] = odd * cosine + even * sine
    return out


def chunked_attention(query: np.ndarray, key: np.ndarray, value: np.ndarray, scale: float, size: int) -> np.ndarray:
    """query [T, H, D], key [T, G, D], value [T, G, V]: position i sees the keys of its own chunk of ``size`` up to itself."""
    tokens, heads, groups = query.shape[0], query.shape[1], key.shape[1]
    shared = np.arange(heads) // (heads // groups)
    key, value = key[:, shared], value[:, shared]
    out = np.zeros((tokens, heads, value.shape[2]))
    for first in range(0, tokens, size):
        part = slice(first, min(first + size, tokens))
        score = np.einsum("ihd,jhd->hij", query[part], key[part]) * scale
        count = score.shape[1]
        score = np.where(np.tril(np.ones((count, count), dtype=bool)), score, -np.inf)
        score -= score.max(axis=2, keepdims=True)
        weight = np.exp(score)
        weight /= weight.sum(axis=2, keepdims=True)
        out[part] = np.einsum("hij,jhv->ihv", weight, value[part])
    return out


def attention_inputs(h: np.ndarray, w: dict, mixer: dict, eps: float):
    """Queries, keys and values of the attention: projection with bias, convolution, norm over the whole projection,
    rotation."""
    tokens, positions = h.shape[0], np.arange(h.shape[0], dtype=np.float64)
    project = lambda name: causal_convolution(h @ w[name].T + w[name + ".b"], w[name + ".conv"])
    query = rms_norm(project("q"), w["q.norm"], eps).reshape(tokens, mixer["heads"], mixer["dim"])
    key = rms_norm(project("k"), w["k.norm"], eps).reshape(tokens, mixer["kv_heads"], mixer["dim"])
    value = project("v").reshape(tokens, mixer["kv_heads"], mixer["vdim"])
    return rotate_adjacent(query, positions, mixer["rot"]), rotate_adjacent(key, positions, mixer["rot"]), value


def attention(h: np.ndarray, w: dict, mixer: dict, eps: float) -> np.ndarray:
    query, key, value = attention_inputs(h, w, mixer, eps)
    attended = chunked_attention(query, key, value, mixer["scale"], mixer["mask"]["size"])
    return attended.reshape(h.shape[0], -1) @ w["o"].T


def delta_recurrence(query: np.ndarray, key: np.ndarray, value: np.ndarray, decay: np.ndarray, beta: np.ndarray,
                     state: np.ndarray):
    """query, key, decay [T, H, K], value [T, H, V], beta [T, H], state [H, K, V]; outputs [T, H, V] and the last state."""
    out = np.zeros(value.shape)
    for t in range(query.shape[0]):
        state = decay[t][:, :, None] * state
        written = beta[t][:, None] * (value[t] - np.einsum("hkv,hk->hv", state, key[t]))
        state = state + key[t][:, :, None] * written[:, None, :]
        out[t] = np.einsum("hkv,hk->hv", state, query[t])
    return out, state


def delta_inputs(h: np.ndarray, w: dict, mixer: dict):
    """What the recurrence reads: unit queries (scaled) and keys, values, decays, write strengths."""
    tokens, heads, groups, dim = h.shape[0], mixer["heads"], mixer["kv_heads"], mixer["dim"]
    project = lambda name: silu(causal_convolution(h @ w[name].T, w[name + ".conv"]))
    shared = np.arange(heads) // (heads // groups)
    query = unit(project("q").reshape(tokens, groups, dim))[:, shared] * dim ** -0.5
    key = unit(project("k").reshape(tokens, groups, dim))[:, shared]
    value = project("v").reshape(tokens, heads, mixer["vdim"])
    step = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).reshape(tokens, heads, dim)
    decay = np.exp(-np.exp(w["A_log"])[:, None] * step)
    return query, key, value, decay, sigmoid(h @ w["b"].T)


def gated_delta(h: np.ndarray, w: dict, mixer: dict, eps: float) -> np.ndarray:
    heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
    out, _ = delta_recurrence(*delta_inputs(h, w, mixer), np.zeros((heads, dim, vdim)))
    out = rms_norm(out, w["norm"], eps).reshape(h.shape[0], -1)
    return (out * sigmoid((h @ w["g1"].T) @ w["g2"].T)) @ w["o"].T


def part(w: dict, name: str) -> dict:
    return {key[len(name) + 1:]: value for key, value in w.items() if key.startswith(name + ".")}


def side_by_side(h: np.ndarray, w: dict, mixer: dict, eps: float) -> np.ndarray:
    left = attention(h, part(w, "left"), mixer["left"], eps)
    right = gated_delta(h, part(w, "right"), mixer["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def gated_mlp(h: np.ndarray, w: dict) -> np.ndarray:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def stream_step(streams: np.ndarray, sublayer, w: dict) -> np.ndarray:
    """streams [S, T, W]: the sublayer reads one blend of them; its output and a blend of the old ones make the new ones."""
    read = np.einsum("s,stw->tw", w["in"], streams)
    return np.einsum("sn,stw->ntw", w["mix"], streams) + w["out"][:, None, None] * sublayer(read)


def forward(config: dict, weights: dict, tokens):
    """Logits [T, vocab] of one sequence and the sum of the streams after every layer [layers, T, width]."""
    eps = config["norm"]["eps"]
    wide = {name: np.asarray(value, dtype=np.float64) for name, value in weights.items()}
    streams = np.stack([wide["embed"][np.asarray(tokens)]] * config["streams"])
    trail = []
    for index, layer in enumerate(config["layers"]):
        w = part(wide, f"l{index}")
        mix = lambda u: side_by_side(rms_norm(u, w["norm1"], eps), part(w, "mix"), layer["mixer"], eps)
        streams = stream_step(streams, mix, part(w, "hc1"))
        if layer.get("mlp") is not None:
            streams = stream_step(streams, lambda u: gated_mlp(rms_norm(u, w["norm2"], eps), part(w, "mlp")), part(w, "hc2"))
        trail.append(streams.sum(axis=0))
    return rms_norm(trail[-1], wide["final.norm"], eps) @ wide["head"].T * config["logit_scale"], np.stack(trail)
