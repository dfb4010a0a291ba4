"""Plain restatement of the layer-list decoder (Kavalorn) on the CPU -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, float64 throughout, whole sequences at once, no cache: every position is computed from the
sequence's first token on.  ``config`` is the parsed ``config.json`` dictionary, ``weights`` maps tensor names to arrays.
"""
from __future__ import annotations

import numpy as np


def layer_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    centred = x - x.mean(axis=-1, keepdims=True)
    return centred / np.sqrt((centred ** 2).mean(axis=-1, keepdims=True) + eps) * weight


def rms_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps) * weight


def sigmoid(z: np.ndarray) -> np.ndarray:
    return np.exp(-np.logaddexp(0.0, -z))


def squared_relu_mlp(h: np.ndarray, up: np.ndarray, down: np.ndarray) -> np.ndarray:
    return (np.maximum(h @ up.T, 0.0) ** 2) @ down.T


def windowed_attention(query: np.ndarray, key: np.ndarray, value: np.ndarray, scale: float, window: int) -> np.ndarray:
    """query [T, H, D], key [T, H, D], value [T, H, V]; position i sees i - window + 1 .. i."""
    tokens = query.shape[0]
    out = np.zeros((tokens, query.shape[1], value.shape[2]))
    for i in range(tokens):
        first = max(0, i - window + 1)
        score = np.einsum("hd,jhd->hj", query[i], key[first:i + 1]) * scale
        score -= score.max(axis=1, keepdims=True)
        weight = np.exp(score)
        weight /= weight.sum(axis=1, keepdims=True)
        out[i] = np.einsum("hj,jhv->hv", weight, value[first:i + 1])
    return out


def latent_attention(h: np.ndarray, w: dict, mixer: dict, eps: float) -> np.ndarray:
    tokens, heads = h.shape[0], mixer["heads"]
    latent_query = rms_norm(h @ w["dq"].T, w["dq.norm"], eps)
    latent = rms_norm(h @ w["dkv"].T, w["dkv.norm"], eps)
    query = (latent_query @ w["uq"].T).reshape(tokens, heads, mixer["dim"])
    key = (latent @ w["uk"].T).reshape(tokens, heads, mixer["dim"])
    value = (latent @ w["uv"].T).reshape(tokens, heads, mixer["vdim"])
    attended = windowed_attention(query, key, value, mixer["scale"], mixer["mask"]["size"])
    attended = attended * sigmoid(h @ w["g"].T)[:, :, None]
    return attended.reshape(tokens, -1) @ w["o"].T


def gated_recurrence(query: np.ndarray, key: np.ndarray, value: np.ndarray, decay: np.ndarray, state: np.ndarray):
    """query, key, decay [T, H, K], value [T, H, V], state [H, K, V]; returns outputs [T, H, V] and the last state."""
    out = np.zeros(value.shape)
    for t in range(query.shape[0]):
        state = decay[t][:, :, None] * state + key[t][:, :, None] * value[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", state, query[t])
    return out, state


def gated_linear_attention(h: np.ndarray, w: dict, mixer: dict, eps: float) -> np.ndarray:
    tokens, heads, dim, vdim = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    query = (h @ w["q"].T).reshape(tokens, heads, dim) / np.sqrt(dim)
    key = (h @ w["k"].T).reshape(tokens, heads, dim)
    value = (h @ w["v"].T).reshape(tokens, heads, vdim)
    z = ((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]).reshape(tokens, heads, dim)
    decay = sigmoid(z) ** (1.0 / mixer["tau"])
    out, _ = gated_recurrence(query, key, value, decay, np.zeros((heads, dim, vdim)))
    out = rms_norm(out, w["norm"], eps).reshape(tokens, -1)
    gate = h @ w["g"].T
    return (out * (gate * sigmoid(gate))) @ w["o"].T


MIXERS = {"latent_attention": latent_attention, "gla": gated_linear_attention}


def owner(config: dict, index: int) -> int:
    """The layer whose tensors layer ``index`` uses."""
    while config["layers"][index].get("weights_of") is not None:
        index = config["layers"][index]["weights_of"]
    return index


def forward(config: dict, weights: dict, tokens):
    """Logits [T, vocab] of one sequence and the residual stream after every layer [layers, T, width]."""
    eps = config["norm"]["eps"]
    wide = {name: np.asarray(value, dtype=np.float64) for name, value in weights.items()}
    x = layer_norm(wide["embed"][np.asarray(tokens)], wide["embed.norm"], eps)
    trail = []
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{owner(config, index)}."
        mix = {name[len(prefix) + 4:]: value for name, value in wide.items() if name.startswith(prefix + "mix.")}
        x = x + MIXERS[layer["type"]](layer_norm(x, wide[prefix + "norm1"], eps), mix, layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + squared_relu_mlp(layer_norm(x, wide[prefix + "norm2"], eps), wide[prefix + "mlp.up"],
                                     wide[prefix + "mlp.down"])
        trail.append(x)
    return layer_norm(x, wide["final.norm"], eps) @ wide["head"].T, np.stack(trail)
