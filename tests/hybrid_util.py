"""Small layer-list models for the tests: configurations with sizes that are all different from one another, seeded
weights rounded to bf16, and snapshot folders."""
import copy
import json
import os

import numpy as np

from singe_b200.checkpoint import save_safetensors


def latent(heads, dim, vdim, q_rank, kv_rank, window, scale, ff=None, weights_of=None):
    return _entry("latent_attention", {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                       "scale": scale, "mask": {"size": window}}, ff, weights_of)


def gla(heads, dim, vdim, tau, ff=None, weights_of=None):
    return _entry("gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, ff, weights_of)


def _entry(kind, mixer, ff, weights_of):
    entry = {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        entry["weights_of"] = weights_of
    return entry


def model(width, vocab, eps, *layers):
    return {"architecture": "Kavalorn", "layers": list(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width}


# tiled bf16 kernels, a borrowed layer of each kind, two windows, a recurrent layer first
MIXED = model(96, 131, 1e-5,
              gla(3, 24, 40, 4.0, ff=72),
              latent(5, 16, 24, 40, 56, 21, 0.3, ff=None),
              latent(3, 40, 32, 24, 72, 70, 0.11, ff=144),
              gla(3, 24, 40, 4.0, ff=72, weights_of=0),
              latent(5, 16, 24, 40, 56, 21, 0.3, weights_of=1))
# sizes no tiled kernel takes and that are no multiples of eight
ODD = model(100, 89, 1e-3,
            latent(3, 13, 21, 19, 27, 9, 0.5, ff=50),
            gla(2, 10, 13, 2.5, ff=33),
            latent(2, 136, 20, 24, 530, 33, 0.08))
# heads, windows and constants that are one
ONES = model(64, 64, 1e-6,
             latent(1, 8, 8, 8, 8, 1, 1.0, ff=8),
             gla(1, 8, 8, 1.0),
             latent(1, 64, 64, 64, 64, 2, 1.0, ff=64))
# more heads than one CTA of the decode kernel takes, the widest latent, a wide recurrence
WIDE = model(256, 300, 1e-6,
             latent(34, 128, 96, 128, 512, 300, 0.088, ff=512),
             gla(2, 128, 256, 10.0),
             latent(18, 64, 64, 96, 320, 150, 0.125),
             gla(4, 40, 72, 8.0, ff=128))


def bf16(values):
    bits = np.ascontiguousarray(values, dtype=np.float32).view(np.uint32).astype(np.uint64)
    rounded = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16
    return rounded.astype(np.uint32).view(np.float32)


def shapes(config, rank=12):
    w, names = config["width"], {}
    names.update({"embed": (config["vocab"], w), "embed.norm": (w,), "final.norm": (w,), "head": (config["vocab"], w)})
    for index, layer in enumerate(config["layers"]):
        if layer.get("weights_of") is not None:
            continue
        prefix, m = f"l{index}.", layer["mixer"]
        names[prefix + "norm1"] = (w,)
        keys, values = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        if layer["type"] == "gla":
            mix = {"q": (keys, w), "k": (keys, w), "v": (values, w), "g": (values, w), "o": (w, values),
                   "norm": (m["vdim"],), "a1": (rank + index, w), "a2": (keys, rank + index), "a2.b": (keys,)}
        else:
            mix = {"dq": (m["q_rank"], w), "dq.norm": (m["q_rank"],), "uq": (keys, m["q_rank"]), "dkv": (m["kv_rank"], w),
                   "dkv.norm": (m["kv_rank"],), "uk": (keys, m["kv_rank"]), "uv": (values, m["kv_rank"]),
                   "g": (m["heads"], w), "o": (w, values)}
        names.update({f"{prefix}mix.{name}": shape for name, shape in mix.items()})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            names.update({prefix + "norm2": (w,), prefix + "mlp.up": (ff, w), prefix + "mlp.down": (w, ff)})
    return names


def make_weights(config, seed=0):
    """bf16-representable float32 arrays by tensor name; scores sharp enough that single keys matter."""
    rng = np.random.default_rng(seed)
    weights = {}
    for name, shape in shapes(config).items():
        values = rng.standard_normal(shape)
        if name.endswith("a2.b"):
            values = 1.5 + 2.0 * values
        elif len(shape) == 1:
            values = 1.0 + 0.2 * values
        elif name != "embed":
            values *= {"uq": 2.0, "uk": 2.0, "a2": 2.0}.get(name.rsplit(".", 1)[-1], 1.0) / np.sqrt(shape[1])
        weights[name] = bf16(values)
    return weights


def write_snapshot(directory, config, weights):
    directory = str(directory)
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as handle:
        json.dump(config, handle)
    save_safetensors(os.path.join(directory, "model.safetensors"),
                     {name: (array.view(np.uint32) >> 16).astype(np.uint16) for name, array in weights.items()})
    return directory


def variant(config, **changes):
    changed = copy.deepcopy(config)
    changed.update(changes)
    return changed
