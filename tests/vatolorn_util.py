"""Small Vatolorn models for the tests: configurations with sizes that are all different from one another, and seeded weights
rounded to bf16."""
import numpy as np

from tests.hybrid_util import bf16, write_snapshot  # noqa: F401  (the tests write snapshots through here)


def rot(dims, base, scaling=None):
    fields = {"dims": dims, "base": base}
    if scaling is not None:
        fields["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return fields


def left(heads, kv_heads, dim, vdim, chunk, taps, rotation, scale):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "conv": taps, "rot": rotation,
            "scale": scale}


def right(heads, kv_heads, dim, vdim, taps):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}


def layer(one, other, ff=None):
    return {"type": "parallel", "mixer": {"left": one, "right": other}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(width, vocab, streams, logit_scale, eps, *layers):
    return {"architecture": "Vatolorn", "layers": list(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "streams": streams, "logit_scale": logit_scale}


# sizes the tiled kernels take; two chunk sizes, one smaller than a page and a half; a layer without a feed-forward
MIXED = model(96, 131, 3, 0.7, 1e-5,
              layer(left(6, 2, 40, 24, 21, 3, rot(16, 500.0, (4.0, 64, 8.0, 1.0)), 0.5), right(4, 2, 24, 40, 2), 72),
              layer(left(4, 4, 16, 56, 70, 2, rot(16, 10000.0, (16.0, 128, 16.0, 2.0)), 0.7), right(3, 3, 32, 16, 5)),
              layer(left(5, 1, 72, 128, 21, 4, rot(64, 2000.0, (2.0, 256, 32.0, 1.0)), 0.3), right(2, 1, 64, 48, 3), 144))
# sizes no tiled kernel takes and that are no multiples of eight
ODD = model(100, 89, 2, 1.9, 1e-3,
            layer(left(3, 1, 13, 21, 9, 4, rot(6, 100.0, (3.0, 40, 4.0, 0.5)), 0.6), right(2, 1, 10, 13, 3), 50),
            layer(left(2, 2, 138, 20, 33, 2, rot(130, 700.0, (8.0, 512, 32.0, 1.0)), 0.1), right(3, 1, 7, 9, 6), 33),
            layer(left(10, 1, 8, 24, 16, 3, rot(8, 300.0, (1.5, 99, 9.0, 3.0)), 0.8), right(1, 1, 12, 300, 2)))
# heads, chunks, taps, streams and constants that are one
ONES = model(64, 64, 1, 1.0, 1e-6,
             layer(left(1, 1, 8, 8, 1, 1, rot(2, 10.0, (1.0, 16, 1.0, 1.0)), 1.0), right(1, 1, 8, 8, 1), 8),
             layer(left(2, 1, 64, 64, 2, 1, rot(64, 10.0, (1.0, 1, 1.0, 1.0)), 1.0), right(2, 1, 16, 16, 1)))
# long chunks, wide states, many streams
WIDE = model(256, 300, 5, 0.3, 1e-6,
             layer(left(16, 2, 128, 96, 300, 4, rot(96, 20000.0, (8.0, 128, 32.0, 1.0)), 0.25), right(4, 2, 128, 128, 4), 512),
             layer(left(8, 4, 64, 64, 128, 3, rot(64, 10000.0, (2.0, 2048, 32.0, 1.0)), 0.4), right(2, 1, 256, 80, 3), 320))


def shapes(config, rank=12):
    w, streams = config["width"], config["streams"]
    names = {"embed": (config["vocab"], w), "final.norm": (w,), "head": (config["vocab"], w)}
    for index, entry in enumerate(config["layers"]):
        l, r = entry["mixer"]["left"], entry["mixer"]["right"]
        low, gate_low = rank + index, rank + 5 - 2 * index
        mix = {"left.out": (w,), "right.out": (w,), "left.o": (w, l["heads"] * l["vdim"]), "right.o": (w, r["heads"] * r["vdim"]),
               "left.q.norm": (l["heads"] * l["dim"],), "left.k.norm": (l["kv_heads"] * l["dim"],), "right.norm": (r["vdim"],),
               "right.b": (r["heads"], w), "right.A_log": (r["heads"],), "right.dt_bias": (r["heads"] * r["dim"],),
               "right.a1": (low, w), "right.a2": (r["heads"] * r["dim"], low), "right.g1": (gate_low, w),
               "right.g2": (r["heads"] * r["vdim"], gate_low)}
        for name, rows in (("left.q", l["heads"] * l["dim"]), ("left.k", l["kv_heads"] * l["dim"]), ("left.v", l["kv_heads"] * l["vdim"])):
            mix.update({name: (rows, w), name + ".b": (rows,), name + ".conv": (rows, l["conv"])})
        for name, rows in (("right.q", r["kv_heads"] * r["dim"]), ("right.k", r["kv_heads"] * r["dim"]), ("right.v", r["heads"] * r["vdim"])):
            mix.update({name: (rows, w), name + ".conv": (rows, r["conv"])})
        prefix = f"l{index}."
        names.update({f"{prefix}mix.{name}": shape for name, shape in mix.items()})
        names[prefix + "norm1"] = (w,)
        sublayers = [1]
        if entry["mlp"] is not None:
            ff = entry["mlp"]["ff"]
            names.update({prefix + "norm2": (w,), prefix + "mlp.gate": (ff, w), prefix + "mlp.up": (ff, w), prefix + "mlp.down": (w, ff)})
            sublayers.append(2)
        for q in sublayers:
            names.update({f"{prefix}hc{q}.in": (streams,), f"{prefix}hc{q}.out": (streams,), f"{prefix}hc{q}.mix": (streams, streams)})
    return names


def make_weights(config, seed=0):
    """bf16-representable float32 arrays by tensor name.  The recurrence's queries resemble its keys: a first token whose query
    and key were all but orthogonal would have its rounding blown up by the norm behind the read-out."""
    rng = np.random.default_rng(seed)
    weights, streams = {}, config["streams"]
    for name, shape in shapes(config).items():
        values = rng.standard_normal(shape)
        kind = name.split(".", 1)[-1]
        if kind.endswith("A_log"):
            values = -1.5 + 0.7 * values
        elif kind.endswith("dt_bias") or (kind.startswith("mix.left") and kind.endswith(".b")):
            values = 0.4 * values
        elif kind.endswith(".conv"):
            values = (0.5 * values + (np.arange(shape[1]) == shape[1] - 1)) / np.sqrt(shape[1])
        elif kind.endswith(".mix"):
            values = np.eye(streams) * 0.8 + 0.3 * values / streams
        elif kind.endswith("hc1.in") or kind.endswith("hc2.in"):
            values = (1.0 + 0.4 * values) / streams
        elif len(shape) == 1:
            values = 1.0 + 0.2 * values
        elif name != "embed":
            values *= 1.0 / np.sqrt(shape[1])
        weights[name] = bf16(values)
    for index in range(len(config["layers"])):
        prefix = f"l{index}.mix.right."
        for part in ("", ".conv"):
            weights[f"{prefix}k{part}"] = bf16(0.9 * weights[f"{prefix}q{part}"] + 0.4 * weights[f"{prefix}k{part}"])
    return weights
