"""Small Kezunex configurations and seeded weights for the tests.

The shapes differ in what a configuration can set: every order of the three mixers, with and without feed-forward; loops
that begin at the first layer, later, and none; one and several groups, norm parts, key heads and blocks; head sizes that fit
no 16-byte group, that fill a tile of the chunked recurrence and that need several; one to six taps; values wider and
narrower than keys; with and without query temperature; scales of exactly 1, below zero and zero.
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch


def left(heads, kv_heads, dim, vdim, scale, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def right(heads, vdim, state, groups=1, conv=4, parts=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": parts}


def parallel(a, b, left_scale=1.0, right_scale=1.0):
    return "parallel", {"left": a, "left_scale": left_scale, "right": b, "right_scale": right_scale}


def rglru(width, blocks, conv=4):
    return "rglru", {"width": width, "blocks": blocks, "conv": conv}


def mlstm(heads, dim, vdim, cap=10.0):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def layer(mix, ff=None):
    return {"type": mix[0], "mixer": mix[1], "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, layers, eps=1e-5, scale=1.0, loop=None):
    cfg = {"architecture": "Kezunex", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# sizes that fit no 16-byte group, a loop that begins behind the first layer, a temperature that changes every few tokens
KA = model(157, 72, [
    layer(rglru(60, 3, conv=5), 52),
    layer(parallel(left(4, 2, 20, 12, 0.3, (0.4, 7)), right(4, 10, 6, groups=2, conv=3, parts=2), 0.7, 1.3)),
    layer(mlstm(3, 10, 7, cap=5.0), 100),
    layer(parallel(left(3, 3, 12, 28, 0.25, (0.2, 48)), right(6, 7, 34, groups=3, conv=2, parts=6), -0.8, 0.9), 40),
    layer(mlstm(2, 34, 22)),
], scale=1.5, loop=(1, 3, 2))

# sizes of the tensor-core kernels, several 64-wide tiles of the recurrence in either direction, a loop from the first layer on
KB = model(263, 128, [
    layer(parallel(left(4, 1, 64, 64, 0.2, (0.3, 40)), right(4, 64, 128, groups=2, parts=4), 1.0, 0.6), 192),
    layer(rglru(128, 2), 96),
    layer(mlstm(2, 72, 136, cap=15.0), 64),
    layer(parallel(left(2, 2, 32, 128, 0.3), right(2, 80, 64, parts=2), 0.5, 1.0)),
    layer(rglru(192, 4, conv=3)),
], eps=1e-6, scale=2.0, loop=(0, 2, 4))

# one head, one block, one tap, no loop, scales of 1, a left side that does not count
KC = model(97, 52, [
    layer(mlstm(1, 9, 25, cap=30.0), 30),
    layer(rglru(33, 1, conv=1)),
    layer(parallel(left(1, 1, 10, 25, 0.4), right(1, 13, 5, conv=1)), 50),
    layer(rglru(40, 5, conv=6), 20),
    layer(parallel(left(2, 1, 16, 16, 0.3, (0.5, 3)), right(3, 8, 16, conv=4, parts=3), 0.0, 0.8)),
], eps=3e-6)

CASES = {"ka": (KA, 81), "kb": (KB, 82), "kc": (KC, 83)}


def tensor_shapes(cfg: dict) -> dict:
    w, v = cfg["width"], cfg["vocab"]
    shapes = {"embed": (v, w), "final.norm": (w,)}
    if cfg.get("loop"):
        shapes["loop.step"] = (cfg["loop"]["times"], w)
    for i, spec in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", spec["mixer"], spec["type"]
        shapes.update({p + "norm1": (w,), p + "norm1b": (w,), p + "ls1": (w,)})
        if kind == "parallel":
            a, b = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            at = p + "mix.left."
            shapes.update({at + "q": (H * d, w), at + "k": (G * d, w), at + "v": (G * dv, w), at + "o": (w, H * dv), at + "q.norm": (d,), at + "k.norm": (d,)})
            H, dv, at = b["heads"], b["vdim"], p + "mix.right."
            inner, gn = H * dv, b["groups"] * b["state"]
            shapes.update({at + "in": (2 * inner + 2 * gn + H, w), at + "conv": (inner + 2 * gn, b["conv"]), at + "conv.b": (inner + 2 * gn,),
                           at + "dt_bias": (H,), at + "A_log": (H,), at + "D": (H,), at + "norm": (inner,), at + "o": (w, inner)})
        elif kind == "rglru":
            n, k, at = m["width"], m["blocks"], p + "mix."
            b = n // k
            shapes.update({at + "y": (n, w), at + "y.b": (n,), at + "x": (n, w), at + "x.b": (n,), at + "conv": (n, m["conv"]), at + "conv.b": (n,),
                           at + "ra": (k, b, b), at + "ra.b": (k, b), at + "ri": (k, b, b), at + "ri.b": (k, b), at + "lam": (n,), at + "o": (w, n)})
        else:
            H, d, dv, at = m["heads"], m["dim"], m["vdim"], p + "mix."
            shapes.update({at + "q": (H * d, w), at + "k": (H * d, w), at + "v": (H * dv, w), at + "g": (H * dv, w), at + "i": (H, w), at + "i.b": (H,),
                           at + "f": (H, w), at + "f.b": (H,), at + "norm": (H * dv,), at + "o": (w, H * dv)})
        if spec.get("mlp"):
            ff = spec["mlp"]["ff"]
            shapes.update({p + "norm2": (w,), p + "norm2b": (w,), p + "ls2": (w,), p + "mlp.gate": (ff, w), p + "mlp.up": (ff, w), p + "mlp.down": (w, ff)})
    return shapes


def make_weights(cfg: dict, seed: int, gain: float = 1.0) -> dict:
    """Seeded weights, every value representable in bfloat16 (so a bfloat16 engine and a float oracle start alike).  Norm
    weights, biases, scales and the recurrences' constants are spread widely, so that leaving one out or swapping two moves
    the logits; decays run from a few tokens to hundreds.  `gain` scales the attention's query norm (a larger one makes the softmax peaked)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = ".".join(name.split(".")[-2:]) if name.endswith((".b", ".norm")) else name.rsplit(".", 1)[-1]
        normal = rng.standard_normal(shape)
        if name == "embed":
            value = normal
        elif name == "loop.step":
            value = 0.5 * normal
        elif leaf == "q.norm":
            value = gain * (1.0 + 0.4 * normal)
        elif leaf.endswith("norm") or leaf in ("norm1", "norm2", "norm1b", "norm2b"):
            value = 1.0 + 0.3 * normal
        elif leaf in ("ls1", "ls2"):
            value = 0.5 + 0.25 * normal
        elif leaf == "conv":
            value = normal / np.sqrt(shape[1])
        elif leaf in ("conv.b", "y.b", "x.b", "i.b", "ra.b", "ri.b"):
            value = 0.5 * normal
        elif leaf == "dt_bias":
            value = -2.0 + 1.5 * normal
        elif leaf == "A_log":
            value = 0.3 + 0.9 * normal
        elif leaf == "D":
            value = normal
        elif leaf == "f.b":
            value = 2.0 + 2.0 * normal
        elif leaf == "lam":
            value = -4.0 + 2.0 * normal
        elif leaf in ("i", "f"):
            value = 1.5 / np.sqrt(shape[-1]) * normal
        else:
            value = normal / np.sqrt(shape[-1])
        out[name] = torch.tensor(np.asarray(value), dtype=torch.float32).to(torch.bfloat16).to(torch.float64)
    return out


def write_model_dir(directory, cfg: dict, weights: dict) -> Path:
    from safetensors.torch import save_file
    directory = Path(directory)
    directory.mkdir(parents=True, exist_ok=True)
    (directory / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights.items()}, str(directory / "model.safetensors"))
    return directory


def random_tokens(cfg: dict, n: int, seed: int) -> list:
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def one_layer(mix, ff=None, width=64, vocab=101, scale=1.0):
    return model(vocab, width, [layer(mix, ff)], scale=scale)
