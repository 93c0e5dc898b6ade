"""Small Tekezen configurations and seeded weights for the tests.

The shapes differ in what a configuration can set: either mixer first; latent attention with windows of a few keys, beyond
one query tile, and none; cache rows that need padding and rows of tensor-core widths; grouped attention with values
narrower and wider than the keys, one group and as many groups as heads, part and whole rotation, with and without slowed
frequencies, windows with no kept token, one, a few, and more than a page of them, scores bent hard, softly and not at all;
layers that share values between layers that do not; layers without a feed-forward; experts with and without a shared one;
routers that take one, two and all experts; a table of token pairs with multipliers beyond its size, and none.
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window=None, base=50000.0, scaling=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": rot}
    if window is not None:
        m["mask"] = {"size": window}
    return "latent_attention", m


def attention(heads, kv_heads, dim, vdim, scale, rot_dims, window=None, keep_first=0, softcap=None, base=10000.0, factor=None, v_mix=False):
    rot = {"base": base, "dims": rot_dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot, "v_mix": v_mix}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep_first}
    if softcap is not None:
        m["softcap"] = softcap
    return "attention", m


def dense(ff, limit=1.8):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top, limit=1.2, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def layer(mix, mlp):
    return {"type": mix[0], "mixer": mix[1], "mlp": mlp}


def model(vocab, width, layers, eps=1e-5, bigram=None):
    out = {"architecture": "Tekezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if bigram is not None:
        out["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    return out


YARN_A, YARN_B = (4.0, 64, 8.0, 1.0), (6.0, 96, 24.0, 2.0)

# padded cache rows (40 + 8 -> 48, values of 40 beside keys of 24); attention first; values shared around a layer that
# does not share; multipliers beyond the table's size
TA = model(157, 72, [
    layer(attention(4, 2, 24, 40, 0.2, 12, window=21, keep_first=3, softcap=4.0, factor=3.0, v_mix=True), moe(40, 5, 2, shared=(56, 0.9))),
    layer(latent(3, 24, 8, 20, 40, 0.21, window=19, scaling=YARN_A), dense(100)),
    layer(attention(3, 3, 20, 24, 0.25, 20, window=33, keep_first=0, softcap=9.0), None),
    layer(attention(4, 1, 24, 80, 0.22, 8, window=18, keep_first=20, softcap=6.0, v_mix=True), moe(24, 3, 1)),
    layer(latent(2, 16, 8, 28, 40, 0.25, window=33, scaling=YARN_A), dense(56, limit=0.7)),
], bigram=(61, 1009, 77))

# tensor-core row widths (64 and 128), windows beyond a query tile and a key range, wide query groups, whole rotation
TB = model(263, 128, [
    layer(latent(8, 32, 16, 32, 48, 0.15, window=150), moe(64, 4, 2, shared=(96, 1.5))),
    layer(attention(8, 2, 64, 32, 0.125, 64, window=140, keep_first=5, softcap=12.0, factor=2.5, v_mix=True), dense(192, limit=2.5)),
    layer(latent(4, 48, 32, 24, 96, 0.12, window=70, base=1000.0, scaling=YARN_B), None),
    layer(attention(40, 2, 16, 32, 0.25, 8, window=300, keep_first=1, softcap=30.0, base=500.0, v_mix=True), moe(64, 4, 2)),
    layer(attention(2, 1, 128, 64, 0.09, 32, softcap=7.0, v_mix=True), dense(64)),
], eps=1e-6, bigram=(509, 31, 5))

# sizes that fit no 16-byte group; one head everywhere; no window, no cap, no table of pairs; every expert taken; a window of one
TC = model(97, 52, [
    layer(latent(1, 10, 6, 7, 13, 0.4), moe(20, 3, 3, shared=(11, 1.1))),
    layer(attention(1, 1, 10, 25, 0.3, 4, v_mix=True), dense(50)),
    layer(attention(5, 5, 6, 5, 0.35, 2, window=1, keep_first=2, softcap=3.0, v_mix=True), None),
    layer(latent(3, 6, 6, 9, 13, 0.35, window=5), dense(30)),
], eps=3e-6)

CASES = {"ta": (TA, 81), "tb": (TB, 82), "tc": (TC, 83)}


def no_choice(cfg: dict) -> dict:
    """The same model with every expert taken: no close call between two experts can change the path."""
    out = json.loads(json.dumps(cfg))
    for spec in out["layers"]:
        if spec.get("mlp") and spec["mlp"]["kind"] == "moe":
            spec["mlp"]["router"]["top"] = spec["mlp"]["router"]["experts"]
    return out


def tensor_shapes(cfg: dict) -> dict:
    w, v = cfg["width"], cfg["vocab"]
    shapes = {"embed": (v, w), "final.norm": (w,)}
    if (cfg.get("embedding") or {}).get("bigram"):
        shapes["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, w)
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = (w,)
        shapes[p + "mix.o"] = (w, H * dv)
        if spec["type"] == "latent_attention":
            r, rank = m["rot_dim"], m["kv_rank"]
            shapes.update({p + "mix.q": (H * (d + r), w), p + "mix.dkv": (rank + r, w), p + "mix.dkv.norm": (rank,),
                           p + "mix.uk": (H * d, rank), p + "mix.uv": (H * dv, rank), p + "mix.g": (H, w)})
        else:
            G = m["kv_heads"]
            shapes.update({p + "mix.q": (H * d, w), p + "mix.k": (G * d, w), p + "mix.v": (G * dv, w), p + "mix.q.norm": (H * d,),
                           p + "mix.k.norm": (G * d,)})
            if m.get("v_mix"):
                shapes[p + "mix.vmix"] = ()
        mlp = spec.get("mlp")
        if not mlp:
            continue
        shapes[p + "norm2"] = (w,)
        sizes = {"": mlp["ff"]} if mlp["kind"] == "dense" else {f"e{e}.": mlp["expert"]["ff"] for e in range(mlp["router"]["experts"])}
        if mlp["kind"] == "moe":
            shapes[p + "mlp.router"] = (mlp["router"]["experts"], w)
            if mlp.get("shared"):
                sizes["shared."] = mlp["shared"]["ff"]
        for which, ff in sizes.items():
            shapes.update({p + f"mlp.{which}gate": (ff, w), p + f"mlp.{which}up": (ff, w), p + f"mlp.{which}down": (w, ff)})
    return shapes


def make_weights(cfg: dict, seed: int, gain: float = 1.0, calm: bool = False) -> dict:
    """Seeded weights, every value representable in bfloat16 (so a bfloat16 engine and a float oracle start alike).
    `gain` scales the queries (of the grouped attention through the weight of their norm): a larger one makes the softmax
    peaked.  Norm weights, gates, routers and feed-forwards are spread widely, so that leaving one out, or a limit, or using
    an offset without its one, moves the logits.  `calm`: flatter softmaxes, gates and routers, for bfloat16 runs of whole
    models: among hundreds of positions some have a sub-block whose output nearly cancels, and its norm magnifies the one
    rounding of what the sub-block read (the plain implementation, given rounded inputs, strays as far there)."""
    gain, spread = (0.5 * gain, 1.0 / 3.0) if calm else (gain, 1.0)
    rng = np.random.default_rng(seed)
    out = {}
    latent_layers = {f"l{i}." for i, spec in enumerate(cfg["layers"]) if spec["type"] == "latent_attention"}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            value = 0.3 * rng.standard_normal(shape)
        elif leaf == "norm":                                   # plain weights: of the latent, of queries and keys
            value = (1.0 + 0.3 * rng.standard_normal(shape)) * (gain if name.endswith("q.norm") else 1.0)
        elif leaf == "vmix":
            value = 0.25 + 0.4 * rng.random()
        elif leaf == "router":
            value = 1.5 * spread / np.sqrt(shape[1]) * rng.standard_normal(shape)
        elif name == "embed":
            value = rng.standard_normal(shape)
        elif name == "bigram":
            value = 0.8 * rng.standard_normal(shape)
        elif ".mix." in name and leaf == "q" and name[:name.index("mix.")] in latent_layers:
            value = gain / np.sqrt(shape[1]) * rng.standard_normal(shape)
        elif leaf == "g":
            value = 1.5 * spread * rng.standard_normal(shape) / np.sqrt(shape[-1])
        elif leaf in ("gate", "up"):
            value = (1.0 if calm else 1.5) * rng.standard_normal(shape) / np.sqrt(shape[-1])
        else:
            value = rng.standard_normal(shape) / np.sqrt(shape[-1])
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


def one_layer(mix, mlp=None, width=64, vocab=101, bigram=None):
    return model(vocab, width, [layer(mix, mlp)], bigram=bigram)
