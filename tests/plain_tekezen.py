"""Tekezen, plainly: float64 torch on whole sequences, one function per mechanism, no cache, no batching.

The engine's kernels are compared with this; it shares no code with them.  `w` maps tensor names to float64
tensors; `cfg` is the config.json dict.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


# ------------------------------------------------------------------ small pieces
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis, eps under the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """The norm of the layers' outputs and of the model's end: the tensor holds the factor's offset from one."""
    return rms(x, eps) * (1.0 + weight)


def keep_all(x: torch.Tensor) -> torch.Tensor:
    return x


# ------------------------------------------------------------------ embedding
def bigram_rows(tokens, bigram: dict):
    """Which row of the pair table each token of a sequence adds: a hash of the token and the one before it; the first
    token of a sequence has no predecessor and takes the row behind the last bucket."""
    buckets, a, b = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    rows = []
    for t, token in enumerate(tokens):
        rows.append(buckets if t == 0 else (int(tokens[t - 1]) * a + int(token) * b) % buckets)
    return rows


def embed(w: dict, cfg: dict, tokens) -> torch.Tensor:
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram:
        x = x + w["bigram"][torch.as_tensor(bigram_rows(tokens, bigram), dtype=torch.long)]
    return x


# ------------------------------------------------------------------ rotation
def plain_frequencies(base: float, dims: int) -> torch.Tensor:
    i = torch.arange(dims // 2, dtype=F)
    return base ** (-2.0 * i / dims)


def slowed_evenly(freq: torch.Tensor, s: dict) -> torch.Tensor:
    return freq / float(s["factor"])


def stretched_by_ramp(freq: torch.Tensor, base: float, dims: int, s: dict):
    """A ramp over the pair index between the pairs that make `fast` and `slow` turns over the original length; returns
    the frequencies and the factor both tables are multiplied by."""
    factor, original = float(s["factor"]), float(s["original"])

    def pair_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(float(s["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(s["slow"]))), dims - 1)
    out = freq.clone()
    for i, f in enumerate(freq.tolist()):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f / factor * ramp + f * (1.0 - ramp)
    return out, 0.1 * math.log(factor) + 1.0


def turn_halves(x: torch.Tensor, freq: torch.Tensor, magnitude: float = 1.0) -> torch.Tensor:
    """x [T, ..., n]: coordinates (i, i + len(freq)) turn by position * freq[i]; those behind 2 len(freq) pass."""
    T, half = x.shape[0], freq.numel()
    out = x.clone()
    pos = torch.arange(T, dtype=F)
    shape = [T] + [1] * (x.dim() - 2)
    for i, f in enumerate(freq.tolist()):
        c = (torch.cos(pos * f) * magnitude).view(shape)
        s = (torch.sin(pos * f) * magnitude).view(shape)
        a, b = x[..., i], x[..., i + half]
        out[..., i] = a * c - b * s
        out[..., i + half] = b * c + a * s
    return out


# ------------------------------------------------------------------ softmax over the keys in sight
def in_sight(T: int, window=None, keep_first: int = 0) -> torch.Tensor:
    """see[i, j]: j is not behind i, and is one of the last `window` keys or one of the sequence's first `keep_first`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    return see if window is None else see & ((i - j < window) | (j < keep_first))


def softmax_rows(scores: torch.Tensor, see: torch.Tensor) -> torch.Tensor:
    s = scores.masked_fill(~see, -math.inf)
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def squashed(scores: torch.Tensor, cap) -> torch.Tensor:
    """Scores bent smoothly into (-cap, cap)."""
    return scores if cap is None else float(cap) * torch.tanh(scores / float(cap))


# ------------------------------------------------------------------ latent attention
def latent_rows(w: dict, p: str, m: dict, h: torch.Tensor, eps: float):
    """Per token: the normed latent, and the turned key part that the heads share."""
    rank = m["kv_rank"]
    down = h @ w[p + "dkv"].T
    freq, magnitude = latent_frequencies(m)
    return rms(down[:, :rank], eps) * w[p + "dkv.norm"], turn_halves(down[:, rank:], freq, magnitude)


def latent_frequencies(m: dict):
    rot = m["rot"]
    freq = plain_frequencies(float(rot["base"]), int(rot["dims"]))
    return stretched_by_ramp(freq, float(rot["base"]), int(rot["dims"]), rot["scaling"]) if rot.get("scaling") else (freq, 1.0)


def latent_attention(w: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, d, r, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    T = h.shape[0]
    c, k_rot = latent_rows(w, p, m, h, eps)
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    q_rot = turn_halves(q[:, :, d:], *latent_frequencies(m))
    k_plain = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    gate = torch.sigmoid(h @ w[p + "g"].T)                       # one number per head
    see = in_sight(T, (m.get("mask") or {}).get("size"))
    heads = []
    for a in range(H):
        scores = (q[:, a, :d] @ k_plain[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        heads.append(gate[:, a:a + 1] * (softmax_rows(scores, see) @ v[:, a]))
    return torch.cat(heads, dim=1) @ w[p + "o"].T


# ------------------------------------------------------------------ grouped attention
def blend_values(v: torch.Tensor, first: torch.Tensor, lam) -> torch.Tensor:
    return (1.0 - lam) * v + lam * first


def attention(w: dict, p: str, m: dict, h: torch.Tensor, eps: float, first_values=None):
    """Returns (output, the layer's values before any blending); `first_values`: the values that join this layer's."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    rot = m["rot"]
    freq = plain_frequencies(float(rot["base"]), int(rot["dims"]))
    if rot.get("scaling"):
        freq = slowed_evenly(freq, rot["scaling"])
    q = turn_halves((rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d), freq)
    k = turn_halves((rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d), freq)
    own = h @ w[p + "v"].T
    v = (own if first_values is None else blend_values(own, first_values, w[p + "vmix"])).view(T, G, dv)
    mask = m.get("mask") or {}
    see = in_sight(T, mask.get("size"), mask.get("keep_first") or 0)
    heads = []
    for a in range(H):
        g = a // (H // G)
        heads.append(softmax_rows(squashed((q[:, a] @ k[:, g].T) * m["scale"], m.get("softcap")), see) @ v[:, g])
    return torch.cat(heads, dim=1) @ w[p + "o"].T, own


# ------------------------------------------------------------------ feed-forwards
def gated(w: dict, p: str, limit: float, h: torch.Tensor) -> torch.Tensor:
    """The one form of every feed-forward here: dense, expert and shared expert."""
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(w: dict, p: str, router: dict, h: torch.Tensor):
    """Per token: the chosen experts (best first) and the softmax over their logits alone."""
    best = torch.topk(h @ w[p + "router"].T, int(router["top"]), dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def routed(w: dict, p: str, mlp: dict, h: torch.Tensor) -> torch.Tensor:
    chosen, weight = route(w, p, mlp["router"], h)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        share = (weight * (chosen == e)).sum(dim=-1, keepdim=True)
        rows = torch.nonzero(share[:, 0] > 0).flatten()
        if rows.numel():
            out[rows] += share[rows] * gated(w, f"{p}e{e}.", float(mlp["expert"]["limit"]), h[rows])
    if mlp.get("shared"):
        out = out + gated(w, p + "shared.", float(mlp["shared"]["limit"]), h)
    return out


# ------------------------------------------------------------------ the model
def forward(cfg: dict, w: dict, tokens, after_layer=None, taken=keep_all) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; `after_layer(i, x)` is called with the stream after every layer; `taken` is
    applied to what a sublayer reads (a rounding, to see what it alone does)."""
    eps = float(cfg["norm"]["eps"])
    x = embed(w, cfg, tokens)
    first_values = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "latent_attention":
            y = latent_attention(w, p + "mix.", m, taken(x), eps)
        elif layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(w, p + "mix.", m, taken(x), eps, first_values if mixes else None)
            if mixes and first_values is None:
                first_values = own
        else:
            raise ValueError(layer["type"])
        x = x + layer_norm(y, w[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = gated(w, p + "mlp.", float(mlp["limit"]), taken(x)) if mlp["kind"] == "dense" else routed(w, p + "mlp.", mlp, taken(x))
            x = x + layer_norm(y, w[p + "norm2"], eps)
        if after_layer is not None:
            after_layer(i, x)
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T
