"""Kezunex, plainly: float64 torch on whole sequences, one function per mechanism, no cache, no batching.

The engine's kernels are compared with this; it shares no code with them.  `w` maps tensor names to float64
tensors; `cfg` is the config.json dict.  The recurrences go token by token; the slow ones are vectorised over heads only.
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
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(dim=-1, keepdim=True) + eps) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return -softplus(-z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, channels], taps [channels, n]: out[t] = bias + sum_j taps[:, n - 1 - j] x[t - j], zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x) + bias
    for j in range(n):
        out[j:] += taps[:, n - 1 - j] * x[:T - j] if j < T else 0.0
    return out


# ------------------------------------------------------------------ softmax attention
def query_temperature(T: int, coef: float, every: float) -> torch.Tensor:
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(T)], dtype=F)


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]: causal, consecutive query heads share a key head."""
    T, H, _ = q.shape
    share = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    future = torch.triu(torch.ones(T, T, dtype=torch.bool), diagonal=1)
    for h in range(H):
        scores = (q[:, h] @ k[:, h // share].T) * scale
        scores[future] = -math.inf
        e = torch.exp(scores - scores.max(dim=-1, keepdim=True).values)
        out[:, h] = (e / e.sum(dim=-1, keepdim=True)) @ v[:, h // share]
    return out


def attention(w: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T).view(T, H, d), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T).view(T, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(T, G, dv)
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"]).view(T, 1, 1)
    return softmax_attention(q, k, v, m["scale"]).reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------ selective state space
def ssd_recurrence(x, B, C, dt, a_log, D):
    """x [T, H, dv], B and C [T, G, N], dt [T, H]: S <- exp(-exp(a_log) dt) S + dt B x^T; y = S^T C + D x, from S = 0."""
    T, H, dv = x.shape
    N, share = B.shape[2], H // B.shape[1]
    y = torch.zeros(T, H, dv, dtype=F)
    S = torch.zeros(H, N, dv, dtype=F)
    for t in range(T):
        Bt, Ct = B[t].repeat_interleave(share, 0), C[t].repeat_interleave(share, 0)
        S = torch.exp(-torch.exp(a_log) * dt[t]).view(H, 1, 1) * S + (dt[t].view(H, 1) * Bt).unsqueeze(2) * x[t].unsqueeze(1)
        y[t] = (S * Ct.unsqueeze(2)).sum(1) + D.view(H, 1) * x[t]
    return y


def mamba2(w: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    u = h @ w[p + "in"].T
    z, conv_in, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    c = silu(short_conv(conv_in, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = c[:, :inner].view(T, H, dv), c[:, inner:inner + G * N].view(T, G, N), c[:, inner + G * N:].view(T, G, N)
    y = ssd_recurrence(x, B, C, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"]).reshape(T, inner)
    y = rms((y * silu(z)).view(T, m["norm_groups"], inner // m["norm_groups"]), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def parallel(w: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    return (m["left_scale"] * attention(w, p + "left.", m["left"], h, eps)
            + m["right_scale"] * mamba2(w, p + "right.", m["right"], h, eps))


# ------------------------------------------------------------------ real-gated linear recurrence
def block_diagonal(u: torch.Tensor, blocks: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """u [T, width] in parts, each times its own square matrix [out, in], plus its bias."""
    n, size, _ = blocks.shape
    return torch.cat([u[:, b * size:(b + 1) * size] @ blocks[b].T + bias[b] for b in range(n)], dim=1)


def rglru_recurrence(u, r, i, lam):
    """u, r, i [T, width], lam [width]: log a = -8 r softplus(lam); S <- a S + sqrt(1 - a^2) i u, from S = 0."""
    out = torch.zeros_like(u)
    S = torch.zeros_like(lam)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def rglru(w: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = short_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_diagonal(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_diagonal(u, w[p + "ri"], w[p + "ri.b"]))
    return (rglru_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


# ------------------------------------------------------------------ matrix memory with exponential gates
def mlstm_recurrence(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, dv], log gates i, f [T, H]: the stabilised matrix memory, token by token, everything zero
    (the running maximum too) before the first."""
    T, H, d = q.shape
    S, n, m = torch.zeros(H, d, v.shape[2], dtype=F), torch.zeros(H, d, dtype=F), torch.zeros(H, dtype=F)
    out = torch.zeros_like(v)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep.view(H, 1, 1) * S + add.view(H, 1, 1) * k[t].unsqueeze(2) * v[t].unsqueeze(1)
        n = keep.view(H, 1) * n + add.view(H, 1) * k[t]
        m = new
        down = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t].unsqueeze(2)).sum(1) / down.view(H, 1)
    return out


def mlstm(w: dict, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q, k = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5, (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o = rms(mlstm_recurrence(q, k, v, i, f), eps).reshape(T, H * dv) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward, layer, model
def gated_ff(w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"parallel": parallel, "rglru": rglru, "mlstm": mlstm}


def layer(w: dict, cfg: dict, i: int, x: torch.Tensor, taken=lambda h: h) -> torch.Tensor:
    """`taken`: what a sub-block makes of its normed input before anything else (a rounding, to see what that alone does)."""
    spec, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    y = MIXERS[spec["type"]](w, p + "mix.", spec["mixer"], taken(layer_norm(x, w[p + "norm1"], eps)), eps)
    x = x + layer_norm(y, w[p + "norm1b"], eps) * w[p + "ls1"]
    if spec.get("mlp"):
        y = gated_ff(w, p + "mlp.", taken(layer_norm(x, w[p + "norm2"], eps)))
        x = x + layer_norm(y, w[p + "norm2b"], eps) * w[p + "ls2"]
    return x


def run_order(cfg: dict) -> list:
    """(layer, pass number or None where no pass begins) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, None) for i in range(start)]
    for t in range(times):
        out += [(i, t if i == start else None) for i in range(start, stop)]
    return out + [(i, None) for i in range(stop, n)]


def streams(cfg: dict, w: dict, tokens, taken=lambda h: h) -> list:
    """The residual stream after every layer run."""
    embedded = w["embed"][torch.tensor(list(tokens))] * cfg["embedding"]["scale"]
    x, out = embedded, []
    for i, t in run_order(cfg):
        if t is not None:
            if t > 0:
                x = x + embedded
            x = x + w["loop.step"][t]
        x = layer(w, cfg, i, x, taken)
        out.append(x)
    return out


def logits_of(cfg: dict, w: dict, x: torch.Tensor) -> torch.Tensor:
    return layer_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T


def forward(cfg: dict, w: dict, tokens, taken=lambda h: h) -> torch.Tensor:
    """Float64 logits [len(tokens), vocab]."""
    return logits_of(cfg, w, streams(cfg, w, tokens, taken)[-1])


def generate_greedy(cfg: dict, w: dict, prompt, n: int) -> list:
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(torch.argmax(forward(cfg, w, seq)[-1])))
    return seq[len(prompt):]
