"""Kezunex through the engine against the plain implementation (tests/plain_kezunex.py).

Each mechanism alone (the seam of two norms between sub-blocks, the short convolution with its kept inputs and step sizes,
the matrix recurrence token by token and chunk by chunk with and without its normaliser, the exponential gates, the real-gated
recurrence on each of its paths, the output norms, per-head query and key norms with the query temperature, the gelu gate
on every product kernel), one-layer models, then whole models under every way of cutting and batching: whole prompts,
prefill against token-by-token decoding, portions down to two and one tokens, unequal requests side by side with pages and
slots used again, a request alone and in a crowd, long decoding, the first tokens of a sequence, tokens made to stand out
far back, graphs with recurrent state, and greedy generation through the scheduler, the command line and the trace program.
"""
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import kezunex_models as km
import plain_kezunex as pk
import replay

pytestmark = pytest.mark.gpu
F = torch.float64
LENGTHS = {"a": 150, "b": 70, "c": 33, "d": 200, "e": 90, "f": 3, "g": 129, "h": 64, "i": 47, "j": 1}
_cache = {}


# ------------------------------------------------------------------ helpers
def plain(cfg, weights, tokens):
    return pk.forward(cfg, weights, tokens).numpy()


def setup(case, dtype, tmp_path_factory, gain=1.0, lengths=None):
    key = (case, dtype, gain, None if lengths is None else tuple(sorted(lengths.items())))
    if key not in _cache:
        from cisr_b200 import Model

        cfg, seed = km.CASES[case]
        weights = km.make_weights(cfg, seed, gain=gain)
        path = km.write_model_dir(tmp_path_factory.mktemp(f"{case}_{dtype}"), cfg, weights)
        model = Model.from_pretrained(path, dtype=dtype)
        requests = {rid: km.random_tokens(cfg, n, 100 + i) for i, (rid, n) in enumerate((lengths or LENGTHS).items())}
        ref_key = (case, gain, key[3])
        if ref_key not in _cache:
            _cache[ref_key] = Reference((rid, plain(cfg, weights, tokens)) for rid, tokens in requests.items())
        reference = _cache[ref_key]
        if dtype == "bfloat16" and not reference.rounding:
            for rid, tokens in requests.items():
                rounded = pk.forward(cfg, weights, tokens, taken=lambda h: h.to(torch.bfloat16).to(F)).numpy()
                reference.rounding[rid] = [replay.relative_rms(row, ref) for row, ref in zip(rounded, reference[rid])]
        _cache[key] = (cfg, weights, path, model, requests, reference)
    return _cache[key]


class Reference(dict):
    """Plain logits by request, and per row the relative RMS error that rounding the sub-blocks' inputs to bfloat16 alone
    makes in the plain implementation."""

    def __init__(self, items):
        super().__init__(items)
        self.rounding = {}


def compare(got, requests, reference, dtype, scale=4.0):
    """float32: the replay tests' bound.  bfloat16: the replay tests' bound, or twice the error that rounding the inputs of
    the sub-blocks alone makes in the plain implementation at that row, where that is larger: a read-out of a matrix memory that
    nearly cancels is divided by its own small root mean square (one row in some thousands, the same under every cut)."""
    if dtype == "float32" or not getattr(reference, "rounding", None):
        return replay.compare(got, requests, reference, dtype, scale=scale)
    wide = 0
    for (rid, pos), row in got.items():
        own = 2.0 * reference.rounding[rid][pos]
        wide += own > replay.RRMS16
        replay.compare({(rid, pos): row}, requests, reference, dtype, rrms=max(replay.RRMS16, own))
    assert wide <= max(8, len(got) // 50), "too many rows with a bound of their own"


def stepper_for(model, steps, slack_pages=0):
    from cisr_b200 import Stepper
    return Stepper(model, n_pages=replay.max_live_tokens(steps) // 16 + slack_pages, page_size=16, max_slots=4)


def model_of(cfg, weights, tmp_path, dtype="float32"):
    from cisr_b200 import Model
    return Model.from_pretrained(km.write_model_dir(tmp_path, cfg, weights), dtype=dtype)


def dev(a):
    return torch.from_numpy(np.asarray(a, dtype=np.int32)).cuda()


def near(got, want, tol=2e-5):
    err = float((got.double().cpu() - want).abs().max() / want.abs().max().clamp(min=1e-30))
    assert err < tol, f"differs by {err} of the largest value"


class Cut:
    """Requests' rows cut into steps: which rows of each request a step holds, with the lists the kernels read."""

    def __init__(self, lengths, cuts, slots):
        self.at = {r: 0 for r in lengths}
        self.cuts = {r: list(c) for r, c in cuts.items()}
        self.slots = slots
        assert all(sum(c) == lengths[r] for r, c in cuts.items())

    def steps(self, taps=1):
        from cisr_b200.engine.batch import HostBatch
        from cisr_b200.parts.gated_linear import recurrent_step_plan
        while any(self.cuts.values()):
            batch = [r for r in sorted(self.cuts, reverse=True) if self.cuts[r]]
            sizes = [self.cuts[r].pop(0) for r in batch]
            starts = [sum(sizes[:i]) for i in range(len(sizes))]
            rows = [(r, self.at[r], n) for r, n in zip(batch, sizes)]
            host = HostBatch(batch, [self.slots[r] for r in batch], starts, sizes, [self.at[r] + n for r, n in zip(batch, sizes)], sum(sizes), [])
            plan = recurrent_step_plan(host, taps)
            lists = {k: dev(v) for k, v in plan.arrays.items()}
            meta = dict(req_slot=dev(host.slots), q_start=dev(starts), q_len=dev(sizes))
            yield rows, meta, plan, lists
            for r, n in zip(batch, sizes):
                self.at[r] += n


LONG_CUTS = {0: [64, 130, 1, 9, 63, 2], 1: [3, 1, 200, 64, 1, 0 + 2]}
SLOTS = {0: 3, 1: 1}


# ------------------------------------------------------------------ each mechanism alone: kernels
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, hidden", [(3, 52), (5, 71), (130, 72), (9, 256), (200, 576), (70, 1024), (4, 4096), (90, 4096), (3, 9000), (70, 6144), (2, 20000)])
def test_seam_of_two_norms(tokens, hidden, dtype):
    """Every combination of what may be pending, both kinds of norm, and rows picked at the end of a model."""
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(hidden)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, y, extra, vec = rnd(tokens, hidden) + 0.7, 30.0 + 5.0 * rnd(tokens, hidden), rnd(tokens, hidden), rnd(hidden)
    post_w, pre_w = 1 + 0.4 * rnd(hidden), 1 + 0.4 * rnd(hidden)
    norm = {"layer": lambda v, w, e: pk.layer_norm(v.to(F), w.to(F), e), "rms": lambda v, w, e: pk.rms(v.to(F), e) * w.to(F)}
    tol = 3e-6 if dtype == torch.float32 else 1e-2
    for has_y, has_extra, has_vec, post, pre in ((1, 0, 0, "layer", "layer"), (1, 1, 1, "layer", "layer"), (0, 0, 1, "layer", "layer"),
                                                 (0, 0, 0, "layer", "layer"), (1, 0, 1, "rms", "layer"), (1, 1, 0, "layer", "rms")):
        want = x.to(F)
        if has_y:
            want = want + norm[post](y, post_w, 1e-3)
        if has_extra:
            want = want + extra.to(F)
        if has_vec:
            want = want + vec.to(F)
        given = dict(y=y.cuda() if has_y else None, post_w=post_w.cuda(), post_eps=1e-3, post_kind=post, extra=extra.cuda() if has_extra else None,
                     vector=vec.cuda() if has_vec else None, pre_w=pre_w.cuda(), pre_eps=1e-5, pre_kind=pre)
        xs, h = x.cuda(), torch.empty((tokens, hidden), dtype=dtype, device="cuda")
        kernels.post_norm(xs, x_out=xs, h=h, **given)
        near(xs, want, 3e-6)
        near(h, norm[pre](want, pre_w, 1e-5), tol)
        rows = dev([tokens - 1, 0, tokens // 2])
        xs, h = x.cuda(), torch.empty((3, hidden), dtype=dtype, device="cuda")
        kernels.post_norm(xs, h=h, rows=rows, **given)
        assert torch.equal(xs.cpu(), x), "picking rows reads only"
        near(h, norm[pre](want[rows.cpu().long()], pre_w, 1e-5), tol)


@pytest.mark.parametrize("channels, taps, silu, blocks", [(37, 4, True, 0), (256, 3, False, 4), (130, 2, True, 0), (48, 1, False, 3), (72, 6, False, 0), (20, 20, True, 0)])
def test_short_convolution_with_kept_inputs(channels, taps, silu, blocks):
    """Portions of every size down to one token, shorter than the kept inputs too; slots that held another request; the
    input's bias is part of what is kept (before the sequence there are zeros, not biases); step sizes; the three summands."""
    from cisr_b200.ops import kernels
    from cisr_b200.parts.gated_linear import conv_tile
    g = torch.Generator().manual_seed(channels * 10 + taps)
    rnd = lambda *s: torch.randn(*s, generator=g)
    cuts = {0: [40, 1, 1, 2, 17, 3], 1: [1, 2, 33, 1, 5, 18]}
    lengths = {r: sum(c) for r, c in cuts.items()}
    heads = 5
    proj = {r: rnd(n, channels + 9) for r, n in lengths.items()}
    w, bias, in_bias = rnd(channels, taps), rnd(channels), rnd(channels)
    dt_bias, a_log = rnd(heads), rnd(heads)
    want = {r: pk.short_conv(p[:, 3:3 + channels].to(F) + in_bias.to(F), w.to(F), bias.to(F)) for r, p in proj.items()}
    if silu:
        want = {r: pk.silu(v) for r, v in want.items()}
    offset = 12
    state = rnd(5, offset + (taps - 1) * channels + 3).cuda()
    for s in SLOTS.values():
        state[s].zero_()
    got, steps = {0: [], 1: []}, {0: [], 1: []}
    for rows, meta, plan, lists in Cut(lengths, cuts, SLOTS).steps(taps):
        p = torch.cat([proj[r][at:at + n] for r, at, n in rows]).cuda()
        out = torch.full((p.shape[0], channels), 7.0, device="cuda")
        la, dt = torch.empty(p.shape[0], heads, device="cuda"), torch.empty(p.shape[0], heads, device="cuda")
        split = torch.zeros((blocks, p.shape[0] + 4, 3, channels // blocks), dtype=torch.bfloat16, device="cuda") if blocks else None
        kernels.short_conv(p, 3, w.t().contiguous().cuda(), bias.cuda(), state, offset, **meta, tile_req=lists["tile_req"], tile_t0=lists["tile_t0"],
                           n_tiles=plan.info["n_tiles"], tile=conv_tile(taps), out=out, silu=silu, in_bias=in_bias.cuda(),
                           steps=(channels + 4, dt_bias.cuda(), a_log.cuda(), la, dt), split=split)
        if blocks:
            whole = split.float().sum(2)[:, :p.shape[0]].permute(1, 0, 2).reshape(p.shape[0], channels)
            assert (whole - out).abs().max() <= 2.0 ** -23 * out.abs().max()
        first = 0
        for r, at, n in rows:
            got[r].append(out[first:first + n].cpu())
            steps[r].append(torch.stack((la, dt))[:, first:first + n].cpu())
            first += n
    for r in lengths:
        near(torch.cat(got[r]), want[r], 3e-6)
        dt = pk.softplus(proj[r][:, channels + 4:channels + 4 + heads].to(F) + dt_bias.to(F))
        near(torch.cat(steps[r], dim=1), torch.stack((-torch.exp(a_log.to(F)) * dt, dt)), 3e-6)
    assert state[[0, 2, 4]].abs().min() > 0 or taps == 1, "other slots are left alone"


@pytest.mark.parametrize("heads, groups, N, dv, norm", [(2, 1, 16, 12, False), (4, 2, 128, 64, False), (3, 3, 6, 7, False), (2, 1, 70, 130, False), (6, 2, 34, 10, False),
                                                        (2, 2, 32, 64, True), (1, 1, 9, 25, True), (2, 2, 72, 136, True), (1, 1, 256, 96, True), (1, 1, 400, 8, True)])
def test_matrix_recurrence_token_by_token_and_chunk_by_chunk(heads, groups, N, dv, norm):
    """Two requests in portions of every kind (one token, a few, a whole chunk, several chunks with a tail), both forms side
    by side in one step, rows not in slot order, slots that held another state; a run of very strong decays inside a chunk in front of weak ones."""
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(heads * 1000 + N)
    rnd = lambda *s: torch.randn(*s, generator=g)
    lengths = {r: sum(c) for r, c in LONG_CUTS.items()}
    q, k, v, la, gain = {}, {}, {}, {}, {}
    for r, n in lengths.items():
        q[r], k[r], v[r] = rnd(n, groups * N + 3), rnd(n, groups * N), rnd(n, heads * dv + 2)
        la[r], gain[r] = -torch.rand(n, heads, generator=g) * torch.tensor([0.02, 0.3, 1.0])[torch.arange(heads) % 3], torch.rand(n, heads, generator=g)
        la[r][70:95] = -20.0
    want, want_n = {}, {}
    for r, n in lengths.items():
        S, nn = torch.zeros(heads, N, dv, dtype=F), torch.zeros(heads, N, dtype=F)
        ys, ns = [], []
        for t in range(n):
            kk = k[r][t].to(F).view(groups, N).repeat_interleave(heads // groups, 0) * gain[r][t].to(F).view(heads, 1)
            qq = 0.5 * q[r][t, 3:].to(F).view(groups, N).repeat_interleave(heads // groups, 0)
            dec = torch.exp(la[r][t].to(F)).view(heads, 1)
            S = dec.unsqueeze(2) * S + kk.unsqueeze(2) * v[r][t, 2:].to(F).view(heads, 1, dv)
            nn = dec * nn + kk
            ys.append((S * qq.unsqueeze(2)).sum(1))
            ns.append((nn * qq).sum(1))
        want[r], want_n[r] = torch.stack(ys), torch.stack(ns)
    size = heads * N * (dv + 1)
    state = rnd(5, -(-size // 4) * 4 + 4).cuda()
    untouched = state[[0, 2, 4]].clone()
    for s in SLOTS.values():
        state[s].zero_()
    got, got_n = {0: [], 1: []}, {0: [], 1: []}
    for rows, meta, plan, lists in Cut(lengths, LONG_CUTS, SLOTS).steps():
        cat = lambda d: torch.cat([d[r][at:at + n] for r, at, n in rows]).cuda()
        y = torch.full((sum(n for _, _, n in rows), heads, dv), 7.0, device="cuda")
        yn = torch.full(y.shape[:2], 7.0, device="cuda") if norm else None
        chunks = (lists["chunk_req"], lists["chunk_t0"], lists["req_chunk0"], plan.info["n_chunks"]) if plan.info["n_chunks"] else None
        kernels.gated_recurrence(cat(q), 3, cat(k), 0, cat(v), 2, cat(la), cat(gain), state, meta["req_slot"], meta["q_start"], meta["q_len"], len(rows), y,
                                 groups, N, q_scale=0.5, yn=yn, least=kernels.GATED_CHUNK if chunks else 0, n_short=plan.info["n_short"], chunks=chunks)
        first = 0
        for r, at, n in rows:
            got[r].append(y[first:first + n].cpu())
            if norm:
                got_n[r].append(yn[first:first + n].cpu())
            first += n
    assert torch.equal(state[[0, 2, 4]], untouched), "other slots are left alone"
    for r in lengths:
        near(torch.cat(got[r]), want[r])
        # behind the run of strong decays nothing of the start is left: a ratio of decays that lost its digits would show
        near(torch.cat(got[r])[96:140], want[r][96:140], 1e-5)
        if norm:
            near(torch.cat(got_n[r]), want_n[r])
    walked = torch.zeros_like(state)
    for r, n in lengths.items():                              # the same tokens, all token by token, leave the same state
        y = torch.empty((n, heads, dv), device="cuda")
        yn = torch.empty((n, heads), device="cuda") if norm else None
        kernels.gated_recurrence(q[r].cuda(), 3, k[r].cuda(), 0, v[r].cuda(), 2, la[r].cuda(), gain[r].cuda(), walked, dev([SLOTS[r]]), dev([0]), dev([n]), 1, y,
                                 groups, N, q_scale=0.5, yn=yn)
        near(y, want[r])
        used = heads * N * (dv + int(norm))
        near(state[SLOTS[r], :used], walked[SLOTS[r], :used].double().cpu(), 5e-5)


@pytest.mark.parametrize("heads, cap", [(3, 12.0), (1, 2.0), (5, 40.0)])
def test_exponential_gates_and_the_running_maximum(heads, cap):
    """m is a scan over a portion of any length, carried from step to step and kept per slot; la and g are formed from the
    stored maxima."""
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(heads)
    cuts = {0: [300, 1, 2, 31, 33], 1: [1, 1, 257, 128, 5]}
    lengths = {r: sum(c) for r, c in cuts.items()}
    proj = {r: 1.5 * cap * torch.randn(n, 2 * heads + 5, generator=g) for r, n in lengths.items()}
    bi, bf = torch.randn(heads, generator=g), torch.randn(heads, generator=g)
    state = torch.randn(5, 7 + heads, generator=g).cuda()
    for s in SLOTS.values():
        state[s].zero_()
    got = {0: [], 1: []}
    for rows, meta, plan, lists in Cut(lengths, cuts, SLOTS).steps():
        p = torch.cat([proj[r][at:at + n] for r, at, n in rows]).cuda()
        out = torch.empty((3, p.shape[0], heads), device="cuda")
        kernels.exp_gates(p, 2, 2 + heads, bi.cuda(), bf.cuda(), cap, state, 7, meta["req_slot"], meta["q_start"], meta["q_len"], len(rows), out[0], out[1],
                          out[2], longest=plan.info["longest"])
        first = 0
        for r, at, n in rows:
            got[r].append(out[:, first:first + n].double().cpu())
            first += n
    for r, n in lengths.items():
        la, gain, m = torch.cat(got[r], dim=1)
        i = cap * torch.tanh((proj[r][:, 2:2 + heads].to(F) + bi.to(F)) / cap)
        f = pk.log_sigmoid(cap * torch.tanh((proj[r][:, 2 + heads:2 + 2 * heads].to(F) + bf.to(F)) / cap))
        want, before = [], torch.zeros(heads, dtype=F)
        for t in range(n):
            new = torch.maximum(f[t] + before, i[t])
            want.append((f[t] + before - new, torch.exp(i[t] - new), new))
            before = new
        for a, b in zip((la, gain, m), (torch.stack(x) for x in zip(*want))):
            assert torch.allclose(a, b, rtol=1e-5, atol=2e-5)
        assert torch.equal(state[SLOTS[r], 7:].double().cpu(), m[-1]), "the kept maximum is the last token's"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, heads, dv, pad", [(3, 2, 25, 6), (70, 4, 136, 0)])
def test_outputs_of_the_matrix_recurrences(tokens, heads, dv, pad, dtype):
    """The normaliser (below and above its floor), the norm per head and the gate; the skip term, the gate before the norm, parts
    of the row, a factor, another operand in front and zeros behind."""
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(dv)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    inner = heads * dv
    y, yn, m, gate, w = rnd(tokens, heads, dv), 2 * rnd(tokens, heads), rnd(tokens, heads), rnd(tokens, inner + 7), 1 + 0.4 * rnd(inner)
    out = torch.full((tokens, inner + pad), 5.0, dtype=dtype, device="cuda")
    kernels.exp_output(y.cuda(), yn.cuda(), m.cuda(), gate.cuda(), 4, w.cuda(), 1e-3, out)
    down = torch.maximum(yn.to(F).abs(), torch.exp(-m.to(F))) + 1e-6
    want = pk.rms(y.to(F) / down.unsqueeze(2), 1e-3).reshape(tokens, inner) * w.to(F) * torch.sigmoid(gate[:, 4:4 + inner].to(F))
    near(out[:, :inner], want, tol)
    assert (out[:, inner:] == 5.0).all()
    x, D = rnd(tokens, inner + 11), rnd(heads)
    for parts, lead_width, scale in ((1, 0, 1.0), (heads, 20, -1.7), (2, 3, 0.5)):
        lead = rnd(tokens, lead_width).to(dtype) if lead_width else None
        out = torch.full((tokens, lead_width + inner + pad), 5.0, dtype=dtype, device="cuda")
        kernels.ssd_output(y.cuda(), x.cuda(), D.cuda(), gate.cuda(), 7, w.cuda(), 1e-3, out, parts=parts, scale=scale, lead=None if lead is None else lead.cuda())
        v = (y.to(F) + D.to(F).view(heads, 1) * x[:, :inner].to(F).view(tokens, heads, dv)).reshape(tokens, inner) * pk.silu(gate[:, 7:7 + inner].to(F))
        want = scale * pk.rms(v.view(tokens, parts, inner // parts), 1e-3).reshape(tokens, inner) * w.to(F)
        near(out[:, lead_width:lead_width + inner], want, tol)
        assert lead is None or torch.equal(out[:, :lead_width].cpu(), lead)
        assert (out[:, lead_width + inner:] == 0).all()


@pytest.mark.parametrize("w_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("blocks, block", [(3, 20), (1, 33), (2, 64), (1, 600), (5, 8)])
def test_real_gated_recurrence_on_each_of_its_paths(blocks, block, w_dtype):
    """Steps of a few tokens (one kernel), longer steps (the row kernel's sums, then the scan over segments of any length), and in
    bfloat16 with 128 tokens and more the three-summand product: outputs, state, and the sums themselves to float accuracy."""
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(blocks * 100 + block)
    rnd = lambda *s: torch.randn(*s, generator=g)
    width = blocks * block
    cuts = {0: [3, 150, 1, 40, 2, 9, 16], 1: [5, 129, 1, 1, 8, 300, 1]}
    lengths = {r: sum(c) for r, c in cuts.items()}
    w = (rnd(blocks, 2 * block, block) / block ** 0.5).to(w_dtype)
    bias, rate, gate_bias = rnd(blocks, 2 * block), -8.0 * torch.nn.functional.softplus(-4 + 2 * rnd(width)), rnd(width)
    u, gate = {r: rnd(n, width) for r, n in lengths.items()}, {r: rnd(n, width + 5) for r, n in lengths.items()}
    sums, want = {}, {}
    for r, n in lengths.items():
        pre = torch.einsum("tbk,bok->bto", u[r].to(F).view(n, blocks, block), w.to(F)) + bias.to(F).unsqueeze(1)
        sums[r] = pre
        a = torch.sigmoid(pre[:, :, :block]).permute(1, 0, 2).reshape(n, width)
        i = torch.sigmoid(pre[:, :, block:]).permute(1, 0, 2).reshape(n, width)
        S, rows = torch.zeros(width, dtype=F), []
        for t in range(n):
            log_a = rate.to(F) * a[t]
            S = torch.exp(log_a) * S + torch.sqrt(1 - torch.exp(log_a) ** 2) * i[t] * u[r][t].to(F)
            rows.append(S)
        want[r] = torch.stack(rows) * pk.gelu_tanh(gate[r][:, 2:2 + width].to(F) + gate_bias.to(F))
    state = rnd(5, 4 + width).cuda()
    for s in SLOTS.values():
        state[s].zero_()
    got = {0: [], 1: []}
    tol = 2e-5 if w_dtype == torch.float32 else 1e-2
    ran = set()
    for rows, meta, plan, lists in Cut(lengths, cuts, SLOTS).steps():
        cat = lambda d: torch.cat([d[r][at:at + n] for r, at, n in rows]).cuda().contiguous()
        us, gs = cat(u), cat(gate)
        tokens = us.shape[0]
        out = torch.full((tokens, width + 2), 7.0, dtype=w_dtype, device="cuda")
        rest = (rate.cuda(), state, 4)
        token_req = dev(sum([[i] * n for i, (_, _, n) in enumerate(rows)], []))
        if tokens <= kernels.RGLRU_FUSED_TOKENS:
            kernels.rglru_step(us, w.cuda(), bias.cuda(), *rest, token_req, meta["req_slot"], meta["q_start"], meta["q_len"], gs, 2, gate_bias.cuda(), out)
            ran.add("one kernel")
        else:
            padded = -(-tokens // 128) * 128
            pre = torch.full((blocks, padded, 2 * block), 7.0, device="cuda")
            given = bias.cuda()
            if w_dtype == torch.bfloat16 and block % 8 == 0 and tokens >= 128:
                x = us.view(tokens, blocks, block).permute(1, 0, 2)
                hi = x.bfloat16()
                mid = (x - hi.float()).bfloat16()
                split = torch.zeros((blocks, padded, 3, block), dtype=torch.bfloat16, device="cuda")
                split[:, :tokens, 0], split[:, :tokens, 1], split[:, :tokens, 2] = hi, mid, (x - hi.float() - mid.float()).bfloat16()
                kernels.gemm_tcgen05_grouped(split.view(blocks * padded, 3 * block), w.repeat(1, 1, 3).cuda().contiguous(), pre.view(blocks * padded, 2 * block),
                                             dev(np.repeat(np.arange(blocks), padded // 128)))
                sums_here, ran_here = pre[:, :tokens] + given.unsqueeze(1), "tensor cores"
            else:
                kernels.rglru_gates(us, w.cuda(), given, pre)
                given, sums_here, ran_here = None, pre[:, :tokens], "row kernel"
            ran.add(ran_here)
            near(sums_here, torch.cat([sums[r][:, at:at + n] for r, at, n in rows], dim=1), 5e-6)      # float sums of up to 1800 terms
            kernels.rglru_scan(pre, given, us, *rest, meta["req_slot"], meta["q_start"], meta["q_len"], len(rows), gs, 2, gate_bias.cuda(), out,
                               longest=plan.info["longest"])
        first = 0
        for r, at, n in rows:
            got[r].append(out[first:first + n, :width].cpu())
            first += n
        assert (out[:, width:] == 7.0).all()
    assert ran >= {"one kernel", "row kernel" if w_dtype == torch.float32 or block % 8 else "tensor cores"}
    for r in lengths:
        near(torch.cat(got[r]), want[r], tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hq, hkv, dk, dv, temp", [(4, 2, 20, 12, (0.4, 7)), (2, 1, 64, 64, None), (3, 3, 10, 26, (0.2, 2.5))])
def test_query_and_key_norm_per_head_and_query_temperature(hq, hkv, dk, dv, temp, dtype):
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(dk)
    width, tokens, page = -(-max(dk, dv) // 16) * 16, 23, 8
    nq, nk, nv = hq * dk, hkv * dk, hkv * dv
    proj = 3 * torch.randn(tokens, nq + nk + nv + 5, generator=g)          # columns behind the values belong to another reader
    qn, kn = 1 + 0.4 * torch.randn(dk, generator=g), 1 + 0.4 * torch.randn(dk, generator=g)
    positions = np.arange(5, 5 + tokens, dtype=np.int32)
    table = dev([[4, 0, 2, 5]])
    q = torch.full((tokens, hq, width), 7.0, dtype=dtype, device="cuda")
    k_cache, v_cache = (torch.full((6, hkv, page, width), 9.0, dtype=dtype, device="cuda") for _ in range(2))
    kernels.attention_rows(proj.cuda(), nq, nq + nk, bias=None, q_norm=qn.cuda(), k_norm=kn.cuda(), eps=1e-3, cos=None, sin=None, rot_half=0, interleaved=False,
                           q_out=q, k_cache=k_cache, v_cache=v_cache, token_req=dev([0] * tokens), positions=dev(positions), req_slot=dev([0]),
                           block_table=table, page_size=page, hq=hq, hkv=hkv, key_dim=dk, value_dim=dv, norm_per_head=True, q_temp=temp)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    want = pk.rms(proj[:, :nq].to(F).view(tokens, hq, dk), 1e-3) * qn.to(F)
    if temp:
        want = want * pk.query_temperature(5 + tokens, *temp)[5:].view(-1, 1, 1)
    near(q[:, :, :dk], want, tol)
    assert (q[:, :, dk:] == 0).all()
    want_k = pk.rms(proj[:, nq:nq + nk].to(F).view(tokens, hkv, dk), 1e-3) * kn.to(F)
    for t, pos in enumerate(positions):
        p, off = [4, 0, 2, 5][pos // page], pos % page
        near(k_cache[p, :, off, :dk], want_k[t], tol)
        near(v_cache[p, :, off, :dv], proj[t, nq + nk:nq + nk + nv].to(F).view(hkv, dv), tol)


@pytest.mark.parametrize("tokens, inter, k", [(3, 72, 128), (16, 1024, 4096), (1, 40, 72), (200, 136, 256), (600, 2048, 64), (50, 36, 50)])
def test_gelu_gate_on_every_product_kernel(tokens, inter, k):
    """down(gelu(gate(h)) * up(h)) takes its activation in the epilogue of the weight-streaming kernels, of the tcgen05
    product, or in a kernel of its own."""
    from cisr_b200.config import PartSpec
    from cisr_b200.ops import kernels
    from cisr_b200.parts import FEED_FORWARDS, build_part
    g = torch.Generator().manual_seed(inter)
    bf = lambda x: x.to(torch.bfloat16)
    gate, up, down = (bf(torch.randn(*s, generator=g) / s[1] ** 0.5) for s in ((inter, k), (inter, k), (k, inter)))
    h = bf(2 * torch.randn(tokens, k, generator=g))
    act = pk.gelu_tanh(h.to(F) @ gate.to(F).T) * (h.to(F) @ up.to(F).T)
    want = act @ down.to(F).T
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        part = build_part(FEED_FORWARDS, PartSpec("swiglu", {"hidden_size": k, "intermediate_size": inter, "activation": "gelu_tanh",
                                                             "names": {"gate": "gate", "up": "up", "down": "down"}}), dtype, "feed-forward")
        part.load({n: t.to(dtype).cuda() for n, t in (("gate", gate), ("up", up), ("down", down))})
        near(part.forward(h.to(dtype).cuda(), None), want, tol)
    if tokens <= 16 and inter % 8 == 0:
        for kind in ("latency", "stream"):
            out = torch.empty((tokens, inter), dtype=torch.bfloat16, device="cuda")
            try:
                kernels.skinny_gemm(torch.cat((gate, up)).cuda(), tokens, act=h.cuda(), epilogue=kernels.EPI_SWIGLU, out=out, kind=kind, gate="gelu_tanh")
            except kernels.KernelError as e:
                assert "does not take this shape" in str(e)
                continue
            near(out, act, 1e-2)


# ------------------------------------------------------------------ one layer is the whole model
MIXES = [km.rglru(60, 3, conv=5), km.rglru(128, 2), km.mlstm(3, 10, 7, cap=5.0), km.mlstm(2, 72, 136),
         km.parallel(km.left(4, 2, 20, 12, 0.3, (0.4, 7)), km.right(4, 10, 6, groups=2, conv=3, parts=2), 0.7, 1.3),
         km.parallel(km.left(2, 1, 64, 64, 0.2, (0.3, 40)), km.right(2, 64, 128), 1.0, -0.4),
         km.parallel(km.left(2, 2, 16, 16, 0.4), km.right(2, 16, 16), 0.0, 1.0), km.parallel(km.left(1, 1, 128, 96, 0.1), km.right(1, 8, 8), 1.2, 0.0),
         km.parallel(km.left(2, 1, 160, 40, 0.1, (0.5, 100)), km.right(2, 24, 40, conv=2), 1.0, 1.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mix", MIXES)
def test_one_layer_of_each_mixer_and_the_stream_after_it(mix, dtype, tmp_path):
    """The residual stream after the layer (output norms, scales) and the logits, whole, decoded and in portions that cut
    inside chunks, pages and convolutions."""
    from cisr_b200 import StepEntry, Stepper
    cfg = km.one_layer(mix, 80, width=72)
    weights = km.make_weights(cfg, 11)
    model = model_of(cfg, weights, tmp_path, dtype)
    requests = {"p": km.random_tokens(cfg, 210, 1), "q": km.random_tokens(cfg, 70, 2)}
    reference = {k: plain(cfg, weights, t) for k, t in requests.items()}
    stream = pk.streams(cfg, weights, requests["p"])[0]
    seen = []
    model.layer_probe = lambda i, s: seen.append(s.total().double().cpu())
    stepper = Stepper(model, n_pages=20, page_size=16, max_slots=2)
    stepper.create("p")
    stepper.step([StepEntry("p", requests["p"], [])])
    model.layer_probe = None
    near(seen[0], stream, 2e-5 if dtype == "float32" else 3e-2)
    for steps in (replay.trace_whole(requests), replay.trace_tail_decode(requests, 40), replay.trace_portions(requests, (64, 2, 65, 1, 70, 3))):
        compare(replay.run_steps(stepper_for(model, steps, slack_pages=1), steps), requests, reference, dtype)


# ------------------------------------------------------------------ whole models under every cut
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(km.CASES))
def test_whole_prompts_and_the_stream_after_every_run(case, dtype, tmp_path_factory):
    from cisr_b200 import StepEntry, Stepper
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    steps = replay.trace_whole(requests)
    compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, dtype)
    seen = []
    model.layer_probe = lambda i, s: seen.append(s.total().double().cpu())
    stepper = Stepper(model, n_pages=20, page_size=16, max_slots=1)
    stepper.create("c")
    stepper.step([StepEntry("c", requests["c"], [])])
    model.layer_probe = None
    want = pk.streams(cfg, weights, requests["c"])
    assert len(seen) == len(want)
    for got, x in zip(seen, want):
        near(got, x, 3e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(km.CASES))
def test_prefill_against_token_by_token_decoding(case, dtype, tmp_path_factory):
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    steps = replay.trace_tail_decode(requests, 60)
    compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case, sizes", [("ka", (16, 2, 15, 17, 3, 64, 33)), ("kb", (2, 2, 1, 5)), ("kc", (128, 7, 2, 130)), ("ka", (1,)), ("kb", (2,)),
                                         ("kb", (65, 63, 2, 64)), ("kc", (4, 3, 5, 2))])
def test_portions_of_several_sizes(case, sizes, dtype, tmp_path_factory):
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    if max(sizes) <= 5:
        requests = {k: requests[k] for k in ("b", "c", "f", "j")}
    steps = replay.trace_portions(requests, sizes)
    compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(km.CASES))
def test_unequal_requests_side_by_side_with_pages_and_slots_used_again(case, dtype, tmp_path_factory):
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    steps = replay.trace_mixed(requests, seed=7, sizes=(9, 2, 17, 5, 3, 70, 2, 11))
    stepper = stepper_for(model, steps)
    compare(replay.run_steps(stepper, steps), requests, reference, dtype)
    assert not stepper.cache.requests and len(stepper.cache.free_slots) == 4
    assert all(g.pool.n_free == g.pool.n_pages for g in stepper.cache.page_groups)
    assert all(g.pool.taken > g.pool.n_pages for g in stepper.cache.page_groups), "no page was used twice"


def test_a_request_alone_and_in_a_crowd(tmp_path_factory):
    """The same request by itself and beside three others of other lengths, portion by portion and token by token:
    float32 logits agree far inside the comparison's bound (the products may choose another kernel by the step's token
    count, and so may the real-gated recurrence; everything else is the same arithmetic in the same order)."""
    from cisr_b200 import StepEntry, Stepper
    cfg, weights, path, model, requests, reference = setup("ka", "float32", tmp_path_factory)
    target = requests["e"]
    cuts = [30, 2, 17, 1, 1, 1, 20, 1, 1] + [1] * 16
    alone = Stepper(model, n_pages=40, page_size=16, max_slots=4)
    crowd = Stepper(model, n_pages=40, page_size=16, max_slots=4)
    alone.create("t")
    for key in ("x", "t", "y", "z"):
        crowd.create(key)
    others = {"x": requests["a"], "y": requests["d"], "z": requests["g"]}
    at, step = 0, 0
    for n in cuts:
        want = list(range(n))
        a = alone.step([StepEntry("t", target[at:at + n], want)]).cpu().numpy()
        entries = [StepEntry("x", others["x"][3 * step:3 * step + 3], []), StepEntry("t", target[at:at + n], want),
                   StepEntry("y", others["y"][step:step + 1], [0]), StepEntry("z", others["z"][4 * step:4 * step + 4], [])]
        b = crowd.step(entries).cpu().numpy()[:n]
        for i in range(n):
            assert replay.relative_rms(a[i], b[i].astype(np.float64)) < 5e-6, f"position {at + i} depends on its neighbours"
            compare({("e", at + i): a[i]}, requests, reference, "float32")
        at += n
        step += 1


@pytest.mark.parametrize("case", ["ka", "kb"])
def test_long_decoding(case, tmp_path_factory):
    """330 tokens one by one from the first: every recurrence runs far past its chunk length token by token."""
    cfg, weights, path, model, _, _ = setup(case, "float32", tmp_path_factory)
    requests = {"long": km.random_tokens(cfg, 330, 77)}
    reference = {"long": plain(cfg, weights, requests["long"])}
    steps = replay.trace_portions(requests, (1,))
    compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, "float32")


@pytest.mark.parametrize("case", list(km.CASES))
def test_first_tokens_of_a_sequence(case, tmp_path_factory):
    """Positions 0, 1, 2, ...: states and the running maximum start at zero, convolutions reach before the sequence, a softmax
    over a single key; whole, in two-token portions and one by one, also with nothing wanted in a step."""
    cfg, weights, path, model, _, _ = setup(case, "float32", tmp_path_factory)
    requests = {f"s{n}": km.random_tokens(cfg, n, 300 + n) for n in (1, 2, 3, 4, 6, 9)}
    reference = {k: plain(cfg, weights, t) for k, t in requests.items()}
    for steps in (replay.trace_whole(requests), replay.trace_portions(requests, (2,)), replay.trace_portions(requests, (1,))):
        compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, "float32")
    nothing_wanted = [{"step": 0, "entries": [{"id": "s9", "tokens": requests["s9"][:5], "want": []}], "end": []},
                      {"step": 1, "entries": [{"id": "s9", "tokens": requests["s9"][5:], "want": [3]}], "end": ["s9"]}]
    got = replay.run_steps(stepper_for(model, nothing_wanted), nothing_wanted)
    assert list(got) == [("s9", 8)]
    compare(got, requests, reference, "float32")


def stands_out(cfg, weights, filler, place):
    """The token of the vocabulary's last eight that moves the last position's plain logits most when put at `place`."""
    without = plain(cfg, weights, filler)[-1]
    effect = {}
    for b in range(cfg["vocab"] - 8, cfg["vocab"], 3):
        tokens = list(filler)
        tokens[place] = b
        effect[b] = replay.relative_rms(plain(cfg, weights, tokens)[-1], without)
    key = max(effect, key=effect.get)
    assert effect[key] > 1e-3, f"a token at {place} does not matter: the test would show nothing"
    return key


def far_model(which):
    """One layer whose last position still sees a token hundreds of places back.  The vocabulary's last eight tokens carry a
    large number in a channel that no other token uses; the layer's keys (the inputs of its state) read that channel, and its
    decays are made weak enough that the state still holds it."""
    if which == "attention":
        cfg = km.one_layer(km.parallel(km.left(2, 1, 32, 32, 0.6, (0.2, 50)), km.right(1, 4, 4), 1.0, 0.0), width=64)
    elif which == "state space":
        cfg = km.one_layer(km.parallel(km.left(1, 1, 16, 16, 0.3), km.right(2, 16, 24), 0.0, 1.0), width=64)
    elif which == "rglru":
        cfg = km.one_layer(km.rglru(48, 2), width=64)
    else:
        cfg = km.one_layer(km.mlstm(2, 24, 16), width=64)
    w = km.make_weights(cfg, 6, gain=3.0)
    w["embed"][:, 0] = 0.0
    w["embed"][-8:, 0] = 8.0
    if which == "attention":                                 # every query has a constant part along the direction those keys take
        w["embed"][:, 1] = 1.0
        w["l0.mix.left.k"][:, 0], w["l0.mix.left.q"][:, 1] = 1.0, 0.5
        w["l0.mix.left.q.norm"] = w["l0.mix.left.q.norm"].abs()
        w["l0.mix.left.k.norm"] = w["l0.mix.left.k.norm"].abs()
    elif which == "state space":
        w["l0.mix.right.A_log"][:] = -4.0
        w["l0.mix.right.dt_bias"][:] = -3.0
        w["l0.mix.right.in"][-2:] *= 0.25
        w["l0.mix.right.in"][:, 0] = 1.0
        w["l0.mix.right.D"][:] = 0.0
    elif which == "rglru":
        w["l0.mix.lam"][:] = -9.0
        w["l0.mix.x"][:, 0] = 1.0
    else:
        w["l0.mix.f.b"][:] = 9.0
        w["l0.mix.f"] *= 0.1
        w["l0.mix.k"][:, 0] = 1.0
    return cfg, {k: v.to(torch.bfloat16).to(F) for k, v in w.items()}


@pytest.mark.parametrize("which", ["attention", "state space", "rglru", "mlstm"])
def test_a_token_far_back(which, tmp_path):
    """A token that occurs once, hundreds of places back (behind several chunks, pages and key ranges), moves the last
    logits: whole, decoded from early on, and in portions."""
    from cisr_b200 import Stepper
    cfg, weights = far_model(which)
    model = model_of(cfg, weights, tmp_path)
    rng = np.random.default_rng(1)
    n = 600
    filler = [int(t) for t in rng.integers(0, cfg["vocab"] - 8, size=n)]
    for place in (3, 255, 256):
        tokens = list(filler)
        tokens[place] = stands_out(cfg, weights, filler, place)
        requests, reference = {"r": tokens}, {"r": plain(cfg, weights, tokens)}
        for steps in (replay.trace_whole(requests), replay.trace_tail_decode(requests, 330), replay.trace_portions(requests, (250, 6, 1, 64, 130))):
            compare(replay.run_steps(Stepper(model, n_pages=40, page_size=16, max_slots=2), steps), requests, reference, "float32", scale=2.0)


def test_sharp_attention_depends_on_single_keys(tmp_path_factory):
    """With the query norm's weights scaled up the softmax is peaked: each query's weight sits on one or two keys, so a wrong,
    missing or stale key shows.  float32 only."""
    lengths = {"x": 300, "y": 170, "z": 61}
    cfg, weights, path, model, requests, reference = setup("kb", "float32", tmp_path_factory, gain=4.0, lengths=lengths)
    for steps in (replay.trace_whole(requests), replay.trace_mixed(requests, seed=3), replay.trace_tail_decode(requests, 160),
                  replay.trace_portions(requests, (16, 2, 15, 17, 3, 64, 33))):
        compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, "float32", scale=8.0)


@pytest.mark.parametrize("case, dtype", [("ka", "float32"), ("kb", "float32"), ("kb", "bfloat16")])
def test_repeated_step_shapes_replay_from_graphs_with_recurrent_state(case, dtype, tmp_path_factory):
    """Steps of the same shape recur: from the second time on the step is a graph replay.  The warm-up run in front of a
    capture must not advance any request's state twice; 140 tokens in a step take the tensor-core gates."""
    from cisr_b200 import StepEntry, Stepper
    cfg, weights, path, model, _, _ = setup(case, dtype, tmp_path_factory)
    stepper = Stepper(model, n_pages=60, page_size=16, max_slots=4, graph=True)
    tokens = {k: km.random_tokens(cfg, 201, 20 + i) for i, k in enumerate("abcd")}
    reference = {k: plain(cfg, weights, t) for k, t in tokens.items()}
    got = {}
    for k in "abcd":
        stepper.create(k)
    plan = [[("a", 0, 140)], [("b", 0, 140)], [("c", 0, 140)], [("d", 0, 140)], [("a", 140, 30)],
            [("b", 140, 20), ("a", 170, 1)], [("c", 140, 20), ("a", 171, 1)], [("d", 140, 20), ("b", 160, 1)],
            [("a", 172, 1), ("b", 161, 1)], [("a", 173, 1), ("b", 162, 1)], [("a", 174, 1), ("b", 163, 1)]]
    for step in plan:
        entries = [StepEntry(k, tokens[k][at:at + n], [n - 1, 0] if n > 1 else [0]) for k, at, n in step]
        logits = stepper.step(entries).cpu().numpy()
        row = 0
        for k, at, n in step:
            for w in ([n - 1, 0] if n > 1 else [0]):
                got[(k, at + w)] = logits[row].copy()
                row += 1
        stepper.cache.check()
    compare(got, tokens, reference, dtype)
    report = stepper.graphs.report()
    assert report["shape_entries"] >= 2 and report["hits"] >= 4


# ------------------------------------------------------------------ generation through the scheduler and the command line
@pytest.mark.parametrize("case, graph", [("ka", False), ("ka", True), ("kc", False)])
def test_greedy_generation_through_the_scheduler(case, graph, tmp_path_factory):
    """More requests than slots, few pages: requests wait, run in portions under a token budget, decode side by side,
    end, and their pages and slots serve the next ones.  float32 tokens equal the plain greedy choice."""
    from cisr_b200 import Engine, Request
    cfg, weights, path, model, _, _ = setup(case, "float32", tmp_path_factory)
    prompts = {f"g{i}": km.random_tokens(cfg, n, 50 + i) for i, n in enumerate((19, 5, 40, 2, 27, 11))}
    engine = Engine.for_model(model, pages=7, page_size=16, max_active=3, token_budget=24, prefill_chunk=9, policy="decode_first", graph=graph)
    for key, prompt in prompts.items():
        engine.submit(Request(key, prompt, max_new_tokens=7))
    got = {r.key: r.generated for r in engine.run()}
    assert got == {k: pk.generate_greedy(cfg, weights, p, 7) for k, p in prompts.items()}
    assert not engine.stepper.cache.requests and all(g.pool.n_free == g.pool.n_pages for g in engine.stepper.cache.page_groups)


def test_a_forked_request_continues_with_a_state_of_its_own(tmp_path_factory):
    """Two continuations of one prompt: pages are shared until written, every state is copied."""
    from cisr_b200 import StepEntry, Stepper
    cfg, weights, path, model, requests, _ = setup("ka", "float32", tmp_path_factory)
    stepper = Stepper(model, n_pages=40, page_size=16, max_slots=3)
    stem, ends = requests["e"][:77], {"u": requests["a"][:30], "v": requests["d"][:30]}
    stepper.create("u")
    stepper.step([StepEntry("u", stem, [])])
    stepper.fork("u", "v")
    got = {k: [] for k in ends}
    for t in range(30):
        logits = stepper.step([StepEntry(k, [ends[k][t]], [0]) for k in ends]).cpu().numpy()
        for i, k in enumerate(ends):
            got[k].append(logits[i])
    reference = {k: plain(cfg, weights, stem + e) for k, e in ends.items()}
    compare({(k, 77 + t): got[k][t] for k in ends for t in range(30)}, {k: stem + e for k, e in ends.items()}, reference, "float32")


def test_command_line_and_trace_program(tmp_path_factory, tmp_path):
    cfg, weights, path, model, requests, reference = setup("kb", "float32", tmp_path_factory)
    short = {k: requests[k] for k in ("c", "f", "i", "j", "h")}
    steps = replay.trace_mixed(short, seed=5, max_live=4)
    for dtype in ("float32", "bfloat16"):
        got = replay.run_trace_program(path, dtype, steps, tmp_path / dtype, replay.max_live_tokens(steps), cfg["vocab"])
        compare(got, short, reference, dtype)
    listing = tmp_path / "requests.json"
    listing.write_text(json.dumps([{"key": "only", "prompt": requests["c"][:9], "max_new_tokens": 4}]))
    proc = subprocess.run([sys.executable, "-m", "cisr_b200", "--config", "kezunex-small", "--dtype", "float32", "--requests", str(listing),
                           "--pages", "16"], capture_output=True, text=True, timeout=900, cwd=str(replay.ROOT))
    assert proc.returncode == 0, proc.stderr[-3000:]
    out = json.loads(proc.stdout[proc.stdout.index("{"):])
    assert out["weights"] == "random-kezunex-small" and len(out["requests"][0]["generated"]) == 4
