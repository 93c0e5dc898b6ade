"""Tekezen through the engine against the plain implementation (tests/plain_tekezen.py).

Each mechanism alone (the table of token pairs with the newest token as state, values blended with an earlier layer's, the
gate per head, the read of the stream without a norm, clamped gated products on every product kernel, the router's
softmax, experts with a plain shared one, bent scores with kept first tokens on every attention kernel, cache rows beyond
256), one-layer models, then whole models under every way of cutting and batching: whole prompts, prefill against
token-by-token decoding, portions down to two and one tokens, unequal requests side by side with pages and slots used
again, a request alone and in a crowd, long decoding, the first tokens of a sequence, tokens made to stand out just inside
and just outside a window and the kept first tokens, peaked attention, replays from graphs, and greedy generation through
the scheduler, the command line and the trace program.
"""
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tekezen as pt
import replay
import tekezen_models as tm

pytestmark = pytest.mark.gpu
F = torch.float64
LENGTHS = {"a": 150, "b": 70, "c": 33, "d": 200, "e": 90, "f": 3, "g": 129, "h": 64, "i": 47, "j": 1}
_cache = {}


# ------------------------------------------------------------------ helpers
def plain(cfg, weights, tokens):
    return pt.forward(cfg, weights, tokens).numpy()


def setup(case, dtype, tmp_path_factory, gain=1.0, lengths=None):
    """bfloat16 runs use calmer weights (`tekezen_models.make_weights`) and routers that take every expert: a close call
    between two experts would send a token down another path than the plain implementation's."""
    key = (case, dtype, gain, None if lengths is None else tuple(sorted(lengths.items())))
    if key not in _cache:
        cfg, seed = tm.CASES[case]
        if dtype == "bfloat16":
            cfg = tm.no_choice(cfg)
        weights = tm.make_weights(cfg, seed, gain=gain, calm=dtype == "bfloat16")
        path = tmp_path_factory.mktemp(f"{case}_{dtype}")
        model = model_of(cfg, weights, path, dtype)
        requests = {rid: tm.random_tokens(cfg, n, 100 + i) for i, (rid, n) in enumerate((lengths or LENGTHS).items())}
        reference = {rid: plain(cfg, weights, tokens) for rid, tokens in requests.items()}
        _cache[key] = (cfg, weights, path, model, requests, reference)
    return _cache[key]


def compare(got, requests, reference, dtype, scale=4.0):
    """float32: every logit within the replay tests' bound.  bfloat16: every row's relative RMS error below twice the
    replay tests' bound, and at most one row in a hundred (or one) above the bound itself: a sub-block's output is divided
    by its root mean square, so where it is nearly zero (a position among hundreds, the same under every cut) the rounding
    of what the sub-block read and cached is magnified, while the float32 run of the same model stays inside its bound."""
    if dtype == "float32":
        return replay.compare(got, requests, reference, dtype, scale=scale)
    assert got, "nothing was compared"
    errors = {key: replay.relative_rms(row, reference[key[0]][key[1]]) for key, row in got.items()}
    assert all(np.isfinite(row).all() for row in got.values())
    worst = max(errors, key=errors.get)
    assert errors[worst] < 2 * replay.RRMS16, f"bfloat16 logits differ for request {worst[0]} at position {worst[1]}: {errors[worst]:.4f}"
    over = sorted(k for k, e in errors.items() if e >= replay.RRMS16)
    assert len(over) <= max(1, len(errors) // 100), f"bfloat16 rows over the bound: {over[:10]}"


def stepper_for(model, steps, slack_pages=0):
    from cisr_b200 import Stepper
    return Stepper(model, n_pages=replay.max_live_tokens(steps) // 16 + slack_pages, page_size=16, max_slots=4)


def model_of(cfg, weights, tmp_path, dtype="float32"):
    from cisr_b200 import Model
    return Model.from_pretrained(tm.write_model_dir(tmp_path, cfg, weights), dtype=dtype)


def dev(a):
    return torch.from_numpy(np.asarray(a, dtype=np.int32)).cuda()


def bf16_exact(x):
    return x.to(torch.bfloat16).to(F)


# ------------------------------------------------------------------ each mechanism alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("buckets, mul_prev, mul_cur, hidden, scale", [(13, 5, 3, 40, 1.0), (7, 1009, 77, 33, 0.5), (1, 4, 9, 64, 1.0), (65537, 40961, 70001, 2048, 2.0)])
def test_pair_table_and_the_newest_token_as_state(buckets, mul_prev, mul_cur, hidden, scale, dtype):
    """Three requests in portions of one, two and more tokens, in changing order and not in slot order; a slot that held
    another request before (its number is still there) starts a new sequence."""
    from cisr_b200.ops import kernels
    vocab = 50
    g = torch.Generator().manual_seed(buckets)
    table, pairs = bf16_exact(torch.randn(vocab, hidden, generator=g)), bf16_exact(torch.randn(buckets + 1, hidden, generator=g))
    rng = np.random.default_rng(3)
    tokens = {r: rng.integers(0, vocab, size=n).tolist() for r, n in {"x": 23, "y": 9, "z": 14}.items()}
    rule = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    want = {r: table[torch.tensor(t)] * scale + pairs[torch.tensor(pt.bigram_rows(t, rule))] for r, t in tokens.items()}
    slot, at = {"x": 2, "y": 0, "z": 3}, {r: 0 for r in tokens}
    last = torch.full((5, 1), 31, dtype=torch.int32).cuda()            # what other requests left behind
    plan = [[("x", 7)], [("y", 1), ("x", 2)], [("x", 1), ("z", 5), ("y", 1)], [("z", 2), ("x", 1)], [("y", 7), ("x", 12), ("z", 1)], [("z", 6)]]
    for step in plan:
        ids, positions, token_req, q_start, q_len = [], [], [], [], []
        for i, (r, n) in enumerate(step):
            q_start.append(len(ids)); q_len.append(n)
            ids += tokens[r][at[r]:at[r] + n]; positions += range(at[r], at[r] + n); token_req += [i] * n
        out = torch.full((len(ids), hidden), float("nan"), device="cuda")
        kernels.embedding_pairs(table.to(dtype).cuda(), pairs.to(dtype).cuda(), dev(ids), out, scale, mul_prev, mul_cur, last,
                                positions=dev(positions), token_req=dev(token_req), req_slot=dev([slot[r] for r, _ in step]),
                                q_start=dev(q_start), q_len=dev(q_len))
        for i, (r, n) in enumerate(step):
            got = out[q_start[i]:q_start[i] + n].double().cpu()
            assert torch.allclose(got, want[r][at[r]:at[r] + n], rtol=1e-6, atol=1e-6), f"request {r} at {at[r]}"
            at[r] += n
            assert int(last[slot[r], 0]) == tokens[r][at[r] - 1]
    assert int(last[1, 0]) == 31 and int(last[4, 0]) == 31


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hq, hkv, key_dim, value_dim, rot", [(4, 2, 24, 40, 12), (3, 3, 20, 9, 20), (1, 1, 64, 64, 32)])
def test_values_blended_with_an_earlier_layers(hq, hkv, key_dim, value_dim, rot, dtype):
    """What the row kernel leaves in the pages: keys normed over the whole projection and turned, values blended with rows
    of a wider tensor; the same call without other values leaves them as projected."""
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(hq * 100 + key_dim)
    tokens, page_size, D, eps, lam = 21, 8, -(-max(key_dim, value_dim) // 16) * 16, 1e-5, 0.37
    nq, nk, nv = hq * key_dim, hkv * key_dim, hkv * value_dim
    proj, wide = torch.randn(tokens, nq + nk + nv, generator=g), torch.randn(tokens, nv + 11, generator=g)
    q_norm, k_norm = 1 + 0.3 * torch.randn(nq, generator=g), 1 + 0.3 * torch.randn(nk, generator=g)
    freq = pt.plain_frequencies(1000.0, rot)
    angle = torch.arange(tokens, dtype=F)[:, None] * freq
    pages = [4, 0, 2]
    cache = lambda: torch.zeros((5, hkv, page_size, D), dtype=dtype, device="cuda")
    for other, blend in ((wide.cuda()[:, 5:5 + nv], lam), (None, 0.0)):
        q_out, kc, vc = torch.empty((tokens, hq, D), dtype=dtype, device="cuda"), cache(), cache()
        kernels.attention_rows(proj.cuda(), nq, nq + nk, bias=None, q_norm=q_norm.cuda(), k_norm=k_norm.cuda(), eps=eps, cos=torch.cos(angle).float().cuda(),
                               sin=torch.sin(angle).float().cuda(), rot_half=rot // 2, interleaved=False, q_out=q_out, k_cache=kc, v_cache=vc,
                               token_req=dev([0] * tokens), positions=dev(range(tokens)), req_slot=dev([1]), block_table=dev([[-1] * 3, pages]),
                               page_size=page_size, hq=hq, hkv=hkv, key_dim=key_dim, value_dim=value_dim, other_values=other, blend=blend)
        own = proj[:, nq + nk:].to(F)
        v = own if other is None else pt.blend_values(own, wide[:, 5:5 + nv].to(F), lam)
        q = pt.turn_halves((pt.rms(proj[:, :nq].to(F), eps) * q_norm.to(F)).view(tokens, hq, key_dim), freq)
        k = pt.turn_halves((pt.rms(proj[:, nq:nq + nk].to(F), eps) * k_norm.to(F)).view(tokens, hkv, key_dim), freq)
        rows = lambda c: torch.cat([c[p] for p in pages], dim=1).permute(1, 0, 2)[:tokens].double().cpu()
        tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
        assert torch.allclose(rows(vc)[:, :, :value_dim], v.view(tokens, hkv, value_dim), **tol)
        assert torch.allclose(rows(kc)[:, :, :key_dim], k, **tol) and torch.allclose(q_out[:, :, :key_dim].double().cpu(), q, **tol)
        assert not rows(vc)[:, :, value_dim:].any() and not rows(kc)[:, :, key_dim:].any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, heads, value_dim, rank", [(5, 3, 20, 40), (16, 4, 64, 96), (1, 7, 9, 13)])
def test_one_output_gate_per_head(tokens, heads, value_dim, rank, dtype):
    """Both kernels that apply the gate: the row kernel with the value product, and the one after a library product."""
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(tokens)
    row = -(-(rank + 8) // 16) * 16
    mixed = torch.randn(tokens, heads, row, generator=g).to(dtype)
    v_up = (torch.randn(heads, value_dim, rank, generator=g) / rank ** 0.5).to(dtype)
    wide = 2.0 * torch.randn(tokens, heads + 9, generator=g)
    values = torch.einsum("thr,hjr->thj", mixed[:, :, :rank].to(F), v_up.to(F))
    want = (values * torch.sigmoid(wide[:, 4:4 + heads].to(F))[:, :, None]).reshape(tokens, -1)
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    out = torch.empty((tokens, heads * value_dim), dtype=dtype, device="cuda")
    kernels.latent_values(mixed.cuda(), v_up.cuda(), wide.cuda(), 4, out, per=value_dim)
    assert torch.allclose(out.double().cpu(), want, **tol)
    out.zero_()
    kernels.latent_gate(values.float().reshape(tokens, -1).cuda(), wide.cuda(), 4, out, per=value_dim)
    assert torch.allclose(out.double().cpu(), want, **tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, width", [(3, 72), (90, 72), (200, 512), (70, 2050), (5, 4096)])
def test_the_stream_read_as_it_is(tokens, width, dtype):
    """The output norm (an offset from one) on the way into the stream, then the stream itself in the compute type; and
    picked rows through the final norm, which leave the stream as it was."""
    from cisr_b200.config import PartSpec
    from cisr_b200.parts import NORMS, STREAMS, build_part
    from cisr_b200.parts.post_norm import float_weight
    g = torch.Generator().manual_seed(width)
    norm = build_part(NORMS, PartSpec("rms_norm_offset", {"size": width, "eps": 1e-5, "weight_name": ""}), dtype, "norm")
    w = bf16_exact(0.3 * torch.randn(width, generator=g))
    norm.load({"": w.to(dtype).cuda()})
    x, y = torch.randn(tokens, width, generator=g), 5.0 * torch.randn(tokens, width, generator=g)
    stream = STREAMS["post_norm"](x.cuda(), PartSpec("post_norm"))
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    assert torch.allclose(stream.read(None, dtype).double().cpu(), x.to(F), **tol)
    stream.write(y.cuda(), (float_weight(norm), norm.eps, norm.kind))
    want = x.to(F) + pt.layer_norm(y.to(F), w, 1e-5)
    rows = [tokens - 1, 0]
    picked = stream.finish(norm, dtype, dev(rows)).double().cpu()
    assert torch.allclose(picked, pt.layer_norm(want[rows], w, 1e-5), **tol)
    h = stream.read(None, dtype)
    assert h.dtype == dtype and torch.allclose(h.double().cpu(), want, **tol)
    assert torch.allclose(stream.x.double().cpu(), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, width, ff", [(3, 72, 100), (16, 512, 4096), (9, 1024, 4096), (40, 128, 96), (300, 136, 200), (2100, 256, 384), (5, 52, 30)])
def test_clamped_gated_feed_forward_on_every_product(tokens, width, ff, dtype):
    """Few tokens (small and large matrices: the latency kernel and the persistent streaming one), tens, hundreds and
    thousands (library and tcgen05 products, both tile widths), sizes that fit no 16-byte group.  The limit cuts many of
    the gates from above and of the ups from both sides."""
    from cisr_b200.config import PartSpec
    from cisr_b200.parts import FEED_FORWARDS, build_part
    g = torch.Generator().manual_seed(tokens + ff)
    limit = 0.8
    part = build_part(FEED_FORWARDS, PartSpec("swiglu", {"hidden_size": width, "intermediate_size": ff, "activation": "gated_clamp", "limit": limit,
                                                         "names": {"gate": "gate", "up": "up", "down": "down"}}), dtype, "feed-forward")
    w = {"gate": bf16_exact(1.5 * torch.randn(ff, width, generator=g) / width ** 0.5), "up": bf16_exact(1.5 * torch.randn(ff, width, generator=g) / width ** 0.5),
         "down": bf16_exact(torch.randn(width, ff, generator=g) / ff ** 0.5)}
    part.load({k: v.to(dtype).cuda() for k, v in w.items()})
    h = bf16_exact(torch.randn(tokens, width, generator=g))
    got = part.forward(h.to(dtype).cuda(), None).double().cpu()
    want = pt.gated(w, "", limit, h)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    assert torch.allclose(got, want, rtol=tol, atol=tol * float(want.abs().max()))


@pytest.mark.parametrize("experts, top", [(5, 2), (3, 1), (40, 6), (4, 4)])
def test_router_weights_are_the_softmax_over_the_chosen_logits(experts, top):
    from cisr_b200.ops import kernels
    g = torch.Generator().manual_seed(experts)
    logits = 3.0 * torch.randn(37, experts, generator=g)
    chosen = torch.empty((37, top), dtype=torch.int32, device="cuda")
    weight = torch.empty((37, top), dtype=torch.float32, device="cuda")
    kernels.moe_select(logits.cuda(), top, 0, 0, 1.0, chosen, weight, scores="softmax", renormalize=True)
    best = torch.topk(logits.to(F), top, dim=-1)
    assert (chosen.cpu().long() == best.indices).all()
    assert torch.allclose(weight.double().cpu(), torch.softmax(best.values, dim=-1), rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, experts, top, ff, hidden, shared", [(6, 5, 2, 40, 72, 56), (1, 3, 1, 24, 64, None), (700, 4, 2, 64, 128, 96), (40, 3, 3, 20, 52, 11),
                                                                     (300, 6, 2, 32, 64, 24)])
def test_gated_experts_with_a_plain_shared_one(tokens, experts, top, ff, hidden, shared, dtype):
    from cisr_b200.config import PartSpec
    from cisr_b200.config.tekezen import EXPERT_NAMES
    from cisr_b200.parts import FEED_FORWARDS, build_part
    g = torch.Generator().manual_seed(tokens + experts)
    w = {"mlp.router": bf16_exact(3.0 / hidden ** 0.5 * torch.randn(experts, hidden, generator=g))}
    for which, size in [(f"e{e}", ff) for e in range(experts)] + ([("shared", shared)] if shared else []):
        for leaf, shape in (("gate", (size, hidden)), ("up", (size, hidden)), ("down", (hidden, size))):
            w[f"mlp.{which}.{leaf}"] = bf16_exact(1.4 * torch.randn(*shape, generator=g) / shape[1] ** 0.5)
    part = build_part(FEED_FORWARDS, PartSpec("routed_experts", {
        "hidden_size": hidden, "expert_size": ff, "experts": experts, "top": top, "scores": "softmax", "renormalize": True, "activation": "gated_clamp",
        "limit": 0.9, "shared": {"size": shared, "limit": 1.6, "scaled": False} if shared else None, "names": EXPERT_NAMES}), dtype, "feed-forward")
    assert set(part.tensor_needs()) == {k[4:] for k in w}
    part.load({k[4:]: v.to(dtype).cuda() for k, v in w.items()})
    h = bf16_exact(torch.randn(tokens, hidden, generator=g))
    got = part.forward(h.to(dtype).cuda(), None).double().cpu()
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": 0.9}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared, "limit": 1.6} if shared else None}
    want = pt.routed(w, "mlp.", mlp, h)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    assert torch.allclose(got, want, rtol=tol, atol=tol * float(want.abs().max()))


# ------------------------------------------------------------------ one layer is the whole model
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, keep", [(4, 2, 64, 32, 45, 7), (2, 1, 128, 128, 131, 70), (40, 2, 16, 16, 17, 1), (3, 3, 40, 48, None, 0),
                                                                    (6, 2, 64, 64, 200, 130), (2, 1, 144, 20, 50, 5), (1, 1, 20, 320, 33, 4)])
def test_bent_scores_and_kept_first_tokens_on_every_attention_kernel(heads, kv_heads, dim, vdim, window, keep, dtype, tmp_path):
    """Head widths of 64 and 128 (tcgen05 and tensor-map kernels in bfloat16), other widths up to 128 (`mma.sync`), wider
    ones, also beyond 256, and float32 (CUDA cores): prompts, single tokens and portions of one attention layer whose scores
    reach several times the cap, so that scores left as they are, or bent before the scale, are far off."""
    cfg = tm.one_layer(tm.attention(heads, kv_heads, dim, vdim, 6.0 / dim ** 0.5, 8, window=window, keep_first=keep, softcap=2.5, factor=1.5))
    weights = tm.make_weights(cfg, 9)
    model = model_of(cfg, weights, tmp_path, dtype)
    requests = {"p": tm.random_tokens(cfg, 333, 1), "q": tm.random_tokens(cfg, 40, 2)}
    reference = {k: plain(cfg, weights, t) for k, t in requests.items()}
    straight = json.loads(json.dumps(cfg))
    straight["layers"][0]["mixer"].pop("softcap")
    assert replay.relative_rms(plain(straight, weights, requests["q"])[-1], reference["q"][-1]) > 0.02, "the cap would not show"
    for steps in (replay.trace_whole(requests), replay.trace_tail_decode(requests, 200), replay.trace_portions(requests, (100, 2, 129, 1, 31))):
        compare(replay.run_steps(stepper_for(model, steps, slack_pages=1), steps), requests, reference, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank, rot, window, heads", [(48, 16, 45, 4), (96, 32, 131, 3), (40, 8, 17, 2), (13, 6, None, 1), (200, 24, 50, 2), (256, 32, 40, 8), (480, 32, 70, 3)])
def test_latent_rows_of_every_width(rank, rot, window, heads, dtype, tmp_path):
    """Cache rows of 64 and 128, other widths up to 128, up to 256 and beyond; the gates are spread widely."""
    cfg = tm.one_layer(tm.latent(heads, 20, rot, 24, rank, 0.2, window=window, scaling=None if rot == 6 else tm.YARN_A))
    weights = tm.make_weights(cfg, 9)
    model = model_of(cfg, weights, tmp_path, dtype)
    requests = {"p": tm.random_tokens(cfg, 300, 1), "q": tm.random_tokens(cfg, 40, 2)}
    reference = {k: plain(cfg, weights, t) for k, t in requests.items()}
    for steps in (replay.trace_whole(requests), replay.trace_tail_decode(requests, 100), replay.trace_portions(requests, (100, 2, 129, 1, 31))):
        compare(replay.run_steps(stepper_for(model, steps, slack_pages=1), steps), requests, reference, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mix", [tm.attention(4, 2, 24, 40, 0.3, 12, window=21, keep_first=3, softcap=4.0, factor=3.0), tm.attention(3, 1, 32, 32, 0.2, 32, softcap=8.0),
                                 tm.latent(3, 24, 8, 20, 40, 0.21, window=19, scaling=tm.YARN_A), tm.latent(2, 8, 16, 32, 24, 0.3)])
@pytest.mark.parametrize("mlp", [tm.dense(80, limit=0.6), tm.moe(40, 4, 4, limit=0.8, shared=(24, 0.5)), None])
def test_one_layer_of_each_kind_and_the_stream_after_it(mix, mlp, dtype, tmp_path):
    """The residual stream after the layer (output norms, clamped products, the pair table) and the logits."""
    from cisr_b200 import StepEntry, Stepper
    cfg = tm.one_layer(mix, mlp, width=72, bigram=(37, 11, 6))
    weights = tm.make_weights(cfg, 11)
    model = model_of(cfg, weights, tmp_path, dtype)
    requests = {"p": tm.random_tokens(cfg, 210, 1), "q": tm.random_tokens(cfg, 70, 2)}
    streams = {}
    reference = {k: pt.forward(cfg, weights, t, after_layer=lambda i, x, k=k: streams.__setitem__(k, x.clone())).numpy() for k, t in requests.items()}
    seen = []
    model.layer_probe = lambda i, s: seen.append(s.total().double().cpu())
    stepper = Stepper(model, n_pages=20, page_size=16, max_slots=2)
    stepper.create("p")
    stepper.step([StepEntry("p", requests["p"], [])])
    model.layer_probe = None
    tol = 2e-5 if dtype == "float32" else 3e-2
    assert torch.allclose(seen[0], streams["p"], rtol=tol, atol=tol * float(streams["p"].abs().max()))
    for steps in (replay.trace_whole(requests), replay.trace_tail_decode(requests, 40), replay.trace_portions(requests, (64, 2, 65, 1, 70, 3))):
        compare(replay.run_steps(stepper_for(model, steps, slack_pages=1), steps), requests, reference, dtype)


# ------------------------------------------------------------------ whole models under every cut
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(tm.CASES))
def test_whole_prompts(case, dtype, tmp_path_factory):
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    steps = replay.trace_whole(requests)
    compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(tm.CASES))
def test_prefill_against_token_by_token_decoding(case, dtype, tmp_path_factory):
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    steps = replay.trace_tail_decode(requests, 60)           # the windows of ta and tc pass over decoded tokens only
    compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case, sizes", [("ta", (16, 2, 15, 17, 3, 64, 33)), ("tb", (2, 2, 1, 5)), ("tc", (128, 7, 2, 130)), ("ta", (1,)), ("tb", (2,)),
                                         ("tb", (65, 63, 2, 64))])
def test_portions_of_several_sizes(case, sizes, dtype, tmp_path_factory):
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    if max(sizes) <= 5:
        requests = {k: requests[k] for k in ("b", "c", "f", "j")}
    steps = replay.trace_portions(requests, sizes)
    compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(tm.CASES))
def test_unequal_requests_side_by_side_with_pages_and_slots_used_again(case, dtype, tmp_path_factory):
    cfg, weights, path, model, requests, reference = setup(case, dtype, tmp_path_factory)
    steps = replay.trace_mixed(requests, seed=7, sizes=(9, 2, 17, 5, 3, 70, 2, 11))
    stepper = stepper_for(model, steps)
    compare(replay.run_steps(stepper, steps), requests, reference, dtype)
    assert not stepper.cache.requests and len(stepper.cache.free_slots) == 4
    assert all(g.pool.n_free == g.pool.n_pages for g in stepper.cache.page_groups)
    assert any(g.pool.taken > g.pool.n_pages for g in stepper.cache.page_groups), "no page was used twice"


def test_a_request_alone_and_in_a_crowd(tmp_path_factory):
    """The same request by itself and beside three others of other lengths, portion by portion and token by token:
    float32 logits agree far inside the comparison's bound (the products may choose another kernel by the step's token
    count; everything else is the same arithmetic in the same order)."""
    from cisr_b200 import StepEntry, Stepper
    cfg, weights, path, model, requests, reference = setup("ta", "float32", tmp_path_factory)
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
            assert replay.relative_rms(a[i], b[i].astype(np.float64)) < 1e-5, f"position {at + i} depends on its neighbours"
            compare({("e", at + i): a[i]}, requests, reference, "float32")
        at += n
        step += 1


def test_long_decoding(tmp_path_factory):
    """330 tokens one by one from the first: every window passes over decoded tokens many times, pages behind it go back
    to their pool while the request lives, and those with kept first tokens stay."""
    cfg, weights, path, model, _, _ = setup("ta", "float32", tmp_path_factory)
    requests = {"long": tm.random_tokens(cfg, 330, 77)}
    reference = {"long": plain(cfg, weights, requests["long"])}
    steps = replay.trace_portions(requests, (1,))
    stepper = stepper_for(model, steps)
    compare(replay.run_steps(stepper, steps), requests, reference, "float32")
    for g in stepper.cache.page_groups:
        if g.use.window is not None:
            assert g.pool.peak <= -(-g.use.window // 16) + 1 + -(-g.use.keep_first // 16), "a window kept pages it had passed"


def test_first_tokens_of_a_sequence(tmp_path_factory):
    """Positions 0, 1, 2, ...: the row of the pair table for a token without a predecessor, in slots that another request
    has just left, windows that are not full yet, kept tokens that are also in the window; whole, in two-token portions and
    one by one, also with nothing wanted in a step."""
    cfg, weights, path, model, _, _ = setup("ta", "float32", tmp_path_factory)
    requests = {f"s{n}": tm.random_tokens(cfg, n, 300 + n) for n in (1, 2, 3, 4, 6, 9)}
    reference = {k: plain(cfg, weights, t) for k, t in requests.items()}
    for steps in (replay.trace_whole(requests), replay.trace_portions(requests, (2,)), replay.trace_portions(requests, (1,))):
        compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, "float32")
    nothing_wanted = [{"step": 0, "entries": [{"id": "s9", "tokens": requests["s9"][:5], "want": []}], "end": []},
                      {"step": 1, "entries": [{"id": "s9", "tokens": requests["s9"][5:], "want": [3]}], "end": ["s9"]}]
    got = replay.run_steps(stepper_for(model, nothing_wanted), nothing_wanted)
    assert list(got) == [("s9", 8)]
    compare(got, requests, reference, "float32")


def test_the_token_before_a_portion(tmp_path):
    """Every token's own row is the same here, so only the pair table tells tokens apart: a portion's first token shows the
    token that an earlier step brought, in long portions as in decoding, and after a fork in both copies."""
    from cisr_b200 import StepEntry, Stepper
    cfg = tm.one_layer(tm.attention(2, 1, 16, 16, 0.3, 8, window=9, softcap=5.0), width=64, bigram=(211, 17, 29))
    weights = tm.make_weights(cfg, 4)
    tied = weights["embed"].clone()
    weights["embed"] = 0.01 * tied + tied[:1]
    weights["embed"] = bf16_exact(weights["embed"])
    model = model_of(cfg, weights, tmp_path)
    requests = {"r": tm.random_tokens(cfg, 60, 5), "s": tm.random_tokens(cfg, 45, 6)}
    reference = {k: plain(cfg, weights, t) for k, t in requests.items()}
    for steps in (replay.trace_portions(requests, (20, 2, 1, 7)), replay.trace_mixed(requests, seed=2), replay.trace_portions(requests, (1,))):
        compare(replay.run_steps(stepper_for(model, steps, slack_pages=1), steps), requests, reference, "float32")
    stepper = Stepper(model, n_pages=20, page_size=16, max_slots=3)
    stepper.create("r")
    stepper.step([StepEntry("r", requests["r"][:21], [])])
    stepper.fork("r", "copy")
    other = requests["r"][:21] + requests["s"][:4]
    got = stepper.step([StepEntry("copy", other[21:], [0, 1, 2, 3]), StepEntry("r", requests["r"][21:22], [0])]).cpu().numpy()
    compare({("o", 21 + i): got[i] for i in range(4)}, {"o": other}, {"o": plain(cfg, weights, other)}, "float32")
    compare({("r", 21): got[4]}, requests, reference, "float32")


def stands_out(cfg, weights, filler, place, seen):
    """The token of the vocabulary's last eight that moves the last position's plain logits most when put at `place`."""
    without = plain(cfg, weights, filler)[-1]
    effect = {}
    for b in range(cfg["vocab"] - 8, cfg["vocab"]):
        tokens = list(filler)
        tokens[place] = b
        effect[b] = replay.relative_rms(plain(cfg, weights, tokens)[-1], without)
    key = max(effect, key=effect.get)
    if seen:
        assert effect[key] > 1e-3, f"a token at {place} does not matter: the test would show nothing"
    else:
        assert effect[key] == 0.0, f"a token at {place}, beyond the mask, moved the plain logits"
    return key


@pytest.mark.parametrize("mix, window, keep", [(tm.latent(3, 24, 8, 20, 40, 0.5, window=37, scaling=tm.YARN_A), 37, 0),
                                               (tm.attention(4, 2, 24, 20, 0.5, 12, window=37, keep_first=5, softcap=20.0), 37, 5),
                                               (tm.attention(2, 1, 32, 48, 0.4, 32, window=50, keep_first=33, softcap=20.0, factor=2.0), 50, 33)])
def test_tokens_just_inside_and_just_outside_the_mask(mix, window, keep, tmp_path):
    """One layer is the whole model, so the last position sees exactly its mask.  A token that occurs nowhere else is put
    at the window's oldest place and one earlier, at the last kept first place and one later (the plain implementation says
    which of these move the last logits); the engine must agree with the prompt whole, decoded (the window passing page
    borders on the way) and in portions that cut at the edges."""
    from cisr_b200 import Stepper
    n = 150
    cfg = tm.one_layer(mix)
    weights = tm.make_weights(cfg, 5, gain=2.0)
    model = model_of(cfg, weights, tmp_path)
    rng = np.random.default_rng(0)
    filler = [int(t) for t in rng.integers(0, cfg["vocab"] - 8, size=n)]
    oldest_seen = n - window
    places = [(oldest_seen, True), (oldest_seen - 1, False), (n - 1, True), (keep, False)] + ([(keep - 1, True), (0, True)] if keep else [])
    for place, seen in places:
        tokens = list(filler)
        tokens[place] = stands_out(cfg, weights, filler, place, seen)
        requests, reference = {"r": tokens}, {"r": plain(cfg, weights, tokens)}
        for steps in (replay.trace_whole(requests), replay.trace_tail_decode(requests, 60),
                      replay.trace_portions(requests, (oldest_seen, 1, window - 2, 1)),
                      replay.trace_portions(requests, (oldest_seen - 1, 2, window - 1, 5)), replay.trace_portions(requests, (max(keep, 2), 1, 70, 2))):
            compare(replay.run_steps(Stepper(model, n_pages=12, page_size=16, max_slots=2), steps), requests, reference, "float32", scale=2.0)


def test_a_first_token_kept_in_sight_from_far_away(tmp_path):
    """Hundreds of places behind the window the kept first tokens are still seen, in bfloat16 kernels too: the query has a
    constant part along the direction of the key of a token that occurs only there."""
    from cisr_b200 import Stepper
    for dtype, dim in (("float32", 32), ("bfloat16", 64), ("bfloat16", 48)):
        cfg = tm.one_layer(tm.attention(2, 1, dim, dim, 8.0 / dim ** 0.5, 8, window=40, keep_first=20, softcap=25.0), width=64)
        weights = tm.make_weights(cfg, 6)
        weights["embed"][:, 0] = 0.0
        weights["embed"][-8:, 0] = 8.0
        weights["embed"][:, 1] = 1.0
        weights["l0.mix.k"][:, 0] = 1.0
        weights["l0.mix.q"][:, 1] = 0.5
        model = model_of(cfg, weights, tmp_path / f"{dtype}{dim}", dtype)
        rng = np.random.default_rng(1)
        n = 600
        filler = [int(t) for t in rng.integers(0, cfg["vocab"] - 8, size=n)]
        for place, seen in ((3, True), (19, True), (20, False), (n - 41, False), (n - 40, True)):
            tokens = list(filler)
            tokens[place] = stands_out(cfg, weights, filler, place, seen)
            requests, reference = {"r": tokens}, {"r": plain(cfg, weights, tokens)}
            for steps in (replay.trace_whole(requests), replay.trace_tail_decode(requests, 330), replay.trace_portions(requests, (250, 6, 1, 64, 130))):
                compare(replay.run_steps(Stepper(model, n_pages=40, page_size=16, max_slots=2), steps), requests, reference, dtype, scale=4.0)


def test_sharp_attention_depends_on_single_keys(tmp_path_factory):
    """With the queries scaled up the softmax is peaked (as far as the caps let it): each query's weight sits on one or
    two keys somewhere in its sight, so a wrong, missing or stale cache row shows.  float32 only."""
    lengths = {"x": 300, "y": 170, "z": 61}
    cfg, weights, path, model, requests, reference = setup("tb", "float32", tmp_path_factory, gain=4.0, lengths=lengths)
    for steps in (replay.trace_whole(requests), replay.trace_mixed(requests, seed=3), replay.trace_tail_decode(requests, 160),
                  replay.trace_portions(requests, (16, 2, 15, 17, 3, 64, 33))):
        compare(replay.run_steps(stepper_for(model, steps), steps), requests, reference, "float32", scale=8.0)


def test_each_constant_moves_the_logits(tmp_path_factory):
    """The plain logits change when a mechanism of the configuration is taken away, so the comparisons above see it."""
    cfg, weights, _, _, requests, reference = setup("ta", "float32", tmp_path_factory)

    def moved(change, w=weights):
        other = json.loads(json.dumps(cfg))
        change(other)
        return replay.relative_rms(plain(other, w, requests["b"])[-1], reference["b"][-1]) > 1e-3

    mixer = lambda c, i: c["layers"][i]["mixer"]
    assert moved(lambda c: mixer(c, 0).pop("softcap")) and moved(lambda c: mixer(c, 0)["mask"].update(keep_first=2))
    assert moved(lambda c: mixer(c, 0)["mask"].update(size=20)) and moved(lambda c: mixer(c, 1)["mask"].update(size=20))
    assert moved(lambda c: mixer(c, 0)["rot"].pop("scaling")) and moved(lambda c: mixer(c, 1)["rot"].pop("scaling"))
    assert moved(lambda c: mixer(c, 3).update(v_mix=False)) and moved(lambda c: c.pop("embedding"))
    assert moved(lambda c: c["layers"][0]["mlp"].pop("shared")) and moved(lambda c: c["layers"][0]["mlp"]["expert"].update(limit=9.0))
    assert moved(lambda c: c["layers"][1]["mlp"].update(limit=9.0)) and moved(lambda c: c["layers"][0]["mlp"]["shared"].update(limit=9.0))
    for name in ("l1.mix.g", "l0.norm1", "l0.norm2", "final.norm", "l0.mix.q.norm", "l0.mix.k.norm", "l1.mix.dkv.norm"):
        assert moved(lambda c: None, {**weights, name: torch.zeros_like(weights[name]) + (1.0 if name.endswith(("q.norm", "k.norm", "dkv.norm")) else 0.0)}), name


def test_repeated_step_shapes_replay_from_graphs(tmp_path_factory):
    """Steps of the same shape recur: from the second time on the step is a graph replay.  The warm-up run in front of a
    capture must not leave a newer token behind than the request has brought."""
    from cisr_b200 import StepEntry, Stepper
    cfg, weights, path, model, _, _ = setup("ta", "float32", tmp_path_factory)
    stepper = Stepper(model, n_pages=60, page_size=16, max_slots=4, graph=True)
    tokens = {k: tm.random_tokens(cfg, 131, 20 + i) for i, k in enumerate("abcd")}
    reference = {k: plain(cfg, weights, t) for k, t in tokens.items()}
    got = {}
    for k in "abcd":
        stepper.create(k)
    plan = [[("a", 0, 70)], [("b", 0, 70)], [("c", 0, 70)], [("d", 0, 70)], [("a", 70, 30)],
            [("b", 70, 20), ("a", 100, 1)], [("c", 70, 20), ("a", 101, 1)], [("d", 70, 20), ("b", 90, 1)],
            [("a", 102, 1), ("b", 91, 1)], [("a", 103, 1), ("b", 92, 1)], [("a", 104, 1), ("b", 93, 1)]]
    for step in plan:
        entries = [StepEntry(k, tokens[k][at:at + n], [n - 1, 0] if n > 1 else [0]) for k, at, n in step]
        logits = stepper.step(entries).cpu().numpy()
        row = 0
        for k, at, n in step:
            for w in ([n - 1, 0] if n > 1 else [0]):
                got[(k, at + w)] = logits[row].copy()
                row += 1
        stepper.cache.check()
    compare(got, tokens, reference, "float32")
    report = stepper.graphs.report()
    assert report["shape_entries"] >= 2 and report["hits"] >= 4


# ------------------------------------------------------------------ generation through the scheduler and the command line
@pytest.mark.parametrize("case, graph", [("ta", False), ("ta", True), ("tc", False)])
def test_greedy_generation_through_the_scheduler(case, graph, tmp_path_factory):
    """More requests than slots, few pages: requests wait, run in portions under a token budget, decode side by side,
    end, and their pages and slots serve the next ones.  float32 tokens equal the plain greedy choice."""
    from cisr_b200 import Engine, Request
    cfg, weights, path, model, _, _ = setup(case, "float32", tmp_path_factory)
    prompts = {f"g{i}": tm.random_tokens(cfg, n, 50 + i) for i, n in enumerate((19, 5, 40, 2, 27, 11))}
    new = 7

    def plain_greedy(prompt):
        seq = list(prompt)
        for _ in range(new):
            seq.append(int(pt.forward(cfg, weights, seq)[-1].argmax()))
        return seq[len(prompt):]

    engine = Engine.for_model(model, pages=7, page_size=16, max_active=3, token_budget=24, prefill_chunk=9, policy="decode_first", graph=graph)
    for key, prompt in prompts.items():
        engine.submit(Request(key, prompt, max_new_tokens=new))
    got = {r.key: r.generated for r in engine.run()}
    assert got == {k: plain_greedy(p) for k, p in prompts.items()}
    assert not engine.stepper.cache.requests and all(g.pool.n_free == g.pool.n_pages for g in engine.stepper.cache.page_groups)


def test_command_line_and_trace_program(tmp_path_factory, tmp_path):
    cfg, weights, path, model, requests, reference = setup("tb", "float32", tmp_path_factory)
    short = {k: requests[k] for k in ("c", "f", "i", "j", "h")}
    steps = replay.trace_mixed(short, seed=5, max_live=4)
    got = replay.run_trace_program(path, "float32", steps, tmp_path / "out", replay.max_live_tokens(steps), cfg["vocab"])
    compare(got, short, reference, "float32")
    cfg16, weights16, path16, _, requests16, reference16 = setup("tb", "bfloat16", tmp_path_factory)
    short16 = {k: requests16[k] for k in short}
    got = replay.run_trace_program(path16, "bfloat16", steps, tmp_path / "out16", replay.max_live_tokens(steps), cfg["vocab"])
    compare(got, short16, reference16, "bfloat16")
    listing = tmp_path / "requests.json"
    listing.write_text(json.dumps([{"key": "only", "prompt": requests["c"][:9], "max_new_tokens": 4}]))
    proc = subprocess.run([sys.executable, "-m", "cisr_b200", "--config", "tekezen-small", "--dtype", "float32", "--requests", str(listing),
                           "--pages", "16"], capture_output=True, text=True, timeout=900, cwd=str(replay.ROOT))
    assert proc.returncode == 0, proc.stderr[-3000:]
    out = json.loads(proc.stdout[proc.stdout.index("{"):])
    assert out["weights"] == "random-tekezen-small" and len(out["requests"][0]["generated"]) == 4
