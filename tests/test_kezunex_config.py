"""Kezunex on the CPU: the configuration class, the spec it emits, the tensors the assembled model asks for, the caches and
states of its layers, the launch plan of the recurrences, and the plain implementation against closed forms."""
import copy

import pytest
import torch

import kezunex_models as km
import plain_kezunex as pk
from cisr_b200.cache import CacheManager
from cisr_b200.config import ConfigError, architecture_for, preset
from cisr_b200.engine.model import Model

F = torch.float64


def spec_of(cfg):
    return architecture_for(cfg).config_class.from_dict(cfg).to_spec()


@pytest.mark.parametrize("case", sorted(km.CASES))
def test_the_model_asks_for_exactly_the_designs_tensors(case):
    cfg, _ = km.CASES[case]
    needs = Model(spec_of(cfg), "float32", config=cfg, device=None).tensor_needs()
    assert {k: tuple(v.shape) for k, v in needs.items() if v.alias is None} == {k: tuple(v) for k, v in km.tensor_shapes(cfg).items()}
    assert [k for k, v in needs.items() if v.alias is not None] == ["head"] and needs["head"].alias == "embed"


def test_spec_carries_every_constant_of_the_configuration():
    spec = spec_of(km.KA)
    assert [(e.layer, e.pass_step, e.add_embedding) for e in spec.run] == [(0, None, False), (1, 0, False), (2, None, False), (1, 1, True),
                                                                           (2, None, False), (3, None, False), (4, None, False)]
    assert [l.mixer.kind for l in spec.layers] == ["rglru", "parallel", "matrix_memory", "parallel", "matrix_memory"]
    r0, p1, m2, p3 = (spec.layers[i].mixer for i in range(4))
    assert (r0["width"], r0["blocks"], r0["conv"], r0["factor"]) == (60, 3, 5, 8.0)
    a, b = p1["left"], p1["right"]
    assert (p1["left_scale"], p1["right_scale"], p3["left_scale"]) == (0.7, 1.3, -0.8)
    assert (a["num_heads"], a["num_kv_heads"], a["key_dim"], a["value_dim"], a["scale"], a["q_temp"], a["qk_norm"], a["eps"]) == (4, 2, 20, 12, 0.3, (0.4, 7.0), "head", 1e-5)
    assert a["window"] is None and a["sink"] is None and a["position"].kind == "none"
    assert (b["num_heads"], b["value_dim"], b["state_dim"], b["groups"], b["conv"], b["norm_groups"], b["eps"]) == (4, 10, 6, 2, 3, 2, 1e-5)
    assert (m2["num_heads"], m2["key_dim"], m2["value_dim"], m2["gate_cap"]) == (3, 10, 7, 5.0)
    assert spec.layers[1].feed_forward is None and "feed_forward_out_norm" not in spec.layers[1].extras
    assert (spec.layers[0].feed_forward.kind, spec.layers[0].feed_forward["activation"]) == ("swiglu", "gelu_tanh")
    assert spec.embedding["scale"] == 1.5 and spec.head["tied_to"] == "embed" and spec.stream["keep_embedding"] and spec.pass_steps["count"] == 2
    plain = spec_of(km.KC)
    assert len(plain.run) == 5 and plain.pass_steps is None and not plain.stream["keep_embedding"]
    assert plain.layers[2].mixer["left"]["q_temp"] is None
    assert len(preset("kezunex-small").to_spec().run) == 6
    once = copy.deepcopy(km.KA)
    once["loop"]["times"] = 1
    assert [(e.layer, e.pass_step, e.add_embedding) for e in spec_of(once).run][1] == (1, 0, False)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba"), "not a mixer"),
    (lambda c: c["layers"][0]["mixer"].update(blocks=7), "divide width"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(vdim=300), "not supported"),
    (lambda c: c["layers"][1]["mixer"]["left"]["q_temp"].update(every=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "lacks"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(groups=3), "groups must divide"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(state=600), "not supported"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "lacks"),
    (lambda c: c["layers"][2]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][2]["mixer"].update(dim=1024), "not supported"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not a feed-forward"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "positive"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(stop=1), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c.pop("embedding"), "lacks"),
    (lambda c: c["norm"].update(eps=0.0), "positive"),
])
def test_refusals_come_before_any_weight_is_read(change, message):
    cfg = copy.deepcopy(km.KA)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        architecture_for(cfg).config_class.from_dict(cfg)


def test_every_pass_of_a_looped_layer_has_pages_and_state_of_its_own():
    model = Model(spec_of(km.KA), "float32", config=km.KA, device=None)
    uses, sides = model.cache_uses(), model.side_states()
    assert [u.kind for u in uses] == ["state", "pages", "state", "pages", "state", "pages", "state"]
    assert [s is not None for s in sides] == [False, True, False, True, False, True, False]
    assert (uses[1].kv_heads, uses[1].head_dim, uses[1].window) == (2, 32, None)
    assert sides[1].state_shape == (4 * 6 * 10 + 2 * (40 + 2 * 12),)                   # the matrices and two kept inputs per channel
    assert uses[0].state_shape == (60 + 4 * 60,) and uses[2].state_shape == (244,)      # 3 (10 x 7 + 10) + 3, filled up to a multiple of four
    cache = CacheManager(uses, n_pages=4, page_size=16, max_slots=2, max_positions=256, device=None, side_states=sides)
    assert cache.entry_side[1] != cache.entry_side[3] and cache.entry_source[1] == 1 and cache.entry_source[3] == 3
    same_pages = next(g for g in cache.page_groups if 1 in g.entries)
    assert same_pages.entries == [1, 3] and same_pages.entry_slot[1] != same_pages.entry_slot[3]
    cache.create("a")
    cache.reserve([("a", 40)])
    cache.commit("a", 40)
    cache.check()
    cache.release("a")
    assert all(g.pool.n_free == g.pool.n_pages for g in cache.page_groups)


def test_launch_plans_of_the_recurrences():
    from cisr_b200.engine.batch import HostBatch
    from cisr_b200.ops import kernels
    from cisr_b200.parts.gated_linear import recurrent_plan_key, recurrent_step_plan
    q_len = [1, 63, 64, 133, 2]
    host = HostBatch(list("abcde"), list(range(5)), [0, 1, 64, 128, 261], q_len, q_len, sum(q_len), [])
    plan = recurrent_step_plan(host)
    assert list(zip(plan.arrays["chunk_req"], plan.arrays["chunk_t0"])) == [(2, 0), (3, 0), (3, 64), (3, 128)]
    assert list(plan.arrays["req_chunk0"]) == [0, 0, 0, 1, 4]
    assert plan.info == {"n_chunks": 4, "n_short": 3, "n_tiles": 1 + 4 + 4 + 9 + 1, "longest": 133}
    tiles = list(zip(plan.arrays["tile_req"], plan.arrays["tile_t0"]))
    assert tiles[:3] == [(0, 0), (1, 0), (1, 16)] and tiles[-2:] == [(3, 128), (4, 0)]
    wide = recurrent_step_plan(host, taps=40)                 # a tile holds at least the kept inputs
    assert wide.info["n_tiles"] == 1 + 2 + 2 + 4 + 1 and recurrent_plan_key(40) != recurrent_plan_key(4) == recurrent_plan_key(1)
    model = Model(spec_of(km.KB), "bfloat16", config=km.KB, device=None)
    planners = model.planners()
    assert len({p.plan_key() for p in planners}) == len(planners) == 4      # attention, the matrix recurrences, two block counts
    gates = next(p for p in planners if "parts" in p.plan_key() and p.blocks == 2)
    assert list(gates.step_plan(host).arrays["part_of_tile"]) == [0, 0, 0, 1, 1, 1]      # 263 tokens: three row tiles per part
    small = HostBatch(["a"], [0], [0], [20], [20], 20, [])
    assert gates.step_plan(small).arrays["part_of_tile"].size == 0 and kernels.TCGEN05_MIN_TOKENS > 20


# ------------------------------------------------------------------ the plain implementation against closed forms
def test_plain_recurrences_against_their_sums():
    """Each recurrence written as the weighted sum over all earlier tokens that it stands for."""
    g = torch.Generator().manual_seed(0)
    T, H, d, dv = 9, 2, 3, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=F) for n in (d, d, dv))
    dt, a_log, D = pk.softplus(torch.randn(T, H, generator=g, dtype=F)), torch.randn(H, generator=g, dtype=F), torch.randn(H, generator=g, dtype=F)
    got = pk.ssd_recurrence(v, k, q, dt, a_log, D)
    for h in range(H):
        for t in range(T):
            want = D[h] * v[t, h]
            for s in range(t + 1):
                want = want + torch.exp(-torch.exp(a_log[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (q[t, h] @ k[s, h]) * v[s, h]
            assert torch.allclose(got[t, h], want, rtol=1e-12)
    i, f = 3 * torch.randn(T, H, generator=g, dtype=F), pk.log_sigmoid(torch.randn(T, H, generator=g, dtype=F))
    got = pk.mlstm_recurrence(q, k, v, i, f)
    for h in range(H):
        for t in range(T):
            weight = [torch.exp(f[s + 1:t + 1, h].sum() + i[s, h]) * (q[t, h] @ k[s, h]) for s in range(t + 1)]      # not stabilised
            # the running maximum starts at zero: exp(-m) times everything, with m at least the decayed start
            m = max([float(f[:t + 1, h].sum())] + [float(f[s + 1:t + 1, h].sum() + i[s, h]) for s in range(t + 1)])
            top = sum(x * v[s, h] for s, x in enumerate(weight)) * torch.exp(torch.tensor(-m, dtype=F))
            down = max(abs(float(sum(weight))) * float(torch.exp(torch.tensor(-m, dtype=F))), float(torch.exp(torch.tensor(-m, dtype=F)))) + 1e-6
            assert torch.allclose(got[t, h], top / down, rtol=1e-10)
    u, r, gate, lam = (torch.randn(T, d, generator=g, dtype=F) for _ in range(4))
    r, gate, lam = torch.sigmoid(r), torch.sigmoid(gate), lam[0]
    got = pk.rglru_recurrence(u, r, gate, lam)
    log_a = -8.0 * r * pk.softplus(lam)
    for t in range(T):
        want = sum(torch.exp(log_a[s + 1:t + 1].sum(0)) * torch.sqrt(1 - torch.exp(log_a[s]) ** 2) * gate[s] * u[s] for s in range(t + 1))
        assert torch.allclose(got[t], want, rtol=1e-10)


def test_plain_convolution_norms_and_activations():
    g = torch.Generator().manual_seed(1)
    x, w, b = torch.randn(7, 5, generator=g, dtype=F), torch.randn(5, 4, generator=g, dtype=F), torch.randn(5, generator=g, dtype=F)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T.unsqueeze(0), (3, 0)), w.unsqueeze(1), b, groups=5)[0].T
    assert torch.allclose(pk.short_conv(x, w, b), want, rtol=1e-12)
    assert torch.allclose(pk.layer_norm(x, b, 1e-3), torch.nn.functional.layer_norm(x, (5,), b, None, 1e-3), rtol=1e-12)
    assert torch.allclose(pk.gelu_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"), rtol=1e-12)
    assert torch.allclose(pk.softplus(30 * x), torch.nn.functional.softplus(30 * x, threshold=1000), rtol=1e-12)
    assert torch.allclose(pk.log_sigmoid(30 * x), torch.nn.functional.logsigmoid(30 * x), rtol=1e-9)
    assert pk.query_temperature(6, 0.5, 3)[[0, 1, 2, 5]].tolist() == pytest.approx([1.0, 1.0, 1 + 0.5 * 0.6931471805599453, 1 + 0.5 * 1.0986122886681098])


def test_the_embedding_comes_back_before_every_pass_but_the_first():
    cfg = copy.deepcopy(km.KA)
    cfg["layers"] = cfg["layers"][:2]
    cfg["loop"] = {"start": 0, "stop": 2, "times": 3}
    w = km.make_weights(cfg, 5)
    x0 = w["embed"][torch.tensor([3, 9, 11])] * cfg["embedding"]["scale"]
    x = x0
    for t in range(3):
        x = x + (x0 if t else 0.0) + w["loop.step"][t]
        x = pk.layer(w, cfg, 1, pk.layer(w, cfg, 0, x))
    assert torch.equal(pk.streams(cfg, w, [3, 9, 11])[-1], x)
