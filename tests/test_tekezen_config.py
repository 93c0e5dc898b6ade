"""Tekezen on the CPU: the configuration class, the spec it emits, the tensors the assembled model asks for, the cache groups
of its layers and the state of its embedding, and the changed rotary frequencies against the plain ones."""
import copy

import pytest
import torch

import plain_tekezen as pt
import tekezen_models as tm
from cisr_b200.cache import CacheManager
from cisr_b200.config import ConfigError, architecture_for, preset
from cisr_b200.engine.model import Model


def spec_of(cfg):
    return architecture_for(cfg).config_class.from_dict(cfg).to_spec()


@pytest.mark.parametrize("case", sorted(tm.CASES))
def test_the_model_asks_for_exactly_the_designs_tensors(case):
    cfg, _ = tm.CASES[case]
    needs = Model(spec_of(cfg), "float32", config=cfg, device=None).tensor_needs()
    assert {k: tuple(v.shape) for k, v in needs.items() if v.alias is None} == {k: tuple(v) for k, v in tm.tensor_shapes(cfg).items()}
    assert [k for k, v in needs.items() if v.alias is not None] == ["head"] and needs["head"].alias == "embed"


def test_spec_carries_every_constant_of_the_configuration():
    spec = spec_of(tm.TA)
    assert [l.mixer.kind for l in spec.layers] == ["windowed_attention", "latent_attention", "windowed_attention", "windowed_attention", "latent_attention"]
    a0, l1, a2, a3 = (spec.layers[i].mixer for i in range(4))
    assert (a0["num_heads"], a0["num_kv_heads"], a0["key_dim"], a0["value_dim"], a0["scale"], a0["softcap"]) == (4, 2, 24, 40, 0.2, 4.0)
    assert (a0["window"], a0["keep_first"], a0["qk_norm"], a0["eps"]) == (21, 3, "whole", 1e-5)
    assert [m["values"] for m in (a0, a2, a3)] == ["give", None, "take"] and a3["keep_first"] == 20
    assert a0["position"].kind == "rotary_half" and a0["position"]["dim"] == 12 and a0["position"]["scaling"] == {"kind": "linear", "factor": 3.0}
    assert a2["position"].get("scaling") is None
    assert (l1["num_heads"], l1["plain_dim"], l1["rot_dim"], l1["value_dim"], l1["kv_rank"], l1["window"], l1["scale"]) == (3, 24, 8, 20, 40, 19, 0.21)
    assert l1["gate"] == "head" and not l1["sink"] and l1["position"].kind == "rotary_half"
    assert l1["position"]["scaling"] == {"kind": "yarn", "factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    f0, f1, f3 = spec.layers[0].feed_forward, spec.layers[1].feed_forward, spec.layers[3].feed_forward
    assert (f0["experts"], f0["top"], f0["limit"], f0["scores"], f0["renormalize"], f0["route_scale"]) == (5, 2, 1.2, "softmax", True, 1.0)
    assert f0["shared"] == {"size": 56, "limit": 0.9, "scaled": False} and f3["shared"] is None and f3["top"] == 1
    assert (f1.kind, f1["activation"], f1["limit"], f1["intermediate_size"]) == ("swiglu", "gated_clamp", 1.8, 100)
    assert spec.layers[2].feed_forward is None and "feed_forward_out_norm" not in spec.layers[2].extras
    assert all(l.mixer_norm is None and l.feed_forward_norm is None and l.extras["mixer_out_norm"].kind == "rms_norm_offset" for l in spec.layers)
    assert spec.embedding["pairs"] == {"buckets": 61, "mul_prev": 1009, "mul_cur": 77, "weight_name": "bigram"} and spec.head["tied_to"] == "embed"
    other = spec_of(tm.TC)
    assert other.embedding["pairs"] is None and other.layers[0].mixer["window"] is None and other.layers[1].mixer["softcap"] is None
    assert preset("tekezen-small").to_spec().embedding["pairs"]


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="lightning"), "not a mixer"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(dim=600), "not supported"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "must not exceed"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(scaling={"factor": 0.0}), "positive"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=2), "keeps no first"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), "must equal rot_dim"),
    (lambda c: c["layers"][1]["mixer"].update(kv_rank=510), "not supported"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=48), "another size"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "top"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][1]["mlp"].pop("limit"), "lacks"),
    (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "not a feed-forward"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "lacks"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "lacks"),
    (lambda c: c["norm"].pop("eps"), "lacks"),
])
def test_refusals_come_before_any_weight_is_read(change, message):
    cfg = copy.deepcopy(tm.TA)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        architecture_for(cfg).config_class.from_dict(cfg)


def test_cache_groups_and_the_embeddings_state():
    """A latent layer's rows are one plane; a windowed layer's group knows its kept first tokens and never gives their pages
    back; the embedding's newest token is one number per request slot, zeroed for a new request and copied by a fork."""
    model = Model(spec_of(tm.TA), "float32", config=tm.TA, device=None)
    uses = model.cache_uses()
    assert (uses[1].planes, uses[1].kv_heads, uses[1].head_dim, uses[1].window) == (1, 1, 48, 19)
    assert (uses[0].planes, uses[0].kv_heads, uses[0].head_dim, uses[0].window, uses[0].keep_first) == (2, 2, 48, 21, 3)
    states = model.side_states()
    assert states[:5] == [None] * 5 and (states[5].kind, states[5].state_shape, states[5].state_dtype) == ("state", (1,), "int32")
    assert Model(spec_of(tm.TC), "float32", config=tm.TC, device=None).side_states() == [None] * 4
    cache = CacheManager(uses, n_pages=12, page_size=8, max_slots=2, max_positions=256, device=torch.device("cpu"), side_states=states)
    cache.create("a")
    cache.reserve([("a", 70)])
    cache.commit("a", 70)
    cache.check()
    by_window = {g.use.window: g for g in cache.page_groups}
    assert by_window[21].pool.n_used == 3 + 1            # positions 50 .. 69 lie on pages 6 to 8; the first page holds kept tokens
    assert by_window[18].pool.n_used == 3 + 3 and by_window[19].pool.n_used == 3
    assert cache.side_state(0) is None and cache.side_state(5).shape == (3, 1)
    cache.side_state(5)[cache.slot("a")] = 17
    cache.fork("a", "b")
    assert cache.side_state(5)[cache.slot("b"), 0] == 17
    cache.release("a")
    cache.create("c")
    assert cache.side_state(5)[cache.slot("c"), 0] == 0
    cache.release("b"); cache.release("c")
    assert all(g.pool.n_free == g.pool.n_pages for g in cache.page_groups)


@pytest.mark.parametrize("base, dims, factor", [(10000.0, 12, 3.0), (500.0, 64, 1.0), (1e6, 2, 0.5)])
def test_frequencies_slowed_evenly(base, dims, factor):
    from cisr_b200.parts.rotary import scaled_frequencies
    plain = pt.plain_frequencies(base, dims)
    got, magnitude = scaled_frequencies(plain.clone(), base, dims, {"kind": "linear", "factor": factor})
    assert magnitude == 1.0 and torch.allclose(got, pt.slowed_evenly(plain, {"factor": factor}), rtol=1e-15, atol=0)


def test_rows_of_the_pair_table():
    rows = pt.bigram_rows([5, 5, 9, 0, 1], {"buckets": 7, "mul_prev": 10, "mul_cur": 3})
    assert rows == [7, (50 + 15) % 7, (50 + 27) % 7, 90 % 7, 3]
