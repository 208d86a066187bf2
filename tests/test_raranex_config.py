"""Raranex without a GPU: config.json to typed configuration and back, what is refused, the model's parts as
data (the order of layer runs and where a pass of the loop begins, both mixers, the mixture), the names and
shapes of its tensors, sizes that only tensors give, the cache's padded rows and kept pages, and the plain
implementation against itself (the recurrence as a decayed causal sum, kept tokens beside a window, groups by
brute force)."""
import copy

import pytest
import torch

import plain_raranex as P
from raranex_models import SMALL, make_weights, without_ranks, write_model


def spec_of(cfg):
    from lumenllm_b200.config import config_from_dict
    return config_from_dict(cfg).model_spec()


def test_round_trip_and_registry():
    from lumenllm_b200.config import config_from_dict
    from lumenllm_b200.config.raranex import RaranexConfig
    for name, d in SMALL.items():
        c = config_from_dict(d)
        assert isinstance(c, RaranexConfig)
        assert c.to_dict() == d, name
        assert config_from_dict(c.to_dict()) == c
    bare = copy.deepcopy(SMALL["X"])
    del bare["layers"][0]["mlp"]["router"]["groups"]          # one group, of which one is kept
    c = config_from_dict(bare)
    assert c.layers[0].mlp.groups == (1, 1) and config_from_dict(c.to_dict()) == c


def test_order_of_layers_and_where_passes_begin():
    runs = lambda cfg: [(e.layer, e.before_index if e.before is not None else None) for e in spec_of(cfg).schedule]
    for name, cfg in SMALL.items():
        assert runs(cfg) == P.runs(cfg), name
    assert runs(SMALL["X"]) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert runs(SMALL["U"]) == [(0, 0), (1, None)] and not spec_of(SMALL["Y"]).stream_parts
    never = dict(SMALL["X"], loop={"start": 1, "stop": 3, "times": 0})
    assert runs(never) == [(0, None), (3, None)]
    assert all(e.cache_from is None for e in spec_of(SMALL["X"]).schedule)       # every pass its own cache and state


def test_parts_of_the_model_as_data():
    spec = spec_of(SMALL["X"])
    l0, l1, l2 = spec.layers[:3]
    assert (l0.block, sorted(l0.norms)) == ("parallel", ["ffn", "mixer"]) and list(l2.norms) == ["mixer"] and l2.ffn is None
    a = l0.mixer
    assert a.kind == "head_norm_attention" and (a.params["window"], a.params["keep_first"]) == (9, 3)
    assert a.params["qk_norm"] == "unit" and a.params["interleaved_rotation"] and a.params["output_gate"] == "head"
    assert a.params["position"].params["rotary_dim"] == 8
    parts = l1.mixer.params["parts"]
    assert [c["scale"] for c in parts] == [0.5, 0.5]
    assert parts[1]["out_norm"] == {"tensor": "l1.mix.right.out", "eps": 1e-6, "size": 64}
    b, c = parts[0]["mixer"], parts[1]["mixer"]
    assert b.params["query_temperature"] == (0.4, 16.0) and b.params["softcap"] == 6.0 and b.params["position"].kind == "none"
    assert c.kind == "time_mixing" and (c.params["num_heads"], c.params["head_dim"], c.params["decay_rank"]) == (3, 12, 5)
    f = l1.ffn
    assert f.kind == "routed_experts" and f.params["groups"] == {"count": 4, "keep": 2} and f.params["normalize"]
    assert f.params["shared_gate"] and f.params["shared"] == {"size": 16}
    assert spec.stream_parts[0].kind == "loop_input" and spec.head.params["tensor"] == "head"


@pytest.mark.parametrize("name", list(SMALL))
def test_names_and_shapes_of_the_tensors(name):
    from lumenllm_b200.engine.model import expected_tensors
    want = {k: tuple(v.shape) for k, v in make_weights(SMALL[name], 1).items()}
    assert {k: tuple(s) for k, (s, _) in expected_tensors(spec_of(SMALL[name])).items()} == want


def test_a_folder_gives_the_decays_rank(tmp_path):
    from lumenllm_b200.config import ConfigError, config_from_dict, load_config
    folder = write_model(SMALL["Y"], tmp_path / "m", seed=2)
    assert load_config(folder).to_dict() == SMALL["Y"]
    with pytest.raises(ConfigError, match="rank"):
        config_from_dict(without_ranks(SMALL["Y"])).model_spec()


@pytest.mark.parametrize("change, message", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d["layers"][0].update(type="rglru"), "not a mixer"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "at most 16"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda d: d["layers"][1]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(softcap=-1.0), "softcap"),
    (lambda d: d["layers"][1]["mixer"]["right"].pop("dim"), "dim"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "feed-forward"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=5), "choices"),
    (lambda d: d["loop"].update(stop=5), "loop"),
    (lambda d: d["norm"].update(eps=-1.0), "eps"),
])
def test_refusals(change, message):
    from lumenllm_b200.config import ConfigError, config_from_dict
    d = copy.deepcopy(SMALL["X"])
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)


def test_schedules_name_stream_parts_that_exist():
    from dataclasses import replace
    from lumenllm_b200.config import ConfigError
    spec = spec_of(SMALL["X"])
    with pytest.raises(ConfigError, match="stream part"):
        replace(spec, stream_parts=()).validate()


def test_cache_rows_padded_to_tiles_and_kept_pages():
    from lumenllm_b200.cache.kv import LAYOUT_LINEAR, LAYOUT_SW128, PAGE, CacheNeed, KVCache
    need = CacheNeed(2, 20, window=10, v_dim=80, keep_first=PAGE + 3, padded=True)
    for dtype, widths, layout in ((torch.bfloat16, (64, 128), LAYOUT_SW128), (torch.float32, (20, 80), LAYOUT_LINEAR)):
        c = KVCache({0: need}, 6 * PAGE, 2, 6 * PAGE, dtype=dtype)
        grp = c.groups[0]
        assert (grp.k_width, grp.v_width, grp.layout, grp.v_layout) == (*widths, layout, layout)
        assert grp.bytes_per_token(2) == 2 * sum(widths) * 2
    slot = c.alloc_slot()
    c.reserve(slot, 5 * PAGE)
    c.commit(slot, 5 * PAGE)            # the next query sees the last nine keys and the first PAGE + 3
    assert [int(x) != 0 for x in c.groups[0].table[slot]] == [True, True, False, False, True, False]
    c.free_slot(slot)
    c.check()


def test_states_of_time_mixing_begin_on_16_bytes():
    """A sequence's row is the last token's row, then the heads' matrices from a multiple of four numbers on."""
    from lumenllm_b200.parts import Runtime, build_part
    cfg = SMALL["X"]
    spec = spec_of(dict(cfg, width=50)).layers[1].mixer.params["parts"][1]["mixer"]
    part = build_part("mixer", spec, make_weights(dict(cfg, width=50), 1), Runtime(torch.device("cpu"), torch.float32))
    assert part.state_at == 52 and part.state_shape()[0] == (52 + 3 * 12 * 12,) and part.pitch == 36


# ------------------------------------------------------------------ the plain implementation against itself

def test_recurrence_is_a_decayed_causal_sum():
    g = torch.Generator().manual_seed(0)
    T, H, d = 9, 2, 5
    r, k, v = (torch.randn(T, H, d, generator=g, dtype=torch.float64) for _ in range(3))
    w, u = torch.rand(T, H, d, generator=g, dtype=torch.float64), torch.randn(H, d, generator=g, dtype=torch.float64)
    ref = torch.zeros(T, H, d, dtype=torch.float64)
    for t in range(T):
        for s in range(t):
            decay = torch.ones(H, d, dtype=torch.float64)
            for j in range(s + 1, t):
                decay = decay * w[j]
            ref[t] += (r[t] * decay * k[s]).sum(-1, keepdim=True) * v[s]
        ref[t] += (r[t] * u * k[t]).sum(-1, keepdim=True) * v[t]
    torch.testing.assert_close(P.bonus_recurrence(r, k, v, w, u), ref)


def test_visible_keys_by_hand():
    seen = P.visible(8, size=3, keep_first=2)
    assert seen[7].tolist() == [True, True, False, False, False, True, True, True]
    assert seen[2].tolist() == [True, True, True] + [False] * 5 and seen[0].sum() == 1
    assert P.visible(8).sum() == 36 and P.visible(8, size=3)[7].sum() == 3


def test_choices_in_groups_by_brute_force():
    g = torch.Generator().manual_seed(1)
    E, count, keep, top = 12, 4, 2, 3
    s, corr = torch.rand(40, E, generator=g), torch.randn(E, generator=g)
    idx = P.choose(s, corr, top, {"count": count, "keep": keep})
    for t in range(40):
        c = [float(x) for x in s[t] + corr]
        score = [sum(sorted(c[3 * j:3 * j + 3])[-2:]) for j in range(count)]
        best = sorted(range(count), key=lambda j: -score[j])[:keep]
        allowed = [e for j in best for e in range(3 * j, 3 * j + 3)]
        assert sorted(idx[t].tolist()) == sorted(sorted(allowed, key=lambda e: -c[e])[:top])


def test_rotation_keeps_lengths_so_the_unit_norm_may_come_first():
    x = torch.randn(5, 2, 12, dtype=torch.float64)
    pos = torch.arange(5)
    torch.testing.assert_close(P.unit_rms(P.rotate_neighbours(x, pos, 100.0, 8), 1e-5),
                               P.rotate_neighbours(P.unit_rms(x, 1e-5), pos, 100.0, 8))


def test_temperature_steps_at_its_period():
    t = P.temperature(torch.arange(10), 0.5, 4, torch.float64)
    assert torch.equal(t[:3], torch.ones(3, dtype=torch.float64)) and float(t[3]) == pytest.approx(1 + 0.5 * 0.6931471805599453)
    assert t[3] == t[6] < t[7]
