"""Mefatar without a GPU: config.json to typed configuration and back, what is refused, the model's parts
as data (the order of layers with a loop, two mixers side by side with normed outputs, the recurrent unit),
the names and shapes of its tensors, sizes that only tensors give, frequencies stretched by wavelength,
states that share a row, and the plain implementation against itself (both recurrences written as decayed
causal sums; a sink as a key of that score without a value; the convolution against torch's)."""
import copy
import math

import pytest
import torch

import plain_mefatar as P
from mefatar_models import SMALL, make_weights, parallel, right, unit, without_ranks, write_model


def spec_of(cfg):
    from lumenllm_b200.config import config_from_dict
    return config_from_dict(cfg).model_spec()


def test_round_trip_and_registry():
    from lumenllm_b200.config import config_from_dict
    from lumenllm_b200.config.mefatar import MefatarConfig
    for name, d in SMALL.items():
        c = config_from_dict(d)
        assert isinstance(c, MefatarConfig)
        assert c.to_dict() == d, name
        assert config_from_dict(c.to_dict()) == c


def test_order_of_layers():
    order = lambda cfg: [e.layer for e in spec_of(cfg).schedule]
    assert order(SMALL["X"]) == [0, 1, 2, 1, 2, 1, 2, 3] == P.runs(SMALL["X"])
    assert order(SMALL["Y"]) == [0, 1, 2] and order(SMALL["Z"]) == [0, 1, 2, 3, 2, 3] and order(SMALL["V"]) == [0, 0]
    once = dict(SMALL["X"], loop={"start": 1, "stop": 3, "times": 1})
    assert order(once) == [0, 1, 2, 3] == order(dict(SMALL["X"], loop=None))
    assert all(e.cache_from is None for e in spec_of(SMALL["X"]).schedule)       # every pass its own cache and state


def test_parts_of_the_model_as_data():
    spec = spec_of(SMALL["X"])
    l0, l1 = spec.layers[0], spec.layers[1]
    assert l0.mixer.kind == "side_by_side" and l1.mixer.kind == "real_gated_lru" and l1.ffn is None
    assert l0.params["update_factors"] == {"mixer": "l0.ls1", "ffn": "l0.ls2"}
    assert l1.params["update_factors"] == {"mixer": "l1.ls1"}
    parts = l0.mixer.params["parts"]
    assert [c["scale"] for c in parts] == [0.5, 0.5]
    assert parts[1]["out_norm"] == {"tensor": "l0.mix.right.out", "eps": 1e-6, "size": 64}
    a, b = parts[0]["mixer"], parts[1]["mixer"]
    assert a.kind == "wide_norm_attention" and a.params["taps"] == 4 and a.params["sink"] and a.params["output_gate"]
    assert not a.params["bias"] and a.params["interleaved_rotation"]
    assert a.params["position"].params["scaling"] == {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64.0}
    assert b.kind == "gated_linear_attention" and (b.params["tau"], b.params["decay_rank"]) == (8.0, 5)
    assert l0.ffn.kind == "swiglu" and l0.ffn.params["activation"] == "gelu"
    assert spec.head.params["tied_to"] == "embed" and spec.final_norm.params["tensor"] == "final.norm"


@pytest.mark.parametrize("name", list(SMALL))
def test_names_and_shapes_of_the_tensors(name):
    from lumenllm_b200.engine.model import expected_tensors
    want = {k: tuple(v.shape) for k, v in make_weights(SMALL[name], 1).items()}
    assert {k: tuple(s) for k, (s, _) in expected_tensors(spec_of(SMALL[name])).items()} == want


def test_a_folder_gives_the_decays_rank(tmp_path):
    from lumenllm_b200.config import ConfigError, config_from_dict, load_config
    folder = write_model(SMALL["Y"], tmp_path / "m", seed=2)
    cfg = load_config(folder)
    assert cfg.to_dict() == SMALL["Y"]
    with pytest.raises(ConfigError, match="rank"):
        config_from_dict(without_ranks(SMALL["Y"])).model_spec()


@pytest.mark.parametrize("change, message", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d["layers"][0].update(type="attention"), "not a mixer"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "at most 16"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(low=9.0), "low at most high"),
    (lambda d: d["layers"][0]["mixer"]["left"].pop("conv"), "conv"),
    (lambda d: d["layers"][0]["mixer"]["right"].update(tau=0.0), "tau"),
    (lambda d: d["layers"][1]["mixer"].update(blocks=3), "divide"),
    (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "feed-forward"),
    (lambda d: d["loop"].update(stop=5), "loop"),
    (lambda d: d["loop"].update(start=4), "loop"),
    (lambda d: d["norm"].update(eps=-1.0), "eps"),
])
def test_refusals(change, message):
    from lumenllm_b200.config import ConfigError, config_from_dict
    d = copy.deepcopy(SMALL["X"])
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)


def test_frequencies_stretched_by_wavelength():
    """The library's table against the plain one, and the three regions by hand."""
    from lumenllm_b200.config.spec import PartSpec
    from lumenllm_b200.parts import Runtime, build_part
    rt = Runtime(torch.device("cpu"), torch.float32)
    for sc in ((8.0, 1.0, 4.0, 512), (4.0, 2.0, 2.0, 100), (16.0, 1.0, 32.0, 8192)):
        s = dict(zip(("factor", "low", "high", "original"), sc))
        part = build_part("position", PartSpec("rotary", {"head_dim": 48, "rotary_dim": 48, "theta": 1e4,
                                                          "wide_frequencies": True, "scaling": s}), {}, rt)
        assert torch.equal(part.inv_freq, P.frequencies(1e4, 48, s).float())
        assert part.magnitude == 1.0
    s = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}
    plain, f = P.frequencies(1e4, 48), P.frequencies(1e4, 48, s)
    length = 2 * math.pi / plain
    fast, slow = length < 128, length > 512
    between = ~(fast | slow)
    assert fast.any() and slow.any() and between.any()
    assert torch.equal(f[fast], plain[fast]) and torch.equal(f[slow], plain[slow] / 8)
    assert ((f[between] < plain[between]) & (f[between] > plain[between] / 8)).all()


def test_states_of_mixers_side_by_side_share_a_row():
    """The attention's convolution inputs and the linear side's matrices lie one behind the other, each
    from a multiple of four numbers on, and a child's view is its own piece."""
    from lumenllm_b200.parts.side_by_side import _ChildView

    class Entry:
        layout = 7
        store = torch.arange(3 * 40, dtype=torch.float32).view(3, 40)

        def state(self, name="mixer"):
            return self.store if name == "mixer" else name

    v = _ChildView(Entry(), 8, (2, 3, 5))
    assert v.layout == 7 and v.state("block") == "block"
    assert v.state().shape == (3, 2, 3, 5) and float(v.state()[1, 0, 0, 0]) == 48.0
    v.state()[2, 1, 2, 4] = -1.0
    assert float(Entry.store[2, 37]) == -1.0


# ------------------------------------------------------------------ the oracle against itself

def test_plain_gated_linear_attention_is_a_decayed_causal_sum():
    g = torch.Generator().manual_seed(0)
    cfg = SMALL["X"]
    w = {k: v.double() for k, v in make_weights(cfg, 5).items()}
    m, pre, D = cfg["layers"][0]["mixer"]["right"], "l0.mix.right", cfg["width"]
    h = torch.randn(9, D, generator=g, dtype=torch.float64)
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + ".q"].T).view(9, H, d) * d ** -0.5
    k, v = (h @ w[pre + ".k"].T).view(9, H, d), (h @ w[pre + ".v"].T).view(9, H, dv)
    z = h @ w[pre + ".a1"].T @ w[pre + ".a2"].T + w[pre + ".a2.b"]
    log_a = (torch.nn.functional.logsigmoid(z) / m["tau"]).view(9, H, d)
    o = torch.zeros(9, H, dv, dtype=torch.float64)
    for t in range(9):
        for s in range(t + 1):
            decay = torch.exp(log_a[s + 1:t + 1].sum(0))
            o[t] += (q[t] * decay * k[s]).sum(-1, keepdim=True) * v[s]
    o = P.rms_norm(o, w[pre + ".norm"], 1e-6).reshape(9, H * dv) * P.silu(h @ w[pre + ".g"].T)
    assert torch.allclose(o @ w[pre + ".o"].T, P.gated_linear_attention(h, w, pre, m, 1e-6), atol=1e-10)


def test_plain_recurrent_unit_is_a_decayed_causal_sum():
    g = torch.Generator().manual_seed(1)
    cfg = SMALL["X"]
    w = {k: v.double() for k, v in make_weights(cfg, 6).items()}
    m, pre = cfg["layers"][1]["mixer"], "l1.mix"
    h = torch.randn(8, cfg["width"], generator=g, dtype=torch.float64)
    C, B = m["width"], m["blocks"]
    bs = C // B
    u = P.causal_conv(h @ w[pre + ".x"].T + w[pre + ".x.b"], w[pre + ".conv"], w[pre + ".conv.b"])
    dense = lambda n: torch.block_diag(*w[pre + n])
    r = torch.sigmoid(u @ dense(".ra").T + w[pre + ".ra.b"].reshape(-1))
    i = torch.sigmoid(u @ dense(".ri").T + w[pre + ".ri.b"].reshape(-1))
    assert dense(".ra").shape == (C, C) and bs * B == C
    a = torch.exp(-8 * r * torch.nn.functional.softplus(w[pre + ".lam"]))
    x = torch.sqrt(1 - a * a) * i * u
    S = torch.stack([sum(torch.prod(a[s + 1:t + 1], dim=0) * x[s] for s in range(t + 1)) for t in range(8)])
    y = torch.nn.functional.gelu(h @ w[pre + ".y"].T + w[pre + ".y.b"], approximate="tanh")
    assert torch.allclose((S * y) @ w[pre + ".o"].T, P.recurrent_unit(h, w, pre, m), atol=1e-9)


def test_plain_sink_convolution_and_rotation():
    g = torch.Generator().manual_seed(2)
    s, sink = torch.randn(2, 5, 5, generator=g), torch.tensor([0.7, -30.0])
    p = P.sink_softmax(s, sink)
    padded = torch.cat([s.masked_fill(torch.ones(5, 5, dtype=torch.bool).triu(1), float("-inf")),
                        sink[:, None, None].expand(2, 5, 1)], dim=-1)
    assert torch.allclose(p, torch.softmax(padded, dim=-1)[..., :5], atol=1e-6)
    assert float(p[0].sum(-1).max()) < 1.0 and torch.allclose(p[1].sum(-1), torch.ones(5), atol=1e-6)
    u, w, b = torch.randn(7, 3, generator=g), torch.randn(3, 4, generator=g), torch.randn(3, generator=g)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (3, 0)), w[:, None], b, groups=3)[0].T
    assert torch.allclose(P.causal_conv(u, w, b), ref, atol=1e-5)
    x = torch.randn(4, 2, 10, generator=g)
    y = P.rotate_neighbours(x, torch.arange(4), 100.0, 6)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    assert torch.allclose(y[..., :2].norm(dim=-1), x[..., :2].norm(dim=-1), atol=1e-6)
    z = torch.view_as_complex(x[3, :, 2:4].contiguous()) * torch.polar(torch.tensor(1.0), torch.tensor(3 * 100.0 ** (-2 / 6)))
    assert torch.allclose(torch.view_as_real(z), y[3, :, 2:4], atol=1e-5)


def test_what_a_mixer_keeps():
    from lumenllm_b200.parts import part_class
    left_spec, right_spec = (c["mixer"] for c in spec_of(SMALL["X"]).layers[0].mixer.params["parts"])
    t = part_class("mixer", left_spec.kind).tensors(left_spec)
    assert t["l0.mix.left.v.conv"][0] == (2 * 24, 4) and t["l0.mix.left.sink"][0] == (4,)
    assert part_class("mixer", right_spec.kind).tensors(right_spec)["l0.mix.right.a2"][0] == (32, 5)
    assert parallel(1, 2) == {"left": 1, "right": 2} and right(1, 2, 3, 4.0, 5)["tau"] == 4.0 and unit(4, 2, 3)["blocks"] == 2
