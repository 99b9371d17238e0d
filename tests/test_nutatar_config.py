"""The Nutatar decoder as far as it goes without a GPU: configuration, tensors,
schedule and caches, the plain implementation's pieces by hand."""
import copy
import math

import pytest
import torch

import plain_nutatar as pn
from nutatar_cases import CASE_A, CASE_B, CASE_C, CASE_D, CASES, make_folder, margin, random_case


def spec_of(cfg):
    from infernum_b200.weights.random_init import model_specs_for
    return model_specs_for(cfg)


def test_every_size_and_constant_comes_from_the_configuration():
    cfg, spec, weights = spec_of(CASE_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale) == (211, 96, 1e-5, 3.0)
    assert spec.embedding.params["scale"] == 3.0
    m = cfg.layers[0].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.kv_from) == (4, 12, 6, 20, 28, 24, 0.3, None)
    assert (m.rot.dims, m.rot.base, m.rot.scaling.factor, m.rot.scaling.original, m.rot.scaling.fast, m.rot.scaling.slow) == \
        (6, 5000.0, 4.0, 64.0, 8.0, 1.0)
    m = cfg.layers[1].mixer
    assert (m.heads, m.kv_heads, m.dim, m.scale, m.window, m.rot_dims, m.rot_base) == (6, 3, 20, 0.25, 21, 8, 10000.0)
    f = cfg.layers[1].mlp
    assert (f.ff, f.limit, f.experts, f.top, f.group_count, f.group_keep, f.shared_ff, f.shared_limit) == \
        (24, 0.9, 6, 2, 3, 2, 40, 1.3)
    m = cfg.layers[3].mixer
    assert (m.heads, m.dim, m.vdim, m.tau) == (3, 12, 20, 4.0)
    shapes = {n: tuple(w.shape) for n, w in weights.items()}
    assert shapes["l0.mix.uq"] == (72, 28) and shapes["l0.mix.dkv"] == (30, 96) and shapes["l0.mix.uk"] == (48, 24)
    assert shapes["l0.mix.uv"] == (80, 24) and shapes["l0.mix.sink"] == (4,) and shapes["l0.mix.g"] == (4, 96)
    assert shapes["l1.mix.q.norm"] == (120,) and shapes["l1.mix.k.norm"] == (60,) and shapes["l1.mix.o"] == (96, 120)
    assert "l1.mix.v" not in weights and "l2.mix.dkv" not in weights and "l2.mix.dkv.norm" not in weights
    assert shapes["l3.mix.a1"] == (-1, 96) and shapes["l3.mix.a2"] == (36, -1) and shapes["l3.mix.a2.b"] == (36,)
    assert shapes["l3.mix.norm"] == (20,) and shapes["l3.mix.o"] == (96, 60)
    assert shapes["l0.mlp.up"] == (176, 96) and "l0.mlp.gate" not in weights
    assert shapes["l1.mlp.router"] == (6, 96) and shapes["l1.mlp.shared.gate"] == (40, 96) and "l1.mlp.router.b" not in weights
    assert weights["l2.norm2"].optional and not weights["l0.norm2"].optional
    assert shapes["head"] == (211, 96)


def test_what_a_configuration_leaves_out():
    cfg, _, weights = spec_of(CASE_B)
    assert cfg.embedding_scale == 1.0
    assert (cfg.layers[0].mixer.vdim, cfg.layers[0].mixer.tau) == (5, 1.0)
    f = cfg.layers[0].mlp
    assert (f.limit, f.group_count, f.group_keep, f.shared_ff) == (None, 1, 1, 0)
    m = cfg.layers[1].mixer
    assert m.scale == pytest.approx(10 ** -0.5) and m.rot_dims == 0 and m.window == 7
    assert (cfg.layers[2].mixer.kv_heads, cfg.layers[2].mixer.window) == (2, 0)
    m = cfg.layers[4].mixer
    assert m.scale == pytest.approx(14 ** -0.5) and m.rot.scaling is None
    assert cfg.layers[5].mlp.shared_limit is None and cfg.layers[5].mlp.limit is None
    assert "l0.mlp.shared.gate" not in weights


def test_schedule_and_caches():
    """Readers name the layer whose cache they read; recurrent layers have a state and no pages."""
    from infernum_b200.models.model import Model
    from infernum_b200.parts.base import Runtime
    _, spec, _ = spec_of(CASE_D)
    assert [s.cache_of for s in spec.schedule] == [None, None, 0, None, None, 1]
    needs = Model(spec, Runtime(torch.device("cpu"), torch.float32)).cache_needs()
    assert [(n.paged is not None, n.state is not None) for n in needs] == \
        [(True, False)] * 3 + [(False, True)] + [(True, False)] * 2
    assert needs[3].state.shape == (2 * 64 * 128,) and needs[3].state.dtype == torch.float32
    assert (needs[0].paged.head_dim, needs[0].paged.value_dim, needs[0].paged.window) == (96, 0, 0)
    assert (needs[4].paged.kv_heads, needs[4].paged.head_dim, needs[4].paged.window) == (1, 128, 128)
    assert Model(spec, Runtime(torch.device("cpu"), torch.float32)).replayable


@pytest.mark.parametrize("change, message", [
    (lambda c: c.pop("vocab"), "vocab"), (lambda c: c.pop("width"), "width"), (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["norm"].pop("eps"), "eps"), (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="conv"), "conv"), (lambda c: c["layers"][0]["mixer"].pop("heads"), "heads"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"), (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "vdim"), (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=22), "at most"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier"), (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "earlier"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "keeps no cache"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=16), "differs"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=7.0), "differs"),
    (lambda c: c["layers"][3]["mixer"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "gated"), (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "choices"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=-1.0), "negative"), (lambda c: c.update(layers={"a": 1}), "layers"),
])
def test_refused_configurations(change, message):
    from infernum_b200.config.nutatar import NutatarConfig
    from infernum_b200.errors import ConfigError
    cfg = copy.deepcopy(CASE_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        NutatarConfig.from_dict(cfg)
    assert message in str(e.value)


def test_registry_knows_the_design():
    from infernum_b200.registry import resolve_config, supported_architectures
    assert "Nutatar" in supported_architectures()
    arch, cfg = resolve_config(CASE_A)
    assert arch.name == "Nutatar" and cfg.architecture == "Nutatar"


def test_a_checkpoint_may_bring_the_norm_of_a_layer_without_a_feed_forward(tmp_path):
    from infernum_b200.errors import WeightError
    from infernum_b200.weights.loader import load_tensors
    for drop in ([], ["l2.norm2"]):
        folder = make_folder(str(tmp_path / f"m{len(drop)}"), CASE_A, 3, drop=drop)
        _, _, specs = spec_of(CASE_A)
        got = load_tensors(folder, specs, torch.float32, "cpu")
        assert ("l2.norm2" in got) == (not drop)
    folder = make_folder(str(tmp_path / "bad"), CASE_A, 3, drop=["l0.norm2"], add={"l1.mix.v": (60, 96)})
    with pytest.raises(WeightError) as e:
        load_tensors(folder, specs, torch.float32, "cpu")
    assert "l0.norm2" in str(e.value) and "l1.mix.v" in str(e.value)


def test_parts_refuse_what_they_cannot_do():
    from infernum_b200.errors import ConfigError
    from infernum_b200.parts import FEED_FORWARDS, MIXERS
    from infernum_b200.parts.base import Runtime
    rt = Runtime(torch.device("cpu"), torch.float32)
    base = {"hidden_size": 16, "num_heads": 2, "head_dim": 8}
    with pytest.raises(ConfigError, match="over"):
        MIXERS.get("attention")({**base, "qk_norm": {"q": "a", "k": "b", "eps": 1e-6, "over": "row"}}, rt)
    with pytest.raises(ConfigError, match="position"):
        MIXERS.get("attention")({**base, "value_from_key": True, "position": {"kind": "rotary", "params": {
            "head_dim": 8, "theta": 10.0}}}, rt)
    with pytest.raises(ConfigError, match="sink"):
        MIXERS.get("attention")({**base, "sink": "s", "sink_logit": 0.0}, rt)
    with pytest.raises(ConfigError, match="tau"):
        MIXERS.get("gla")({**base, "eps": 1e-6, "tau": 0.0}, rt)
    with pytest.raises(ConfigError, match="activation"):
        FEED_FORWARDS.get("mlp")({"hidden_size": 8, "intermediate_size": 8, "activation": "relu3"}, rt)
    moe = {"hidden_size": 8, "expert_size": 8, "experts": 6, "top": 2, "scoring": "softmax_all", "groups": {"count": 3, "keep": 2}}
    with pytest.raises(ConfigError, match="groups"):
        FEED_FORWARDS.get("moe")({**moe, "identity": 1}, rt)
    assert FEED_FORWARDS.get("moe")(moe, rt).renormalize and not FEED_FORWARDS.get("moe")({**moe, "renormalize": False}, rt).renormalize


def test_ramp_frequencies_agree():
    from infernum_b200.parts.rope import rotary_inv_freq, rotary_magnitude
    for dims, base, s in ((16, 500.0, (4.0, 512, 32.0, 1.0)), (6, 5000.0, (2.0, 64, 8.0, 1.0)), (64, 1e5, (8.0, 4096, 16.0, 2.0)),
                          (4, 100.0, (1.0, 16, 2.0, 2.0)), (2, 10.0, (3.0, 7, 1.0, 1.0))):
        scaling = dict(zip(("factor", "original", "fast", "slow"), s))
        f, mag = pn.ramp_frequencies(dims, base, scaling)
        assert rotary_inv_freq(dims, base, {**scaling, "rope_type": "ramp"}) == pytest.approx(f, rel=1e-12)
        assert rotary_magnitude({**scaling, "rope_type": "ramp"}) == pytest.approx(mag)
        assert rotary_inv_freq(dims, base, None) == pytest.approx(pn.ramp_frequencies(dims, base, None)[0])


# ---- the plain implementation's pieces, by hand ----------------------------------------
def test_plain_softmaxes_and_windows():
    see = pn.visible(6, 3)
    assert see.tolist() == [[0 <= i - j < 3 for j in range(6)] for i in range(6)]
    assert pn.visible(4, None).tolist() == [[j <= i for j in range(4)] for i in range(4)]
    s = torch.tensor([[0.3, -2.0, 5.0]] * 3, dtype=torch.float64)
    for sink in (0.0, 3.0, -50.0):
        p = pn.softmax_beside(s, pn.visible(3, 2), sink)
        e = [math.exp(v) for v in (0.3, -2.0, 5.0)]
        assert float(p[0, 0]) == pytest.approx(e[0] / (e[0] + math.exp(sink)))
        assert float(p[2, 1]) == pytest.approx(e[1] / (e[1] + e[2] + math.exp(sink))) and float(p[2, 0]) == 0.0
    tiny = pn.softmax_beside(s - 800.0, pn.visible(3, None), 0.0)
    assert float(tiny.sum()) == 0.0 and bool(torch.isfinite(tiny).all())


def test_plain_rotations():
    x = torch.zeros(4, 1, 5, dtype=torch.float64)
    x[3, 0] = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0])
    a, b = 3.0, 3.0 * 100.0 ** -0.5
    half = pn.rotate_half(x, 4, 100.0)[3, 0]
    near = pn.rotate_neighbours(x, 4, 100.0, None)[3, 0]
    c = math.cos
    s = math.sin
    assert half.tolist() == pytest.approx([c(a) - 3 * s(a), 2 * c(b) - 4 * s(b), 3 * c(a) + s(a), 4 * c(b) + 2 * s(b), 5.0])
    assert near.tolist() == pytest.approx([c(a) - 2 * s(a), 2 * c(a) + s(a), 3 * c(b) - 4 * s(b), 4 * c(b) + 3 * s(b), 5.0])
    grown = pn.rotate_neighbours(x, 4, 100.0, {"factor": math.e, "original": 1e-9, "fast": 1.0, "slow": 1.0})[3, 0]
    assert float((grown[:4] ** 2).sum()) == pytest.approx(1.1 ** 2 * 30.0) and float(grown[4]) == 5.0


def test_plain_recurrence_and_decays():
    w = {"a1": torch.eye(1).double(), "a2": torch.tensor([[1.0], [2.0]]).double(), "a2.b": torch.tensor([0.5, -1.0]).double()}
    a = pn.decays(torch.tensor([[0.3]], dtype=torch.float64), 4.0, w, "")[0]
    assert a.tolist() == pytest.approx([(1 / (1 + math.exp(-0.8))) ** 0.25, (1 / (1 + math.exp(0.4))) ** 0.25])
    q, k = torch.tensor([[1.0, 2.0], [3.0, 1.0]]).double(), torch.tensor([[0.5, 1.0], [2.0, -1.0]]).double()
    v, al = torch.tensor([[2.0], [3.0]]).double(), torch.tensor([[0.1, 0.2], [0.5, 0.25]]).double()
    o = pn.decayed_state(q, k, v, al)
    assert o[:, 0].tolist() == pytest.approx([1 * 1.0 + 2 * 2.0, 3 * (0.5 * 1.0 + 6.0) + (0.25 * 2.0 - 3.0)])


def test_plain_feed_forwards_and_routing():
    one = torch.ones(1, 1, dtype=torch.float64)
    assert [float(pn.squared_relu(one * v, {"up": one, "down": one}, "")) for v in (3.0, -3.0)] == [9.0, 0.0]
    for gate, up, limit, want in [(3.0, -9.0, 2.0, 2 / (1 + math.exp(-3.404)) * -1.0),
                                  (-5.0, 0.5, 2.0, -5 / (1 + math.exp(8.51)) * 1.5),
                                  (3.0, 9.0, None, 3 / (1 + math.exp(-5.106)) * 10.0)]:
        w = {"gate": one * gate, "up": one * up, "down": one}
        assert float(pn.expert(one, limit, w, "")) == pytest.approx(want, rel=1e-9)
    z = torch.tensor([3.0, -9.0, 2.0, 2.5, 2.0, 2.0], dtype=torch.float64)
    e = torch.exp(z)
    got = pn.route(z, 2, 3, 2)  # groups (0, 1), (2, 3), (4, 5): the first two by their best
    assert [i for i, _ in got] == [0, 3] and float(got[1][1]) == pytest.approx(float(e[3] / e.sum()))
    assert [i for i, _ in pn.route(z, 3, 1, 1)] == [0, 3, 2] and margin(z, 2, 3, 2) == pytest.approx(0.5)
    assert [i for i, _ in pn.route(torch.zeros(4).double(), 2, 2, 1)] == [0, 1]


def test_configurations_drawn_at_random_are_valid(tmp_path):
    kinds = set()
    for seed in range(40):
        cfg, spec, _ = spec_of(random_case(seed))
        kinds |= {layer.type for layer in cfg.layers}
    assert kinds == {"attention", "gla", "latent_attention"}
    assert len(CASES) == 4 and CASE_C["layers"][3]["mixer"]["kv_from"] == 2


def test_steady_models_choose_far_from_close_calls(tmp_path):
    folder = make_folder(str(tmp_path / "m"), CASE_A, 4, steady=True)
    w = pn.read_weights(folder)
    x = w["embed"] * CASE_A["embedding"]["scale"]
    z = x @ w["l1.mlp.router"].T
    assert min(margin(row, 2, 3, 2) for row in z) > 0.02
    assert float(w["l0.norm1"][:12].abs().max()) == 0.0
