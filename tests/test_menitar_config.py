"""The Menitar decoder as far as it goes without a GPU: configuration, tensors,
schedule, the pages of runs of positions, the plain implementation's pieces."""
import copy
import math

import pytest
import torch

import plain_menitar as pm
from menitar_cases import CASE_A, CASE_B, CASE_C, CASES, make_folder, random_case


def spec_of(cfg):
    from infernum_b200.weights.random_init import model_specs_for
    return model_specs_for(cfg)


def test_every_size_and_constant_comes_from_the_configuration():
    cfg, spec, weights = spec_of(CASE_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.logit_scale) == (211, 96, 1e-5, 4.0, 1.5)
    assert cfg.loop == (1, 3, 3)
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.chunk, m.rot_dims, m.rot_base) == (4, 2, 16, 24, 0.3, 21, 8, 10000.0)
    assert (cfg.layers[0].mlp.ff, cfg.layers[0].mlp.limit) == (176, 0.8)
    assert cfg.layers[2].mlp is None and cfg.layers[2].mixer.chunk == 0 and cfg.layers[2].mixer.rot_dims == 0
    assert tuple(weights["loop.step"].shape) == (3, 96)
    assert tuple(weights["l0.mix.q.norm"].shape) == (64,) and tuple(weights["l0.mix.k.norm"].shape) == (32,)
    assert tuple(weights["l0.mix.talk"].shape) == (4, 4) and tuple(weights["l0.mix.temp"].shape) == (4,)
    assert tuple(weights["l0.mix.g"].shape) == (4, 96) and tuple(weights["l0.mix.o"].shape) == (96, 96)
    assert tuple(weights["l0.mix.v"].shape) == (48, 96)
    assert weights["l2.norm2"].optional and not weights["l0.norm2"].optional
    assert "l2.mlp.gate" not in weights and "head" not in weights
    assert spec.lm_head.params["tied_to"] == "embed"


def test_what_a_configuration_leaves_out():
    cfg, spec, weights = spec_of(CASE_B)
    assert cfg.embedding_scale == 1.0 and cfg.logit_scale == 1.0 and cfg.loop is None
    assert cfg.layers[0].mixer.scale == pytest.approx(10 ** -0.5)
    assert (cfg.layers[1].mixer.kv_heads, cfg.layers[1].mixer.vdim, cfg.layers[1].mixer.chunk) == (2, 14, 0)
    assert cfg.layers[0].mlp.limit is None
    assert "loop.step" not in weights and spec.pass_entry is None


def test_schedule_of_looped_layers():
    _, spec, _ = spec_of(CASE_A)
    assert [(s.layer, s.enter) for s in spec.schedule] == \
        [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert [(i, e) for i, e in pm.run_order(CASE_A)] == [(s.layer, s.enter) for s in spec.schedule]
    _, spec, _ = spec_of(CASE_C)
    assert [(s.layer, s.enter) for s in spec.schedule] == [(0, 0), (1, None), (2, None), (0, 1), (1, None), (2, None)]


@pytest.mark.parametrize("change, message", [
    (lambda c: c.pop("vocab"), "vocab"), (lambda c: c.pop("width"), "width"), (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["norm"].pop("eps"), "eps"), (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="conv"), "conv"), (lambda c: c["layers"][0]["mixer"].pop("heads"), "heads"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "dim"), (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe"), (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=1), "loop"), (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "times"), (lambda c: c.update(layers={"a": 1}), "layers"),
])
def test_refused_configurations(change, message):
    from infernum_b200.config.menitar import MenitarConfig
    from infernum_b200.errors import ConfigError
    cfg = copy.deepcopy(CASE_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        MenitarConfig.from_dict(cfg)
    assert message in str(e.value)


def test_registry_knows_the_design():
    from infernum_b200.registry import resolve_config, supported_architectures
    assert "Menitar" in supported_architectures()
    arch, cfg = resolve_config(CASE_A)
    assert arch.name == "Menitar" and cfg.architecture == "Menitar"


@pytest.mark.parametrize("name", list(CASES))
def test_cases_and_random_cases_describe_models(name):
    spec_of(CASES[name])
    for seed in range(20):
        _, spec, _ = spec_of(random_case(seed * 4 + ord(name)))
        assert spec.layers


def test_a_second_norm_without_a_feed_forward_may_be_there_or_not(tmp_path):
    from infernum_b200.errors import WeightError
    from infernum_b200.weights.loader import check_against_specs
    from infernum_b200.weights.safetensors_io import open_model_folder
    _, _, weights = spec_of(CASE_A)
    with_norm = make_folder(str(tmp_path / "a"), CASE_A, seed=1)
    without = make_folder(str(tmp_path / "b"), CASE_A, seed=1, drop=["l2.norm2"])
    for folder in (with_norm, without):
        check_against_specs(weights, open_model_folder(folder))
    with pytest.raises(WeightError):
        check_against_specs(weights, open_model_folder(make_folder(str(tmp_path / "c"), CASE_A, seed=1, drop=["l0.norm2"])))
    with pytest.raises(WeightError):
        check_against_specs(weights, open_model_folder(make_folder(str(tmp_path / "d"), CASE_A, seed=1, add={"l2.extra": (3,)})))


# ---- pages of runs of positions -------------------------------------------------------
class Need:
    def __init__(self, position, paged):
        self.position, self.paged, self.state, self.cache_of, self.block_state = position, paged, None, None, None


def manager(chunk, page_size=4, pages=64, window=0):
    from infernum_b200.cache import CacheManager
    from infernum_b200.parts.base import PagedCacheSpec
    return CacheManager([Need(0, PagedCacheSpec(2, 8, window, v_head_dim=16, chunk=chunk)), Need(1, PagedCacheSpec(2, 8))],
                        page_size=page_size, num_pages=pages, max_requests=2)


@pytest.mark.parametrize("chunk,page_size", [(10, 4), (8, 4), (3, 4), (1, 2), (16, 16), (21, 8)])
def test_pages_of_earlier_runs_are_given_back_and_no_sooner(chunk, page_size):
    m = manager(chunk, page_size)
    rc = m.admit("a")
    fed = 0
    for n in [1, 2, 5, 1, 1, 7, 3, 1, 11, 2, 1, 1, 1, 4]:
        m.extend(rc, n)
        # what the step's queries read is held: everything from the first query's run on
        first = fed // chunk * chunk
        for pos in range(first, fed + n):
            assert rc.tables[0][pos // page_size] >= 0
        m.commit(rc, n)
        fed += n
        keep_from = fed // chunk * chunk
        for b, page in enumerate(rc.tables[0]):
            gone = (b + 1) * page_size <= keep_from
            assert (page < 0) == gone, (fed, b)
        assert all(page >= 0 for page in rc.tables[1])  # the other group keeps everything
        m.check_invariants()
    m.release(rc)
    m.check_invariants()
    assert m.free_pages() == [64, 64]


def test_most_pages_a_request_holds_with_runs_of_positions():
    m = manager(10, 4)
    for step in (1, 3, 8):
        rc = m.admit("a")
        peak, fed = 0, 0
        while fed < 120:
            m.extend(rc, step)
            peak = max(peak, sum(p >= 0 for p in rc.tables[0]))
            m.commit(rc, step)
            fed += step
        assert peak <= m.peak_pages(120, step)[0] < m.peak_pages(120, step)[1]
        m.release(rc)
    both = manager(10, 4, window=3)
    rc = both.admit("a")
    both.extend(rc, 30)
    both.commit(rc, 30)  # the run begins at 30, the window at 28: the later counts
    assert [p >= 0 for p in rc.tables[0]] == [False] * 7 + [True]


# ---- the plain implementation's pieces, by hand ----------------------------------------
def test_plain_visibility():
    see = pm.visible(7, 3)
    assert see.tolist() == [[j <= i and j // 3 == i // 3 for j in range(7)] for i in range(7)]
    assert pm.visible(4, None).tolist() == [[j <= i for j in range(4)] for i in range(4)]


def test_plain_scores_are_exchanged_over_all_heads():
    T, H, G, d = 3, 4, 2, 5
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(T, H, d, generator=g).double(), torch.randn(T, G, d, generator=g).double()
    temp, talk = torch.rand(H, generator=g).double(), torch.randn(H, H, generator=g).double()
    s = pm.mixed_scores(q, k, 0.3, temp, talk)
    for h in range(H):
        for i in range(T):
            for j in range(T):
                want = sum(float(talk[h, a]) * float(temp[a]) * 0.3 * float(q[i, a] @ k[j, a // 2]) for a in range(H))
                assert float(s[h, i, j]) == pytest.approx(want, rel=1e-12)


def test_plain_rotation_norm_and_activation():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=torch.float64)
    y = pm.rotate_half(x, torch.tensor([3]), 4, 100.0)[0, 0]
    a, b = 3.0, 3.0 * 100.0 ** -0.5
    want = [1 * math.cos(a) - 3 * math.sin(a), 2 * math.cos(b) - 4 * math.sin(b),
            3 * math.cos(a) + 1 * math.sin(a), 4 * math.cos(b) + 2 * math.sin(b), 5.0]
    assert torch.allclose(y, torch.tensor(want, dtype=torch.float64))
    n = pm.rms_norm(torch.tensor([[3.0, 4.0]], dtype=torch.float64), torch.tensor([1.0, 2.0], dtype=torch.float64), 0.5)
    assert torch.allclose(n, torch.tensor([[3.0, 8.0]], dtype=torch.float64) / math.sqrt(13.0))
    one = torch.ones(1, 1, dtype=torch.float64)
    for gate, up, limit, want in [(3.0, -9.0, 2.0, 2 / (1 + math.exp(-3.404)) * -1.0),
                                  (-5.0, 0.5, 2.0, -5 / (1 + math.exp(8.51)) * 1.5),
                                  (3.0, 9.0, None, 3 / (1 + math.exp(-5.106)) * 10.0)]:
        w = {"gate": one * gate, "up": one * up, "down": one}
        assert float(pm.clamped_gated(one, {"limit": limit}, w, "")) == pytest.approx(want, rel=1e-9)


# ---- the host's part of the tensor-core attention ---------------------------------------
def test_slices_of_the_keys():
    from infernum_b200.ops.attention_talk import choose_splits, key_span
    for rows, entries, kv, chunk, window in [(1, 1, 1000, 512, 0), (1, 8, 5000, 0, 0), (5, 3, 700, 100, 0), (8, 1, 900, 300, 64)]:
        span = key_span(kv, rows, chunk, window, 32)
        splits, slice_len = choose_splits(rows, entries, 1, span, 32, 148)
        assert splits == 1 or (slice_len % 32 == 0 and splits * slice_len >= span > (splits - 1) * slice_len)
        # every key from the first of a row tile's run, rounded down, to its last row lies in a slice
        for last in range(0, kv, 7):
            first_row = max(0, last - min(rows, 8) + 1)
            lo = first_row // chunk * chunk if chunk else 0
            lo = max(lo, first_row - window + 1) if window else lo
            assert last - lo // 32 * 32 + 1 <= span
    assert choose_splits(2048, 1, 1, 1100, 16, 148) == (1, 0)      # row tiles enough
    assert choose_splits(1, 1, 1, 60, 32, 148) == (1, 0)           # few keys
    assert choose_splits(1, 1, 1, 1100, 16, 148)[0] > 16


def test_sizes_with_a_tensor_core_variant():
    from infernum_b200.ops.attention_talk import layout, queries_of_few, supported
    assert supported(16, 4, 64, 64) and supported(32, 8, 128, 128) and supported(5, 5, 64, 16) and supported(1, 1, 16, 256)
    assert not supported(4, 2, 24, 32) and not supported(4, 2, 32, 40) and not supported(64, 64, 128, 128)
    for h, g, d, e in [(16, 4, 64, 64), (12, 4, 16, 32), (10, 1, 16, 80), (32, 8, 128, 128)]:
        for queries in (8, queries_of_few(h, g)):
            bn, blocks, smem, fits = layout(h, g, d, e, queries)
            assert fits and bn in (16, 32) and e % (blocks * 16) == 0 and smem <= 227 * 1024
    assert [queries_of_few(h, g) for h, g in ((32, 8), (8, 8), (16, 1), (12, 4))] == [2, 8, 1, 2]
