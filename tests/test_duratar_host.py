"""Duratar on the host: its configuration and the errors it names, the layout of parts against the tensors the plain implementation
expects, what the cache is asked for (an owner keeps what the layers that read it see), and the sizes read from tensors' shapes."""

from __future__ import annotations

import copy

import numpy as np
import pytest

import plain_duratar as pd
from borrowed_compute_b200.cache.slots import PAGE, GroupPlan, SlotTable
from borrowed_compute_b200.config import ConfigError, DuratarConfig
from borrowed_compute_b200.engine.model import model_for_config
from borrowed_compute_b200.parts import CacheNeed


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_layout_asks_for_exactly_the_tensors_of_the_plain_model(name):
    cfg = pd.SMALL[name]
    _, model = model_for_config(cfg)
    want = {n: s for n, s in model.expected_tensors().items() if not s.optional}
    shapes = pd.tensor_shapes(cfg)
    assert {n: tuple(s.shape) for n, s in want.items()} == {n: tuple(s) for n, s in shapes.items()}
    float32 = (".A_log", ".dt_bias", ".conv", ".ls1", ".ls2", ".in", ".out", ".mix", ".act", ".lq1", ".lk2")
    assert all(want[n].role == "vector" for n in want if n.endswith(float32) or "norm" in n)


def test_every_size_and_constant_comes_from_the_file():
    typed = DuratarConfig.from_dict(pd.SMALL["A"])
    assert (typed.vocab, typed.width, typed.streams, typed.norm_eps) == (131, 72, 3, 1e-5)
    own, delta, reader, light = (layer.mixer for layer in typed.layers)
    assert (own.heads, own.kv_heads, own.dim, own.vdim, own.window, own.keep_first, own.rot_dims, own.rot_base, own.diff, own.kv_from) == \
        (4, 2, 16, 24, 24, 3, 8, 500.0, 0.5, None)
    assert (own.rot_scaling.factor, own.rot_scaling.low, own.rot_scaling.high, own.rot_scaling.original) == (3.0, 1.0, 4.0, 60)
    assert (reader.window, reader.keep_first, reader.diff, reader.kv_from) == (50, 5, 0.3, 0)
    assert (delta.heads, delta.kv_heads, delta.dim, delta.vdim, delta.taps, delta.decay_rank, delta.gate_rank) == (4, 2, 12, 20, 4, 8, 16)
    assert (light.heads, light.dim, light.vdim) == (3, 16, 12) and light.decay == tuple(pd.SMALL["A"]["layers"][3]["mixer"]["decay"])
    assert [layer.ff for layer in typed.layers] == [40, 56, 0, 40]
    b = DuratarConfig.from_dict(pd.SMALL["B"])
    assert b.streams == 1 and b.layers[1].mixer.window == 0 and b.layers[1].mixer.rot_dims == 0 and b.layers[2].mixer.taps == 1


def test_the_ranks_of_the_low_rank_projections_come_from_the_tensors():
    cfg = copy.deepcopy(pd.SMALL["A"])
    for layer in cfg["layers"]:
        layer["mixer"].pop("decay_rank", None), layer["mixer"].pop("gate_rank", None)
    with pytest.raises(ConfigError, match="decay_rank"):
        model_for_config(cfg)
    typed, _ = model_for_config(cfg, pd.tensor_shapes(pd.SMALL["A"]))
    assert (typed.layers[1].mixer.decay_rank, typed.layers[1].mixer.gate_rank) == (8, 16)


def broken(change):
    cfg = copy.deepcopy(pd.SMALL["A"])
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,names", [
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.pop("norm"), "norm.eps"),
    (lambda c: c["layers"][0].update(type="convolution"), "layers[0].type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "layers[0].mixer.heads"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "layers[0].mixer.diff"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "layers[0].mixer.rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("high"), "layers[0].mixer.rot.scaling.high"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(high=1.0), "layers[0].mixer.rot.scaling.high"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "layers[0].mixer.mask.keep_first"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "layers[2].mixer.kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "layers[2].mixer.kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=32), "layers[2].mixer.kv_from"),
    (lambda c: c["layers"][3]["mixer"]["decay"].pop(), "layers[3].mixer.decay"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "layers[1].mixer.conv"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "layers[0].mlp.kind"),
])
def test_a_wrong_configuration_is_refused_with_the_key_named(change, names):
    with pytest.raises(ConfigError) as e:
        DuratarConfig.from_dict(broken(change))
    assert names in str(e.value)


def test_what_the_cache_is_asked_for():
    _, model = model_for_config(pd.SMALL["A"])
    needs, states, memory_of = model.memory_needs()
    assert memory_of == [None, None, 0, None]
    # two key maps a kv head, one set of values; the owner keeps the wider window and the more of the first positions
    assert needs[0].planes == ((4, 16), (2, 24)) and (needs[0].window, needs[0].keep_first) == (50, 5)
    assert states[1].shape == (4, 20, 12) and states[3].shape == (3, 12, 16) and states[0] is states[2] is None
    more = model.more_state_needs()
    assert more[1]["mixer.conv"].shape == (3, 2 * 2 * 12 + 4 * 20) and more[0] == more[2] == more[3] == {}
    _, b = model_for_config(pd.SMALL["B"])
    assert b.memory_needs()[0][1].window == 0          # the owner sees everything, its reader's window does not narrow that


@pytest.mark.parametrize("a,b,want", [((24, 3), (50, 5), (50, 5)), ((50, 5), (24, 70), (50, 70)), ((0, 0), (9, 4), (0, 4)), ((9, 4), (0, 0), (0, 4))])
def test_a_need_widened_by_another(a, b, want):
    planes = ((2, 8), (1, 16))
    w = CacheNeed(planes, a[0], keep_first=a[1]).widened(CacheNeed(planes, b[0], keep_first=b[1]))
    assert (w.window, w.keep_first, w.planes) == (*want, planes)
    with pytest.raises(ValueError, match="cannot read planes"):
        CacheNeed(planes).widened(CacheNeed(((2, 8),)))


def test_pages_a_reader_with_a_wider_window_sees_are_kept():
    _, model = model_for_config(pd.SMALL["C"])
    need = model.memory_needs()[0][0]
    assert need.window == 0                             # layer 1 reads layer 0's keys without a window
    need = CacheNeed(need.planes, 24, keep_first=3).widened(CacheNeed(need.planes, 150, keep_first=66))
    table = SlotTable(1, 64, 20 * PAGE, [GroupPlan(need.window, need.chunk, need.keep_first)])
    s = table.acquire()
    for n in range(1, 700):
        table.reserve(s, n, rows=1)
        table.commit(s, n)
        held = {i for i, p in enumerate(table.tables[0][s]) if p >= 0}
        seen = {j // PAGE for j in range(n) if (n - 1) - j < 150 or j < 66}
        assert seen <= held, n
    table.check()


def test_a_bundle_of_streams_goes_with_its_blocks_only():
    from borrowed_compute_b200.engine.model import DecoderModel
    from dataclasses import replace

    spec = model_for_config(pd.SMALL["A"])[1].spec
    with pytest.raises(ValueError, match="bundle of streams"):
        DecoderModel(replace(spec, streams=0))


def test_plain_mechanisms_on_numbers_worked_by_hand():
    # two streams: a swap with half of the result on the second
    X = np.array([[[1.0, 2.0]], [[3.0, 5.0]]])
    out = pd.spread(X, np.array([[10.0, 20.0]]), np.array([[0.0, 1.0], [1.0, 0.0]]), [0.0, 0.5])
    assert out[0].tolist() == [[3.0, 5.0]] and out[1].tolist() == [[6.0, 12.0]]
    assert pd.collapse(X, [2.0, -1.0]).tolist() == [[-1.0, -1.0]]
    # visibility: a window of 2 that keeps the first position
    assert pd.visible(4, {"size": 2, "keep_first": 1}).astype(int).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [1, 1, 1, 0], [1, 0, 1, 1]]
    # the delta rule on one head of one channel: S = 0.5; decay to 0.25, r = 0.5 (3 - 0.25 * 2), S = 0.25 + 2 r, o = S * 1
    o, S = pd.delta_scan(np.full((1, 1, 1), 1.0), np.full((1, 1, 1), 2.0), np.full((1, 1, 1), 3.0), np.full((1, 1, 1), 0.5), np.full((1, 1), 0.5),
                         np.full((1, 1, 1), 0.5))
    assert np.isclose(S[0, 0, 0], 2.75) and np.isclose(o[0, 0, 0], 2.75)
    # xIELU: continuous with slope 1/2 at zero, softplus(0) = ln 2
    z = np.array([-1e-9, 0.0, 1e-9, 2.0, -1.0])
    y = pd.xielu(z, (0.0, 0.0))
    assert np.allclose(y[:3], 0.5 * z[:3], atol=1e-15) and np.isclose(y[3], np.log(2.0) * 4 + 1.0)
    assert np.isclose(y[4], (0.5 + np.log(2.0)) * (np.exp(-1.0) - 1.0 + 1.0) - 0.5)
