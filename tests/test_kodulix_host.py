"""Kodulix on the host: its configuration and the errors it names, the layout of parts against the tensors the plain implementation
expects, what the cache is asked for, the buckets of distances and their table, and which blocks hand the stream over."""

from __future__ import annotations

import copy
import math

import numpy as np
import pytest

import plain_kodulix as pk
from borrowed_compute_b200.cache import PagedCache
from borrowed_compute_b200.config import ConfigError, KodulixConfig
from borrowed_compute_b200.config.kodulix import complete_from_shapes
from borrowed_compute_b200.engine.model import model_for_config

torch = pytest.importorskip("torch")


@pytest.mark.parametrize("name", ["A", "B"])
def test_the_layout_asks_for_exactly_the_tensors_of_the_plain_model(name):
    cfg = pk.SMALL[name]
    _, model = model_for_config(cfg)
    want = {n: s for n, s in model.expected_tensors().items() if not s.optional}
    assert {n: tuple(s.shape) for n, s in want.items()} == {n: tuple(s) for n, s in pk.tensor_shapes(cfg).items()}
    assert all(want[n].role == "vector" for n in want if n.endswith((".rel", ".router", ".correction")) or "norm" in n)


def test_every_size_and_constant_comes_from_the_file():
    typed = KodulixConfig.from_dict(pk.SMALL["A"])
    assert (typed.vocab, typed.width, typed.norm_eps, typed.residual_mult, typed.logit_scale) == (150, 64, 1e-5, 0.6, 0.5)
    assert (typed.bigram.buckets, typed.bigram.mul_prev, typed.bigram.mul_cur) == (211, 37, 11)
    first, bare, last = typed.layers
    assert (first.mixer.heads, first.mixer.kv_heads, first.mixer.dim, first.mixer.vdim, first.mixer.bias_rows, first.mixer.bias_max) == (6, 2, 32, 32, 12, 90)
    assert (first.mixer.q_temp.coef, first.mixer.q_temp.every) == (0.4, 50)
    m = first.mlp
    assert (m.experts, m.top, m.groups, m.keep, m.identity, m.ff, m.limit, m.shared_ff, m.shared_limit) == (10, 3, 3, 2, 2, 24, 1.5, 40, 0.75)
    assert bare.mlp is None and bare.mixer.q_temp is None
    assert (last.mlp.groups, last.mlp.keep, last.mlp.shared_ff, last.mlp.identity) == (1, 1, 0, 1)
    plain = copy.deepcopy(pk.SMALL["A"])
    for key in ("embedding", "residual_mult", "logit_scale"):
        plain.pop(key)
    typed = KodulixConfig.from_dict(plain)
    assert typed.bigram is None and (typed.residual_mult, typed.logit_scale) == (1.0, 1.0)


def test_the_rows_of_a_bias_table_are_read_from_its_tensor():
    cfg = copy.deepcopy(pk.SMALL["A"])
    for layer in cfg["layers"]:
        layer["mixer"].pop("bias_rows")
    with pytest.raises(ConfigError, match="bias_rows"):
        KodulixConfig.from_dict(cfg)
    full = complete_from_shapes(cfg, pk.tensor_shapes(pk.SMALL["A"]))
    assert full == pk.SMALL["A"] and "bias_rows" not in cfg["layers"][0]["mixer"]


def broken(change):
    cfg = copy.deepcopy(pk.SMALL["A"])
    change(cfg)
    return cfg


@pytest.mark.parametrize("change,names", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("norm"), "norm.eps"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["embedding"]["bigram"].pop("buckets"), "embedding.bigram.buckets"),
    (lambda c: c["embedding"]["bigram"].update(mul_cur=-1), "embedding.bigram.mul_cur"),
    (lambda c: c["layers"][0].update(type="recurrence"), "layers[0].type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "layers[0].mixer.heads"),
    (lambda c: c["layers"][0]["mixer"].update(bias_rows=7), "layers[0].mixer"),
    (lambda c: c["layers"][0]["mixer"].update(bias_max=6), "layers[0].mixer.bias_max"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "layers[0].mixer.q_temp.every"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "layers[0].mlp.kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "layers[0].mlp.router.top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=3), "layers[0].mlp.router.groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "layers[0].mlp.router.groups"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "layers[0].mlp.expert.limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "layers[0].mlp.shared.ff"),
])
def test_a_wrong_configuration_is_refused_with_the_key_named(change, names):
    with pytest.raises(ConfigError) as e:
        KodulixConfig.from_dict(broken(change))
    assert names in str(e.value)


@pytest.mark.parametrize("rows,reach", [(2, 3), (4, 3), (12, 90), (16, 128), (32, 128), (32, 17), (64, 1024), (6, 64), (8, 5000)])
def test_buckets_of_distances(rows, reach):
    """Every distance's bucket, and at borders that whole numbers decide: (32, 128) has a border wherever 8^k/16 comes to one."""
    from borrowed_compute_b200.ops import BIAS_BACK, BIAS_FRONT
    from borrowed_compute_b200.parts.distance_bias import bias_table

    heads, kv_heads = 6, 2
    rel = np.random.default_rng(rows).standard_normal((rows, heads)).astype(np.float32)
    table = bias_table(torch.from_numpy(rel), reach, heads, kv_heads, factor=2.0).numpy()
    distances = table.shape[1] - BIAS_FRONT - BIAS_BACK
    assert table.shape[0] == kv_heads and table.shape[2] == heads // kv_heads and distances <= reach + 1
    for n in list(range(min(reach + 70, 400))) + [reach - 1, reach, reach + 1]:
        b = pk.distance_bucket(n, rows, reach)
        exact = n if n < rows // 2 else rows // 2 + math.log(n / (rows // 2)) / math.log(reach / (rows // 2)) * (rows - rows // 2)
        assert b == min(rows - 1, math.floor(exact + 1e-9)) or b == min(rows - 1, math.floor(exact - 1e-9)), n
        at = BIAS_FRONT + min(n, distances - 1)
        assert np.array_equal(table[:, at].reshape(-1), 2.0 * rel[b]), n
    assert np.array_equal(table[:, -BIAS_BACK:].transpose(1, 0, 2).reshape(BIAS_BACK, -1), np.repeat(2.0 * rel[-1:], BIAS_BACK, axis=0))


def test_what_the_cache_is_asked_for():
    _, model = model_for_config(pk.SMALL["A"])
    needs, states, memory_of = model.memory_needs()
    assert [n.planes for n in needs] == [((2, 32), (2, 32)), ((4, 16), (4, 48)), ((1, 64), (1, 32)), ((1, 1),)]
    assert needs[-1].dtype == torch.int32 and all(n.dtype is None for n in needs[:-1]), "token ids are kept behind the layers' keys and values"
    assert states == [None] * 4 and memory_of == [None] * 4
    assert not any(model.more_state_needs())
    from borrowed_compute_b200.parts import Runtime

    cache = PagedCache(Runtime(torch.device("cpu"), torch.bfloat16), needs, states, memory_of, max_tokens=256, n_slots=2, max_seq=256)
    ids = cache.memory(3).planes
    assert len(ids) == 1 and ids[0].dtype == torch.int32 and tuple(ids[0].shape) == (4, 1, 64, 1)
    assert cache.memory(0).planes[0].dtype == torch.bfloat16
    without = copy.deepcopy(pk.SMALL["A"])
    without["embedding"] = {}
    assert len(model_for_config(without)[1].memory_needs()[0]) == 3


def test_blocks_hand_the_stream_over_from_layer_to_layer():
    _, model = model_for_config(pk.SMALL["A"])
    assert all(b.enters_plain for b in model.blocks) and model.hand_over == [True, True, False]
    assert model.position_joined, "the sinusoids ride in the embedding's kernel"
    from borrowed_compute_b200.parts import BLOCKS, LayerSpec, PartSpec

    norm = PartSpec("rmsnorm", {"size": 8, "eps": 1e-5})
    mix = model.spec.layers[0].parts["mixer"]
    with pytest.raises(ValueError, match="no norm ahead of its feed-forward"):
        BLOCKS.get("sandwich").build(LayerSpec("sandwich", mixer=mix, norm1b=norm, norm2=norm, norm2b=norm, feed_forward=PartSpec("plain_mlp", {"hidden_size": 8, "intermediate_size": 8})), 8)
    with pytest.raises(ValueError, match="both of its norms"):
        BLOCKS.get("sandwich").build(LayerSpec("sandwich", mixer=mix, norm1b=norm, norm2b=norm), 8)


@pytest.mark.parametrize("params,says", [
    (dict(experts=4, top=2, intermediate_size=8, expert="clipped", limit=0.0, weight_on="output"), "bounds"),
    (dict(experts=4, top=2, intermediate_size=8, expert="clipped", limit=1.0, weight_on="input"), "bounds"),
    (dict(experts=4, top=3, intermediate_size=8, groups=(2, 1)), "groups"),
    (dict(experts=5, top=1, intermediate_size=8, groups=(2, 1)), "groups"),
    (dict(experts=4, top=1, intermediate_size=8, identity=1, weight_on="input"), "identity"),
    (dict(experts=4, top=1, intermediate_size=8, router="table", vocab_size=9, weight_on="output", correction=True), "table"),
])
def test_experts_refuse_what_does_not_fit(params, says):
    from borrowed_compute_b200.parts import FEED_FORWARDS

    with pytest.raises(ValueError, match=says):
        FEED_FORWARDS.get("routed_experts")(hidden_size=16, **params)


def test_attention_refuses_what_does_not_fit():
    from borrowed_compute_b200.parts import MIXERS

    kw = dict(hidden_size=16, heads=2, kv_heads=1, head_dim=8, value_dim=8, position={"kind": "none"})
    for more in (dict(distance_bias={"rows": 5, "reach": 9}), dict(distance_bias={"rows": 8, "reach": 4}), dict(query_temperature={"coef": 1.0, "every": 3}),
                 dict(query_temperature={"coef": 1.0, "every": 0}, qk_norm="head", qk_norm_eps=1e-5)):
        with pytest.raises(ValueError):
            MIXERS.get("gqa_attention_kv")(**kw, **more)


def test_the_plain_model_is_causal_and_its_parts_matter():
    """The oracle's own checks: a later token changes no earlier row, and every mechanism moves the scores."""
    cfg = pk.SMALL["A"]
    w = pk.make_weights(cfg, 5)
    toks = [int(t) for t in np.random.default_rng(1).integers(0, cfg["vocab"], 40)]
    ref, _ = pk.forward(cfg, w, toks)
    other = list(toks)
    other[30] = (other[30] + 1) % cfg["vocab"]
    changed, _ = pk.forward(cfg, w, other)
    assert np.array_equal(ref[:30], changed[:30]) and not np.allclose(ref[30:], changed[30:])
    for change in (lambda c: c["embedding"]["bigram"].update(mul_prev=38), lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=20),
                   lambda c: c["layers"][0]["mixer"].update(bias_max=60), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=1) or c["layers"][0]["mlp"]["router"].update(top=2),
                   lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.5), lambda c: c.update(residual_mult=0.5)):
        c2 = copy.deepcopy(cfg)
        change(c2)
        assert not np.allclose(pk.forward(c2, w, toks)[0], ref)
