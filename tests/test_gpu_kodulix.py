"""The Kodulix decoder on the engine against the plain implementation (plain_kodulix.py): each new mechanism alone through its
kernels, then whole models through the engine's step function, cache, scheduler and entry points: whole prompts, token-by-token
decoding, portions down to two tokens, unequal batches, slots and pages used again, sequences cut back, keys at the edges of every
bucket of distances and of pages, and far away, the first tokens, long decoding, drawn configurations, and greedy generation.

Where a bias by distance is checked, one position's key wins every softmax, and one bucket of distances takes it away again: a bucket
that begins or ends one distance off then changes whole rows.

float32 is held to the float64 oracle at 1e-4 (1 + max), bfloat16 parts at 6e-2 (1 + max), whole bfloat16 models by how far the rows
whose experts are chosen by a clear margin lie from the oracle's, relative to the scores' spread."""

from __future__ import annotations

import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import plain_kodulix as pk
from conftest import BF16_TOL, F32_TOL, ROOT

pytestmark = pytest.mark.gpu
torch = pytest.importorskip("torch")
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]


def tol(dtype, ref):
    return (F32_TOL if dtype == "float32" else 2 * BF16_TOL) * (1.0 + float(np.abs(ref).max()))


def close(got, ref, dtype, what=""):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, f"{what}: {got.shape} against {ref.shape}"
    assert np.isfinite(got).all(), f"{what}: not finite"
    worst = np.abs(got - ref).reshape(got.shape[0], -1).max(axis=-1)
    assert worst.max() <= tol(dtype, ref), f"{what}: row {int(worst.argmax())} differs by {worst.max():.4g} (allowed {tol(dtype, ref):.4g})"


def scores_close(got, ref, clear, dtype, what=""):
    """``clear``: rows whose routers choose by a margin that rounding does not bridge."""
    if dtype == "float32":
        return close(got, ref, dtype, what)
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape and np.isfinite(got).all(), f"{what}: shape or numbers"
    off = np.sqrt(((got - ref) ** 2).mean(axis=-1)) / ref.std()
    mine = off[clear] if clear.any() else off
    assert np.median(mine) <= 0.02 and np.quantile(mine, 0.9) <= 0.08, \
        f"{what}: of {mine.size} clear rows the median is off by {np.median(mine):.4g}, the 90th percentile by {np.quantile(mine, 0.9):.4g} of the spread"


def dev(a, dtype=None):
    t = torch.from_numpy(np.ascontiguousarray(a)).to(DEV)
    return t if dtype is None else t.to(dtype)


def torch_type(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def context(entries, starts):
    """A StepContext on the device for parts run outside an engine."""
    from borrowed_compute_b200.engine.batch import plan_step
    from borrowed_compute_b200.parts import StepContext

    p = plan_step(entries, starts)
    return StepContext(rows=p.rows, seqs=p.seqs, tokens=dev(p.tokens), row_pos=dev(p.row_pos), row_slot=dev(p.row_slot),
                       seq_rows=dev(p.seq_rows), seq_slot=dev(p.seq_slot), seq_start=dev(p.seq_start), max_new=p.max_new,
                       max_total=p.max_total, decode=p.decode, host_seq_rows=tuple(int(x) for x in p.seq_rows),
                       host_seq_slot=tuple(int(x) for x in p.seq_slot), host_seq_start=tuple(int(x) for x in p.seq_start))


def load_part(part, w, dtype, prefix=""):
    from borrowed_compute_b200.parts import Runtime

    rt = Runtime(torch.device(DEV), dtype, max_positions=1024)
    part.load({k: dev(w[prefix + k], torch.float32 if s.role == "vector" else dtype) for k, s in part.tensors().items()}, rt)
    return rt


@pytest.fixture(autouse=True)
def _the_parts_choose_again():
    from borrowed_compute_b200 import ops
    from borrowed_compute_b200.parts import attention_kv, moe

    yield
    attention_kv.force_rows = attention_kv.force_tiles = moe.force_simt = False
    ops.set_attention_prefill_tc_tiles(0)


# ---------------------------------------------------------------------- what enters the stream

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,joined", [(16, True), (37, True), (250, False), (1032, True)])
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(1, 3, 5), (509, 2147483647, 2147483646), (64, 1, 0)])
def test_embedding_of_two_tokens_and_a_sinusoid(dtype, E, joined, buckets, mul_prev, mul_cur):
    """Portions of every size, beside other sequences, across a page's border, and a slot that is handed out again: the token before
    is the sequence's own, wherever it came in."""
    from borrowed_compute_b200 import StepEntry
    from borrowed_compute_b200.cache import PagedCache
    from borrowed_compute_b200.parts import EMBEDDINGS, POSITION_ENCODINGS

    V, rng = 300, np.random.default_rng(E + buckets)
    w = {"embed": pk.to_bf16(rng.standard_normal((V, E))), "bigram": pk.to_bf16(rng.standard_normal((buckets + 1, E)))}
    part = EMBEDDINGS.get("token_embedding")(vocab_size=V, hidden_size=E, tensor="embed", bigram={"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur})
    position = POSITION_ENCODINGS.get("sinusoidal")(width=E)
    rt = load_part(part, w, torch_type(dtype))
    position.load({}, rt)
    if joined:
        assert part.join(position)
    cfg = {"width": E, "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    t64 = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    cache = PagedCache(rt, [part.cache_need()], [None], [None], max_tokens=1024, n_slots=3, max_seq=512)
    for round_ in range(2):
        seqs = [[int(t) for t in rng.integers(0, V, n)] for n in (200, 70, 130)]
        slots, at, got = [cache.acquire() for _ in seqs], [0, 0, 0], [[], [], []]
        for portion in (2, 1, 61, 1, 3, 64, 1, 1, 200):
            entries, starts, who = [], [], []
            for i, s in enumerate(seqs):
                n = min(portion if i != 1 else 1 + portion % 3, len(s) - at[i])
                if n > 0:
                    entries.append(StepEntry(slots[i], s[at[i]:at[i] + n]))
                    starts.append(at[i])
                    who.append((i, n))
                    cache.slots.reserve(slots[i], at[i] + n, rows=n)
            cache.sync_tables()
            ctx = context(entries, starts)
            out = torch.empty((ctx.rows, E), dtype=torch.float32, device=DEV)
            part.forward(ctx, out, mem=cache.memory(0))
            if not joined:
                position.on_embeddings(out, ctx)
            r = 0
            for i, n in who:
                got[i].append(out[r:r + n].cpu().numpy())
                cache.slots.commit(slots[i], at[i] + n)
                at[i] += n
                r += n
        for i, s in enumerate(seqs):
            rows = np.concatenate(got[i])
            close(rows, pk.embedded(cfg, t64, s)[: len(rows)], "float32", f"sequence {i}, round {round_}")
        for s in slots:
            cache.release(s)


def test_sinusoids_far_out():
    """Angles of hundreds of thousands of radians keep their fraction of a turn."""
    from borrowed_compute_b200 import ops
    from borrowed_compute_b200.parts import POSITION_ENCODINGS, Runtime

    E, at = 96, [0, 1, 63, 4097, 65535, 131072, 999983]
    position = POSITION_ENCODINGS.get("sinusoidal")(width=E)
    position.load({}, Runtime(torch.device(DEV), torch.bfloat16))
    out = torch.zeros((len(at), E), dtype=torch.float32, device=DEV)
    pos = dev(np.asarray(at, dtype=np.int32))
    ops.embed_sum(None, torch.zeros_like(pos), pos, torch.zeros_like(pos), out, frequencies=position.frequencies)
    assert np.abs(out.cpu().numpy() - pk.sinusoid(at, E)).max() < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E", [8, 37, 264, 4096])
def test_a_result_normed_into_the_stream_with_a_multiplier(dtype, E):
    """x + m norm(y), the stream rounded for the next sublayer, and the buffer cleared for its result."""
    from borrowed_compute_b200 import ops
    from borrowed_compute_b200.parts import NORMS

    rng = np.random.default_rng(E)
    w = {"n": pk.to_bf16(0.5 * rng.standard_normal(E) - 0.5)}
    part = NORMS.get("rmsnorm")(size=E, eps=1e-3, tensor="n", offset=1.0, factor=0.35)
    load_part(part, w, torch_type(dtype))
    x, y = rng.standard_normal((7, E)).astype(np.float32), (3.0 * rng.standard_normal((7, E))).astype(np.float32)
    stream, buf, h = dev(x), dev(y), torch.empty((7, E), dtype=torch_type(dtype), device=DEV)
    ops.enter_plain(stream, h, torch.empty_like(buf))
    assert torch.equal(h, stream.to(h.dtype))
    want = x + 0.35 * pk.offset_norm(y.astype(np.float64), np.asarray(w["n"], dtype=np.float64), 1e-3)
    ops.norm_add_norm(buf, part.weight, stream, part.eps, None, h, part.eps)
    close(stream.cpu().numpy(), want, "float32")
    assert torch.equal(h, stream.to(h.dtype)) and not buf.any()


# ----------------------------------------------------------------------------------- attention

def biased_part(m, E, eps):
    from borrowed_compute_b200.parts import MIXERS

    return MIXERS.get("gqa_attention_kv")(hidden_size=E, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], position={"kind": "none"},
                                          scale=m["scale"], qk_norm_eps=eps, qk_norm="head", distance_bias={"rows": m["bias_rows"], "reach": m["bias_max"]},
                                          query_temperature=m.get("q_temp"))


def run_part(part, rt, x, portions, E):
    """The mixer's output for one sequence's rows, fed in portions (then one row a step), from a cache of its own."""
    from borrowed_compute_b200 import StepEntry
    from borrowed_compute_b200.cache import PagedCache

    cache = PagedCache(rt, [part.cache_need()], [part.state_need()], [None], max_tokens=1024, n_slots=2, max_seq=1024)
    for plane in cache.memory(0).planes:
        plane.fill_(float("nan"))               # what an earlier owner of a page left must reach nobody
    slot, at, got = cache.acquire(), 0, []
    for n in list(portions) + [1] * len(x):
        if at >= len(x):
            break
        rows = x[at:at + n]
        cache.slots.reserve(slot, at + len(rows), rows=len(rows))
        cache.sync_tables()
        residual = torch.zeros((len(rows), E), dtype=torch.float32, device=DEV)
        part.forward(dev(rows, rt.dtype), residual, context([StepEntry(slot, [0] * len(rows))], [at]), cache.memory(0))
        cache.slots.commit(slot, at + len(rows))
        got.append(residual.cpu().numpy())
        at += len(rows)
    return np.concatenate(got)


def planted(rng, m, E, star, T):
    """Weights and inputs of one mixer in which position ``star``'s key wins every softmax that sees it without a bias: input channel 0
    is zero but at ``star`` and alone drives every key head along one direction; channel 1 (one everywhere) drives every query along it."""
    H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mat = lambda r, c, s=1.0: rng.standard_normal((r, c)) * s / math.sqrt(c)                 # noqa: E731
    w = {"q": mat(H * D, E, 0.3), "k": mat(G * D, E), "v": mat(G * DV, E, 2.0), "o": mat(E, H * DV), "q.norm": np.ones(D), "k.norm": np.ones(D),
         "rel": np.zeros((m["bias_rows"], H))}
    w["k"][:, 0] = 0.0
    for g in range(G):
        u = rng.choice([-1.0, 1.0], D)
        w["k"][g * D:(g + 1) * D, 0] = 2.0 * u
        for h in range(g * (H // G), (g + 1) * (H // G)):
            w["q"][h * D:(h + 1) * D, 0] = 0.0
            w["q"][h * D:(h + 1) * D, 1] = 6.0 * u
    x = rng.standard_normal((T, E)) * 0.5
    x[:, 0], x[:, 1] = 0.0, 1.0
    x[star, 0] = 8.0
    return {k: pk.to_bf16(v) for k, v in w.items()}, pk.to_bf16(x)


def as64(w):
    return {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}


PATHS = [("float32", "rows"), ("bfloat16", "rows"), ("bfloat16", "tiles"), ("bfloat16", "own")]


def take(path):
    from borrowed_compute_b200.parts import attention_kv

    attention_kv.force_rows, attention_kv.force_tiles = path == "rows", path == "tiles"


@pytest.mark.parametrize("dtype,path", PATHS)
@pytest.mark.parametrize("H,G,D,DV", [(4, 1, 64, 64), (4, 2, 128, 64), (3, 3, 32, 32), (5, 1, 64, 128), (2, 1, 20, 12), (6, 2, 64, 16)])
def test_one_key_and_the_bucket_of_distances_that_takes_it_away(dtype, path, H, G, D, DV):
    """The planted key wins a row unless its distance lies in the one bucket whose bias is far below zero: single distances, wide
    buckets, the last one, whose distances never end; at pages' borders; whole, in portions and row by row."""
    E, T, rows, reach = 48, 300, 12, 90
    firsts = [next(n for n in range(1000) if pk.distance_bucket(n, rows, reach) == b) for b in range(rows)]
    assert len(set(firsts)) == rows
    m = pk.mixer(H, G, D, DV, rows, reach, scale=10.0 / D, temp=None)
    take(path)
    for star, bucket in ((0, 0), (5, 3), (63, 6), (64, 9), (10, 11), (127, 11)):
        w, x = planted(np.random.default_rng(star * 7 + bucket), m, E, star, T)
        w["rel"][bucket] = -30.0
        ref = pk.attention(np.asarray(x, dtype=np.float64), m, as64(w), "", 1e-5)
        shifted = dict(as64(w), rel=np.zeros((rows, H)))
        without = pk.attention(np.asarray(x, dtype=np.float64), m, shifted, "", 1e-5)
        inside = [i for i in range(star + 1, T) if pk.distance_bucket(i - star, rows, reach) == bucket]
        outside = [i for i in range(star + 1, T) if i not in inside]
        size = np.abs(ref).max()
        assert all(np.abs(ref[i] - without[i]).max() > 0.1 * size for i in inside), "the bucket decides its rows"
        assert not outside or np.median([np.abs(ref[i] - without[i]).max() for i in outside]) < 0.05 * size
        part = biased_part(m, E, 1e-5)
        rt = load_part(part, w, torch_type(dtype))
        for portions in ([T], [star + 1, 2], [2, 61, 3, 62, 2, 9, 64]):
            close(run_part(part, rt, x, portions, E), ref, dtype, f"star {star}, bucket {bucket}, portions {portions}")


@pytest.mark.parametrize("dtype,path", PATHS)
@pytest.mark.parametrize("star", [0, 63, 64, 200])
def test_one_far_key_among_hundreds(dtype, path, star):
    """Hundreds of positions behind, past the table's reach and with the last bucket's bias against it, the planted key still decides
    the last rows; a sequence's first rows see what little there is."""
    E, T = 64, 600
    m = pk.mixer(4, 2, 64, 64, 8, 40, scale=14.0 / 64, temp=(0.3, 100))
    w, x = planted(np.random.default_rng(star), m, E, star, T)
    w["rel"] = pk.to_bf16(np.linspace(1.0, -2.0, 8)[:, None] + 0.1 * np.arange(4)[None, :])
    ref = pk.attention(np.asarray(x, dtype=np.float64), m, as64(w), "", 1e-5)
    lost = np.array(x)
    lost[star] = 0.0
    assert np.abs(pk.attention(np.asarray(lost, dtype=np.float64), m, as64(w), "", 1e-5)[-1] - ref[-1]).max() > 0.2 * np.abs(ref).max()
    take(path)
    part = biased_part(m, E, 1e-5)
    rt = load_part(part, w, torch_type(dtype))
    for portions in ([T], [star + 1, 2, 2], [1, 2, 500, 64]):
        close(run_part(part, rt, x, portions, E), ref, dtype, f"portions {portions}")


@pytest.mark.parametrize("dtype,path", PATHS)
@pytest.mark.parametrize("H,G,D,DV,rows,reach,temp", [(1, 1, 64, 64, 2, 3, (0.7, 1)), (8, 1, 128, 128, 32, 128, (1.0, 64)), (10, 2, 64, 64, 64, 1000, None),
                                                      (16, 1, 32, 64, 16, 300, (2.0, 17)), (3, 1, 128, 32, 6, 500, (0.1, 250)), (7, 7, 96, 96, 4, 5, None),
                                                      (40, 2, 64, 128, 20, 64, (0.5, 33)), (4, 4, 200, 136, 10, 700, (0.5, 99)), (6, 3, 10, 18, 2, 2, (1.0, 3))])
def test_biases_and_temperatures_in_other_sizes(dtype, path, H, G, D, DV, rows, reach, temp):
    """One head; groups of five, sixteen and twenty heads; values narrower and wider than keys; tables of one distance each, and
    tables longer than the sequence; temperatures that change every position and every hundred."""
    from borrowed_compute_b200 import ops

    E, T = 40, 330
    m = pk.mixer(H, G, D, DV, rows, reach, scale=1.5 / math.sqrt(D), temp=temp)
    w = {k[len("l0.mix."):]: v for k, v in pk.make_weights(pk.model(10, E, [(m, None)]), H + D).items() if k.startswith("l0.mix.")}
    x = pk.to_bf16(np.random.default_rng(D).standard_normal((T, E)))
    ref = pk.attention(np.asarray(x, dtype=np.float64), m, as64(w), "", 1e-6)
    take(path)
    part = biased_part(m, E, 1e-6)
    rt = load_part(part, w, torch_type(dtype))
    for portions in ([T], [200, 2, 100]):
        close(run_part(part, rt, x, portions, E), ref, dtype, f"portions {portions}")
    if dtype == "bfloat16" and path == "own":
        for tiles in (1, 2):                    # query tiles a block of the tcgen05 kernel
            ops.set_attention_prefill_tc_tiles(tiles)
            close(run_part(part, rt, x, [T], E), ref, dtype, f"{tiles} query tiles a block")


@pytest.mark.parametrize("via_scratch", [False, True])
@pytest.mark.parametrize("splits", [1, 2, 3, 8, 16])
@pytest.mark.parametrize("H,G,D,DV", [(4, 1, 128, 64), (8, 2, 64, 128), (6, 3, 64, 32), (16, 1, 128, 32), (4, 2, 32, 64), (8, 2, 128, 128), (12, 2, 48, 48)])
def test_split_decode_with_values_of_their_own_width_and_biases(H, G, D, DV, splits, via_scratch):
    """Every number of splits, merged in clusters and through scratch memory, against the one-warp-a-row kernel."""
    from borrowed_compute_b200 import ops
    from borrowed_compute_b200.parts.distance_bias import bias_table

    if via_scratch and splits == 1:
        pytest.skip("one split merges nothing")
    g = torch.Generator(device=DEV).manual_seed(H * D + DV)
    lengths = [1, 64, 65, 700, 333]
    pages = [-(-n // 64) for n in lengths]
    table = torch.full((len(lengths), 12), -1, dtype=torch.int32, device=DEV)
    at = 0
    for i, n in enumerate(pages):
        table[i, :n] = torch.arange(at, at + n, dtype=torch.int32, device=DEV)
        at += n
    k = torch.randn((at, G, 64, D), generator=g, device=DEV).bfloat16()
    v = torch.randn((at, G, 64, DV), generator=g, device=DEV).bfloat16()
    q = torch.randn((len(lengths), H * D), generator=g, device=DEV).bfloat16()
    pos = torch.tensor([n - 1 for n in lengths], dtype=torch.int32, device=DEV)
    slot = torch.tensor([0, 1, 2, 3, 4], dtype=torch.int32, device=DEV)
    rel = torch.randn((16, H), generator=g, device=DEV)
    plain, log2 = bias_table(rel, 200, H, G), bias_table(rel, 200, H, G, factor=1.0 / math.log(2.0))
    want = torch.empty((len(lengths), H * DV), dtype=torch.bfloat16, device=DEV)
    for bias in (None, (plain, log2)):
        ops.attention_rows(q, H * D, k, v, table, pos, slot, want, H, G, D, value_dim=DV, bias=None if bias is None else bias[0])
        got = torch.empty_like(want)
        ops.attention_decode(q, H * D, k, v, table, pos, slot, got, H, G, D, value_dim=DV, splits=splits, via_scratch=via_scratch, bias=None if bias is None else bias[1])
        close(got.float().cpu().numpy(), want.float().cpu().numpy(), "bfloat16", f"bias {bias is not None}")


# ------------------------------------------------------------------------------------- experts

def experts_part(f, E, dtype):
    from borrowed_compute_b200.parts import FEED_FORWARDS

    r, groups = f["router"], f["router"].get("groups") or {"count": 1, "keep": 1}
    shared = f.get("shared") or {"ff": 0, "limit": 0.0}
    return FEED_FORWARDS.get("routed_experts")(
        hidden_size=E, experts=r["experts"], top=r["top"], intermediate_size=f["expert"]["ff"], shared_size=shared["ff"], score="softmax", renormalize=True,
        weight_on="output", expert="clipped", limit=f["expert"]["limit"], shared_limit=shared["limit"], correction=True,
        groups=(groups["count"], groups["keep"]), identity=r.get("identity", 0))


def clear_rows(rng, w, f, E, rows):
    """Inputs whose routers choose by a margin, so that rounding chooses the same."""
    r, groups = f["router"], f["router"].get("groups") or {"count": 1, "keep": 1}
    x = pk.to_bf16(rng.standard_normal((rows * 4, E)))
    z = x.astype(np.float64) @ np.asarray(w["router"], dtype=np.float64).T
    p = np.exp(z - z.max(axis=-1, keepdims=True))
    c = p / p.sum(axis=-1, keepdims=True) + np.asarray(w["correction"], dtype=np.float64)
    gap = np.asarray([pk.choice_margin(row, r["top"], groups["count"], groups["keep"]) for row in c])
    return x[np.argsort(-gap, kind="stable")[:rows]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("simt", [False, True])
@pytest.mark.parametrize("E,f,rows", [
    (32, pk.moe(6, 2, 16, 0.75), 50),
    (40, pk.moe(10, 3, 24, 0.5, identity=2, groups=(3, 2), shared=(16, 0.25)), 200),
    (24, pk.moe(1, 1, 8, 1.0, identity=5), 9),
    (64, pk.moe(36, 8, 32, 1.5, identity=12, groups=(12, 5), shared=(64, 1.0)), 300),
    (50, pk.moe(7, 4, 14, 1.0, identity=1, groups=(2, 1), shared=(18, 2.0)), 33),
    (128, pk.moe(100, 16, 64, 0.6, identity=28, groups=(4, 1)), 70),
    (16, pk.moe(3, 3, 8, 7.0, shared=(8, 7.0)), 1),
])
def test_experts_in_groups_beside_identity_experts(dtype, simt, E, f, rows):
    """Choice scores mostly below zero (a group left out must not win by counting as zero), corrections that choose and do not weigh,
    bounds that gates and up branches meet, rows whose every choice is an identity expert."""
    from borrowed_compute_b200 import StepEntry
    from borrowed_compute_b200.parts import moe

    rng = np.random.default_rng(E + rows)
    cfg = pk.model(10, E, [(pk.mixer(1, 1, 8, 8, 2, 3), f)])
    w = {k[len("l0.mlp."):]: v for k, v in pk.make_weights(cfg, E).items() if k.startswith("l0.mlp.")}
    assert (w["correction"] < 0).any()
    x = clear_rows(rng, w, f, E, rows)
    ref = pk.experts(x.astype(np.float64), f, as64(w), "")
    moe.force_simt = simt
    part = experts_part(f, E, dtype)
    rt = load_part(part, w, torch_type(dtype))
    out = torch.zeros((rows, E), dtype=torch.float32, device=DEV)
    part.forward(dev(x, rt.dtype), out, context([StepEntry(0, [0] * rows)], [0]))
    close(out.cpu().numpy(), ref, dtype)


@pytest.mark.parametrize("n,top,groups,keep", [(12, 3, 1, 1), (12, 3, 4, 2), (48, 6, 8, 3), (300, 16, 30, 4), (8, 8, 8, 8), (64, 2, 64, 2)])
def test_choices_and_weights_of_the_router(n, top, groups, keep):
    """Choice for choice, in order; scores that tie go to the lower index; padding rows choose nothing; corrections so negative that a
    group left out would win if it counted as zero."""
    from borrowed_compute_b200 import ops

    rng = np.random.default_rng(n + keep)
    rows, E = 90, 24
    router, x = (0.25 * rng.standard_normal((n, E))).astype(np.float32), rng.standard_normal((rows, E)).astype(np.float32)
    correction = (0.3 * rng.standard_normal(n) - 2.0).astype(np.float32)
    x[0] = 0.0                                            # every score alike
    flat = np.full(n, -1.5, dtype=np.float32)
    slot = np.zeros(rows, dtype=np.int32)
    slot[5] = -1
    for c in (correction, flat, None):
        choice, weight = torch.empty((rows, top), dtype=torch.int32, device=DEV), torch.empty((rows, top), dtype=torch.float32, device=DEV)
        ops.moe_route(dev(x), dev(router), dev(slot), torch.empty((rows, n), dtype=torch.float32, device=DEV), choice, weight, softmax=True, renorm=True,
                      correction=None if c is None else dev(c), groups=groups, keep=keep)
        want, weights = pk.route(x.astype(np.float64), router.astype(np.float64), np.zeros(n) if c is None else c.astype(np.float64), top, groups, keep)
        got, gw = choice.cpu().numpy(), weight.cpu().numpy()
        assert (got[5] == -1).all() and (gw[5] == 0).all()
        if c is not correction:
            assert got[0].tolist() == want[0].tolist(), "ties go to the lower index"
        z = x.astype(np.float64) @ router.astype(np.float64).T
        p = np.exp(z - z.max(axis=-1, keepdims=True))
        scores = p / p.sum(axis=-1, keepdims=True) + (0.0 if c is None else c)
        # rows whose order float32 does not turn: clear margins, and clear gaps between one choice and the next
        clear = [i for i in range(1, rows) if i != 5 and pk.choice_margin(scores[i], top, groups, keep) > 1e-6
                 and (top == 1 or np.abs(np.diff(scores[i][want[i]])).min() > 1e-6)]
        assert len(clear) > rows // 2
        assert got[clear].tolist() == want[clear].tolist()
        assert np.abs(gw[clear] - weights[clear]).max() < 1e-5


# --------------------------------------------------------------------------------- whole models

def engine_for(cfg, weights, dtype, **kw):
    from borrowed_compute_b200.engine import Engine

    kw.setdefault("max_tokens", 4096)
    kw.setdefault("max_slots", 6)
    kw.setdefault("max_seq", 1024)
    return Engine.from_tensors(cfg, {n: torch.from_numpy(np.ascontiguousarray(a)) for n, a in weights.items()}, dtype=dtype, **kw)


_made = {}


def small(name, dtype):
    key = (name, dtype)
    if key not in _made:
        cfg = pk.SMALL[name]
        w = pk.make_weights(cfg, seed=31 if name == "A" else 32)
        _made[key] = (engine_for(cfg, w, dtype), cfg, w)
    return _made[key]


def tokens(cfg, n, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def oracle(cfg, w, toks):
    """(scores, streams, which rows choose their experts by a clear margin)."""
    ref, streams = pk.forward(cfg, w, toks)
    return ref, streams, pk.row_margins(cfg, w, toks) > 0.02


def run_whole(eng, toks):
    from borrowed_compute_b200.engine import StepEntry

    s = eng.acquire()
    out = eng.step([StepEntry(s, toks, tuple(range(len(toks))))]).cpu().numpy()
    eng.release(s)
    return out


def run_cut(eng, toks, cuts):
    """The same tokens in portions of the given sizes (the rest one token at a time)."""
    from borrowed_compute_b200.engine import StepEntry

    s, at, rows = eng.acquire(), 0, []
    for n in list(cuts) + [1] * len(toks):
        if at >= len(toks):
            break
        part = toks[at:at + n]
        rows.append(eng.step([StepEntry(s, part, tuple(range(len(part))))]).cpu().numpy())
        at += len(part)
    eng.release(s)
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_whole_prompts_and_the_stream_after_every_layer(name, dtype):
    eng, cfg, w = small(name, dtype)
    toks = tokens(cfg, 150, seed=1)
    ref, streams, clear = oracle(cfg, w, toks)
    got = []
    eng.model.after_run = lambda i, res: got.append(res.detach().float().cpu().numpy().copy())
    try:
        out = run_whole(eng, toks)
    finally:
        eng.model.after_run = None
    assert len(got) == len(streams)
    for i, (g, s) in enumerate(zip(got, streams)):
        scores_close(g[: len(toks)], s, clear, dtype, f"the stream after layer {i}")
    scores_close(out, ref, clear, dtype, "scores")
    for n in (1, 2, 3):            # the first tokens of a sequence, alone
        scores_close(run_whole(eng, toks[:n]), ref[:n], clear[:n], dtype, f"a prompt of {n}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_prefill_against_token_by_token_and_portions(name, dtype):
    eng, cfg, w = small(name, dtype)
    toks = tokens(cfg, 200, seed=2)
    ref, _, clear = oracle(cfg, w, toks)
    for cuts in ([], [120], [2] * 100, [2, 2, 60, 3, 64, 1, 2, 40], [64, 64], [63, 2, 63], [199]):
        scores_close(run_cut(eng, toks, cuts), ref, clear, dtype, f"portions {cuts}")
    eng.cache.slots.check()


@pytest.mark.parametrize("name", ["A", "B"])
def test_cuts_and_batches_give_the_same_bits_in_float32(name):
    from borrowed_compute_b200.engine import StepEntry

    eng, cfg, w = small(name, "float32")
    toks = tokens(cfg, 140, seed=3)
    whole = run_whole(eng, toks)
    assert np.array_equal(run_cut(eng, toks, [70, 2, 30]), whole)
    others = [tokens(cfg, n, seed=4 + n) for n in (5, 90)]
    slots = [eng.acquire() for _ in range(3)]
    out = eng.step([StepEntry(slots[0], others[0], (4,)), StepEntry(slots[1], toks, tuple(range(len(toks)))), StepEntry(slots[2], others[1], ())]).cpu().numpy()
    for s in slots:
        eng.release(s)
    assert np.array_equal(out[1:], whole)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_batches_against_each_alone_then_decoded_together(name, dtype):
    from borrowed_compute_b200.engine import StepEntry

    eng, cfg, w = small(name, dtype)
    lengths, tail = [1, 37, 130, 66], 40
    seqs = [tokens(cfg, n + tail, seed=10 + n) for n in lengths]
    refs = [oracle(cfg, w, s) for s in seqs]
    slots = [eng.acquire() for _ in seqs]
    rows = [[] for _ in seqs]
    out = eng.step([StepEntry(sl, s[:n], tuple(range(n))) for sl, s, n in zip(slots, seqs, lengths)]).cpu().numpy()
    at = 0
    for i, n in enumerate(lengths):
        rows[i].append(out[at:at + n])
        at += n
    live = list(range(len(seqs)))
    for t in range(tail):
        if t == 25:                 # a shorter request ends earlier
            eng.release(slots[1])
            live.remove(1)
        out = eng.step([StepEntry(slots[i], [seqs[i][lengths[i] + t]], (0,)) for i in live]).cpu().numpy()
        for k, i in enumerate(live):
            rows[i].append(out[k:k + 1])
    for i in live:
        eng.release(slots[i])
    for i, r in enumerate(rows):
        got = np.concatenate(r)
        scores_close(got, refs[i][0][: len(got)], refs[i][2][: len(got)], dtype, f"sequence {i}")
    eng.cache.slots.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_used_again(dtype):
    """What a sequence left behind (keys, values, token ids) does not reach the next one in its slot and pages."""
    eng, cfg, w = small("A", dtype)
    a, b = tokens(cfg, 190, seed=20), tokens(cfg, 75, seed=21)
    ref_a, ref_b = oracle(cfg, w, a), oracle(cfg, w, b)
    for _ in range(3):
        scores_close(run_cut(eng, a, [100]), ref_a[0], ref_a[2], dtype, "the long one")
        scores_close(run_cut(eng, b, [3, 70]), ref_b[0], ref_b[2], dtype, "the short one in the same slot")
    eng.cache.slots.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cut", [0, 1, 63, 64, 65, 100])
def test_a_sequence_cut_back_goes_on_as_if_it_had_never_been_longer(dtype, cut):
    """Keys, values and the token before the cut: nothing a dropped token left reaches the rows that follow."""
    from borrowed_compute_b200.engine import StepEntry

    eng, cfg, w = small("A", dtype)
    a, b = tokens(cfg, 130, seed=22), tokens(cfg, 60, seed=23)
    joined = a[:cut] + b
    ref, _, clear = oracle(cfg, w, joined)
    s = eng.acquire()
    eng.step([StepEntry(s, a, ())])
    eng.rollback(s, cut)
    rows = [eng.step([StepEntry(s, b[:1], (0,))]).cpu().numpy(), eng.step([StepEntry(s, b[1:], tuple(range(len(b) - 1)))]).cpu().numpy()]
    eng.release(s)
    scores_close(np.concatenate(rows), ref[cut:], clear[cut:], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    eng, cfg, w = small("B", dtype)
    toks = tokens(cfg, 420, seed=30)
    ref, _, clear = oracle(cfg, w, toks)
    scores_close(run_cut(eng, toks, [20]), ref, clear, dtype)


@pytest.mark.parametrize("dtype,seed", [("float32", s) for s in range(12)] + [("bfloat16", s) for s in range(100, 110)])
def test_drawn_configurations(dtype, seed):
    rng = np.random.default_rng(seed)
    cfg = pk.draw_config(rng)
    w = pk.make_weights(cfg, seed)
    eng = engine_for(cfg, w, dtype, max_tokens=1024, max_slots=2, max_seq=512)
    toks = tokens(cfg, 150, seed=seed)
    ref, _, clear = oracle(cfg, w, toks)
    scores_close(run_whole(eng, toks), ref, clear, dtype, f"whole, {json.dumps(cfg)}")
    scores_close(run_cut(eng, toks, [2, 66, 30]), ref, clear, dtype, f"portions, {json.dumps(cfg)}")


# ------------------------------------------------------------------------------ the entry points

def folder_for(tmp_path, name, seed):
    """A model folder whose config.json leaves the tables' rows to the tensors' shapes."""
    from borrowed_compute_b200.weights.safetensors_io import write_safetensors

    cfg = pk.SMALL[name]
    w = pk.make_weights(cfg, seed)
    folder = str(tmp_path / f"kodulix_{name}")
    os.makedirs(folder, exist_ok=True)
    written = json.loads(json.dumps(cfg))
    for layer in written["layers"]:
        layer["mixer"].pop("bias_rows")
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(written, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {n: torch.from_numpy(a).to(torch.bfloat16) for n, a in w.items()})
    return folder, cfg, w


def test_greedy_generation_through_the_library_and_the_command_line(tmp_path):
    from borrowed_compute_b200 import Local, Sampling

    folder, cfg, w = folder_for(tmp_path, "A", 41)
    prompts = [tokens(cfg, n, seed=50 + n) for n in (9, 30)]
    want = [pk.generate(cfg, w, p, 12) for p in prompts]
    out, stats = Local.load(folder, dtype="float32", max_tokens=1024, max_slots=4, max_seq=256).generate(prompts, 12, Sampling(), stop_ids=())
    assert [list(g) for g in out] == want and stats.generated == 24
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "bc-infer"), "generate", folder, ";".join(",".join(map(str, p)) for p in prompts),
                          "--max-tokens", "12", "--dtype", "float32", "--stop-ids", ""], capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [[int(t) for t in line.split(",")] for line in res.stdout.strip().splitlines()] == want
    # bfloat16 decodes through captured graphs, tokens going from sampler to embedding on the device (the second embedding takes the
    # token before from its pages): the tokens are the oracle's wherever its two best scores lie well apart
    out16, _ = Local.load(folder, dtype="bfloat16", max_tokens=1024, max_slots=4, max_seq=256).generate(prompts, 12, Sampling(), stop_ids=())
    for p, mine in zip(prompts, out16):
        toks = list(p)
        assert len(mine) == 12
        for t in mine:
            last = pk.forward(cfg, w, toks)[0][-1]
            best = np.sort(last)
            if best[-1] - best[-2] > 0.1 * (1.0 + np.abs(last).max()):
                assert t == int(last.argmax()), "a clear choice was missed"
            toks.append(int(t))


def test_more_prompts_than_slots_take_turns(tmp_path):
    from borrowed_compute_b200 import Local, Sampling

    folder, cfg, w = folder_for(tmp_path, "B", 43)
    prompts = [tokens(cfg, n, seed=70 + n) for n in (5, 70, 1, 33, 64)]
    out, _ = Local.load(folder, dtype="float32", max_tokens=512, max_slots=2, max_seq=256).generate(prompts, 8, Sampling(), stop_ids=(), max_batch=2)
    assert [list(g) for g in out] == [pk.generate(cfg, w, p, 8) for p in prompts]


@pytest.mark.parametrize("dtype", DTYPES)
def test_replaying_steps_with_the_trace_tool(tmp_path, dtype):
    folder, cfg, w = folder_for(tmp_path, "B", 42)
    a, b = tokens(cfg, 80, seed=60), tokens(cfg, 33, seed=61)
    (ref_a, _, clear_a), (ref_b, _, clear_b) = oracle(cfg, w, a), oracle(cfg, w, b)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:50], "want": list(range(50))}, {"id": "y", "tokens": b[:20], "want": []}], "end": []}]
    steps += [{"step": 1 + t, "entries": [{"id": "x", "tokens": a[50 + t:51 + t], "want": [0]}] +
               ([{"id": "y", "tokens": b[20 + t:21 + t], "want": [0]}] if t < 13 else []), "end": ["y"] if t == 12 else []} for t in range(30)]
    out = str(tmp_path / "scores")
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out, "--max-tokens", "256"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [line for line in res.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(31)]
    read = lambda i: np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])      # noqa: E731
    rows_a = np.concatenate([read(0)] + [read(1 + t)[:1] for t in range(30)])
    rows_b = np.concatenate([read(1 + t)[1:] for t in range(13)])
    scores_close(rows_a, ref_a, clear_a, dtype, "the longer request")
    scores_close(rows_b, ref_b[20:], clear_b[20:], dtype, "the shorter request")
