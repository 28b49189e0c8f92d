"""The Duratar decoder on the engine against the plain implementation (plain_duratar.py): each new mechanism alone through its
kernels, then whole models through the engine's step function, cache, scheduler and entry points: whole prompts, token-by-token
decoding, portions down to two tokens, unequal batches, slots and pages used again, keys at the edges of windows, of the kept
first positions and of pages, and far away, the first tokens, long decoding, drawn configurations, and greedy generation.

Differential attention is run on inputs and weights made so that ONE position's key wins one map's softmax wherever it is seen: a
mask that is one position off then changes whole rows.

float32 engines are held to the float64 oracle tightly (1e-4 (1 + max|score|)), bfloat16 ones within 6e-2 (1 + max|score|)."""

from __future__ import annotations

import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import plain_duratar as pd
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


def mostly_close(got, ref, dtype, what="", least=0.0):
    """Whole bfloat16 models: norms of small results (a difference of two maps, a read-out of a state that nearly cancels) magnify
    rounding at single rows.  Nine rows in ten are held to the tolerance and the median row to a third of it (``least``: a wider
    one, for models whose rows rounding alone moves further); a wrong key, window or state moves every row that follows."""
    if dtype == "float32":
        return close(got, ref, dtype, what)
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape and np.isfinite(got).all(), f"{what}: shape or numbers"
    worst, allowed = np.abs(got - ref).reshape(got.shape[0], -1).max(axis=-1), max(tol(dtype, ref), least)
    assert np.quantile(worst, 0.9) <= allowed and np.median(worst) <= allowed / 3, \
        f"{what}: the 90th percentile of the rows differs by {np.quantile(worst, 0.9):.4g}, the median by {np.median(worst):.4g} (allowed {allowed:.4g})"


def tokens_for(cfg, n, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def dev(a, dtype=None):
    t = torch.from_numpy(np.array(a, order="C")).to(DEV)
    return t if dtype is None else t.to(dtype)


def torch_type(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def engine_for(cfg, weights, dtype, **kw):
    from borrowed_compute_b200.engine import Engine

    kw.setdefault("max_tokens", 4096)
    kw.setdefault("max_slots", 6)
    kw.setdefault("max_seq", 1024)
    return Engine.from_tensors(cfg, {n: torch.from_numpy(np.array(a)) for n, a in weights.items()}, dtype=dtype, **kw)


_made = {}
NAMES = ["A", "B", "C"]


def small(name, dtype):
    key = (name, dtype)
    if key not in _made:
        cfg = pd.SMALL[name]
        w = pd.make_weights(cfg, seed=40 + NAMES.index(name))
        _made[key] = (engine_for(cfg, w, dtype), cfg, w)
    return _made[key]


def run_whole(eng, toks):
    from borrowed_compute_b200.engine import StepEntry

    s = eng.acquire()
    out = eng.step([StepEntry(s, toks, tuple(range(len(toks))))]).cpu().numpy()
    eng.raise_on_kernel_error()
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
    eng.raise_on_kernel_error()
    eng.release(s)
    return np.concatenate(rows)


@pytest.fixture(autouse=True)
def _the_parts_choose_again():
    from borrowed_compute_b200.parts import channel_delta, diff_attention

    yield
    diff_attention.force, diff_attention.force_splits = None, 0
    channel_delta.split_steps = False


# ------------------------------------------------------------------ each mechanism alone

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


def weights_of(m, E, seed):
    """The tensors of one mixer, by their names inside it."""
    return {k[len("l0.mix."):]: v for k, v in pd.make_weights(pd.model(10, E, 1, [(m, 0)]), seed).items() if k.startswith("l0.mix.")}


def run_part(part, rt, x, portions, E, spoil=False):
    """The mixer's output for one sequence's rows, fed in portions (then one row a step), from a cache of its own; ``spoil`` fills the
    cache's pages with not-a-numbers first (what another sequence might have left)."""
    from borrowed_compute_b200 import StepEntry
    from borrowed_compute_b200.cache import PagedCache

    cache = PagedCache(rt, [part.cache_need()], [part.state_need()], [None], max_tokens=1024, n_slots=2, max_seq=1024,
                       more_states=[{"mixer." + n: need for n, need in part.more_state_needs().items()}])
    if spoil:
        for group in cache.groups:
            for plane in group.planes:
                plane.fill_(float("nan"))
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
    cache.slots.check()
    cache.release(slot)
    return np.concatenate(got)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,E,rows", [(1, 8, 3), (2, 20, 70), (3, 33, 5), (4, 264, 130), (5, 50, 2), (7, 96, 9), (8, 1030, 3), (9, 40, 6), (20, 12, 4), (4, 4096, 2)])
def test_streams_between_two_sublayers(dtype, S, E, rows):
    """The one kernel between sublayers against the three steps one after another: a bundle started from normed rows, entered, left,
    entered again with its result pending, and finished for some of its rows, each with connections of its own."""
    from borrowed_compute_b200.parts import CONNECTIONS, NORMS, SCALES
    from borrowed_compute_b200.parts.streams import StreamBundle

    rng = np.random.default_rng(S * 100 + E)
    td = torch_type(dtype)
    conns, scales, norms, w = [], [], [], []
    for i in range(2):
        t = {"in": pd.to_bf16(rng.standard_normal(S)), "out": pd.to_bf16(rng.standard_normal(S)), "mix": pd.to_bf16(rng.standard_normal((S, S)) / math.sqrt(S)),
             "ls": pd.to_bf16(rng.uniform(0.5, 1.5, E)), "n": pd.to_bf16(np.array(1.0 + 0.5 * i, dtype=np.float32))}
        w.append({k: np.asarray(v, dtype=np.float64) for k, v in t.items()})
        c, s, n = CONNECTIONS.get("hyper")(streams=S), SCALES.get("channel_scale")(width=E, tensor="ls"), NORMS.get("rmsnorm")(size=E, eps=1e-4, tensor="n", scalar=True)
        for part in (c, s, n):
            load_part(part, t, td)
        conns.append(c), scales.append(s), norms.append(n)
    e = rng.standard_normal((rows, E)).astype(np.float32)
    ys = [rng.standard_normal((rows, E)).astype(np.float32) for _ in range(2)]
    bundle = StreamBundle(rows, S, E, torch.device(DEV))
    bundle.start(dev(e), norms[0])
    X = np.repeat((pd.over_rms(e.astype(np.float64), 1e-4) * w[0]["n"])[None], S, axis=0)
    close(bundle.total().cpu().numpy(), X.sum(axis=0), "float32", "start")
    h = torch.empty((rows, E), dtype=td, device=DEV)
    for i in range(2):
        y = bundle.enter(conns[i], norms[i], h)
        close(h.float().cpu().numpy(), pd.over_rms(pd.collapse(X, w[i]["in"]), 1e-4) * w[i]["n"], dtype, f"enter {i}")
        assert not y.any(), "the buffer a sublayer adds into is not cleared"
        y += dev(ys[i])
        bundle.leave(conns[i], scales[i] if i == 0 else None)
        X = pd.spread(X, ys[i] * (w[i]["ls"] if i == 0 else 1.0), w[i]["mix"], w[i]["out"])
        close(bundle.total().cpu().numpy(), X.sum(axis=0), "float32", f"leave {i}")
    want = np.array([rows - 1, 0, rows // 2], dtype=np.int32)
    out = torch.empty((3, E), dtype=td, device=DEV)
    bundle.finish(norms[1], out, dev(want))
    ref = pd.over_rms(X.sum(axis=0), 1e-4) * w[1]["n"]
    close(out.float().cpu().numpy(), ref[want], dtype, "finish, some rows")
    every = torch.empty((rows, E), dtype=td, device=DEV)
    bundle.finish(norms[1], every, None)
    close(every.float().cpu().numpy(), ref, dtype, "finish, all rows")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,F,rows,spread", [(16, 24, 5, 1.0), (40, 52, 70, 4.0), (64, 128, 300, 1.0), (512, 1024, 9, 0.1), (264, 384, 700, 2.0), (50, 22, 40, 3.0)])
def test_feed_forward_with_xielu(dtype, E, F, rows, spread):
    """Rows on both sides of zero, near it and far out (where the exponential of the positive side would overflow)."""
    from borrowed_compute_b200.parts import FEED_FORWARDS

    rng = np.random.default_rng(F)
    w = {"up": pd.to_bf16(rng.standard_normal((F, E)) / math.sqrt(E)), "down": pd.to_bf16(rng.standard_normal((E, F)) / math.sqrt(F)),
         "act": pd.to_bf16(rng.uniform(-2, 2, 2))}
    x = pd.to_bf16(rng.standard_normal((rows, E)) * spread)
    x[0] *= 40.0
    part = FEED_FORWARDS.get("plain_mlp")(hidden_size=E, intermediate_size=F, activation="xielu")
    rt = load_part(part, w, torch_type(dtype))
    out = torch.zeros((rows, E), dtype=torch.float32, device=DEV)
    part.forward(dev(x, rt.dtype), out, None)
    ref = pd.feed_forward(x.astype(np.float64), {k: v.astype(np.float64) for k, v in w.items()}, "")
    for r in (slice(0, 1), slice(1, rows)):
        close(out.cpu().numpy()[r], ref[r], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,P,slow", [(1, 8, 8, 0.9), (3, 10, 33, 0.999), (2, 64, 40, 0.99), (5, 128, 64, 0.995), (2, 200, 12, 0.9), (4, 16, 128, 1.0)])
def test_lightning_attention(dtype, H, D, P, slow):
    """Heads that forget at once and heads that hardly do, whole, in portions and row by row."""
    from borrowed_compute_b200.parts import MIXERS

    E, T = 48, 150
    m = pd.lightning_mixer(H, D, P, slow)
    w = weights_of(m, E, D + P)
    x = pd.to_bf16(np.random.default_rng(P).standard_normal((T, E)))
    ref = pd.lightning(x.astype(np.float64), m, {k: v.astype(np.float64) for k, v in w.items()}, "", 1e-5)
    part = MIXERS.get("lightning_attention")(hidden_size=E, heads=H, head_dim=D, value_dim=P, decay=m["decay"], norm_eps=1e-5)
    rt = load_part(part, w, torch_type(dtype))
    for portions in ([T], [70, 2, 2, 40], [1, 1, 64]):
        close(run_part(part, rt, x, portions, E), ref, dtype, f"portions {portions}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("split_steps", [False, True])
@pytest.mark.parametrize("H,G,D,P,taps,ra,rg", [(1, 1, 8, 8, 4, 8, 8), (4, 2, 12, 20, 3, 5, 7), (3, 3, 32, 64, 1, 24, 16), (6, 2, 64, 33, 2, 3, 40), (2, 1, 100, 72, 6, 16, 4),
                                                (2, 2, 128, 128, 4, 32, 32), (1, 1, 200, 24, 4, 8, 12), (5, 1, 18, 10, 9, 11, 1)])
def test_the_delta_rule_with_a_decay_a_channel(dtype, split_steps, H, G, D, P, taps, ra, rg):
    """Every convolution width down to one tap, heads that share q and k, low ranks nothing divides; single rows through the one-launch step
    and through the kernels of a prompt step."""
    from borrowed_compute_b200.parts import MIXERS, channel_delta

    E, T = 48, 150
    m = pd.delta_mixer(H, G, D, P, taps, ra, rg)
    w = weights_of(m, E, D + P)
    x = pd.to_bf16(np.random.default_rng(P).standard_normal((T, E)))
    ref = pd.channel_delta(x.astype(np.float64), m, {k: v.astype(np.float64) for k, v in w.items()}, "", 1e-3)
    part = MIXERS.get("channel_delta")(hidden_size=E, heads=H, kv_heads=G, head_dim=D, value_dim=P, taps=taps, decay_rank=ra, gate_rank=rg, norm_eps=1e-3)
    rt = load_part(part, w, torch_type(dtype))
    channel_delta.split_steps = split_steps
    for portions in ([T], [70, 2, 2, 40], [1, 1, 1, 3, 64]):
        close(run_part(part, rt, x, portions, E), ref, dtype, f"portions {portions}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_lost_state_shows(dtype):
    """A channel that never forgets carries the first token's write past hundreds of others: the last rows change when it is left out."""
    from borrowed_compute_b200.parts import MIXERS

    E, T = 32, 400
    m = pd.delta_mixer(2, 2, 16, 16, 2, 8, 8)
    w = weights_of(m, E, 5)
    w["A_log"], w["dt_bias"] = pd.to_bf16(np.full(2, -6.0)), pd.to_bf16(np.full(32, -4.0))
    w["b"] = pd.to_bf16(np.zeros((2, E)))
    w["b"][:, 0] = 8.0                                       # only rows with channel 0 set write (and only the first row has it)
    x = np.random.default_rng(0).standard_normal((T, E)) * 0.5
    x[:, 0], x[0, 0] = -2.0, 3.0
    x = pd.to_bf16(x)
    t64 = {k: v.astype(np.float64) for k, v in w.items()}
    ref = pd.channel_delta(x.astype(np.float64), m, t64, "", 1e-6)
    lost = pd.channel_delta(x[1:].astype(np.float64), m, t64, "", 1e-6)
    assert np.abs(ref[-1] - lost[-1]).max() > 0.3 * np.abs(ref).max()
    part = MIXERS.get("channel_delta")(hidden_size=E, heads=2, kv_heads=2, head_dim=16, value_dim=16, taps=2, decay_rank=8, gate_rank=8, norm_eps=1e-6)
    rt = load_part(part, w, torch_type(dtype))
    for portions in ([T], [1, 300], [2, 2, 100]):
        close(run_part(part, rt, x, portions, E), ref, dtype, f"portions {portions}")


def diff_part(m, E, eps, own_kv=True):
    from borrowed_compute_b200.parts import MIXERS

    position = {"kind": "none"}
    if m.get("rot"):
        position = {"kind": "rotary", "head_dim": m["rot"]["dims"], "theta": m["rot"]["base"], "pairing": "half", "max_positions": 1024}
        if m["rot"].get("scaling"):
            sc = m["rot"]["scaling"]
            position["scaling"] = {"rope_type": "llama3", "factor": sc["factor"], "low_freq_factor": sc["low"], "high_freq_factor": sc["high"],
                                   "original_max_position_embeddings": sc["original"]}
    mask = m.get("mask") or {"size": 0}
    return MIXERS.get("differential_attention")(hidden_size=E, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], norm_eps=eps,
                                                diff=m["diff"], position=position, scale=m["scale"], window=mask["size"], keep_first=mask.get("keep_first", 0),
                                                own_kv=own_kv)


def plain_diff(x, m, w, eps):
    t = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    x = np.asarray(x, dtype=np.float64)
    return pd.attention(x, m, t, "", eps, pd.keys_values(x, m, t, "", eps))


def planted_diff(rng, m, E, star, T, which):
    """Weights and inputs of one differential mixer in which position ``star``'s key wins map ``which``'s softmax wherever it is seen: input
    channel 0 is zero but at ``star`` and drives that key map along a direction of the dimensions that do not turn; input channel 1 (one
    everywhere) drives that query map along the same direction.  The other map sees ordinary keys."""
    H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]["dims"] if m.get("rot") else 0
    w = weights_of(dict(m), E, int(rng.integers(1000)))
    q, k = w["q"].reshape(H, 2, d, E), w["k"].reshape(G, 2, d, E)
    q[..., :2], k[..., :2] = 0.0, 0.0
    for g in range(G):
        u = np.zeros(d)
        u[rot:] = rng.choice([-1.0, 1.0], d - rot)
        k[g, which, :, 0] = 3.0 * u
        for h in range(g * (H // G), (g + 1) * (H // G)):
            q[h, which, :, 1] = 6.0 * u
    w["q.norm"], w["k.norm"] = np.ones(d, dtype=np.float32), np.ones(d, dtype=np.float32)
    w["v"][:, :2] = 0.0
    w["lq2"], w["lq1"], w["lk1"] = 0.0 * w["lq2"], np.full(d, 0.4 / d), np.ones(d)      # lambda = e^0.4 - 1 + diff: both maps count
    x = rng.standard_normal((T, E)) * 0.5
    x[:, 0], x[:, 1] = 0.0, 1.0
    x[star, 0] = 8.0
    return {n: pd.to_bf16(a) for n, a in w.items()}, pd.to_bf16(x)


DIFF_PATHS = [("float32", "rows"), ("bfloat16", "rows"), ("bfloat16", "tiles"), ("bfloat16", "tc")]


def takes(part, rt, path):
    from borrowed_compute_b200 import StepEntry
    from borrowed_compute_b200.parts import diff_attention

    diff_attention.force = path
    return part.path(context([StepEntry(0, [0] * 40)], [0]), rt.dtype) == path


@pytest.mark.parametrize("dtype,path", DIFF_PATHS)
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("window,keep,star", [(9, 0, 5), (9, 0, 63), (1, 0, 64), (64, 0, 63), (64, 2, 64), (70, 0, 127), (9, 3, 2), (9, 3, 3), (40, 64, 63),
                                              (40, 65, 64), (33, 70, 69), (200, 4, 10), (129, 1, 0)])
def test_one_key_that_matters_at_every_edge(dtype, path, which, window, keep, star):
    """Rows that see the planted key take its value in one map, the row just past the window's edge does not, unless the key is one of the
    kept first positions: in a whole prompt, in portions of two and more rows whose borders fall beside the key, the edge and the pages'
    borders, and row by row."""
    E, T = 48, 300
    m = pd.attention_mixer(4, 2, 64, 64, window, keep, 16, 10000.0, scale=14.0 / 64, diff=0.4)
    w, x = planted_diff(np.random.default_rng(window * 7 + keep + star), m, E, star, T, which)
    ref = plain_diff(x, m, w, 1e-5)
    edge = star + window
    if edge + 1 < T:
        longer = plain_diff(x, dict(m, mask={"size": window + 1, "keep_first": keep}), w, 1e-5)
        assert (np.abs(longer[edge] - ref[edge]).max() > 0.05 * np.abs(ref).max()) == (star >= keep)
    part = diff_part(m, E, 1e-5)
    rt = load_part(part, w, torch_type(dtype))
    if not takes(part, rt, path):
        pytest.skip("these sizes do not take this path")
    for portions in ([T], [star + 1], [max(star, 1), 2, 2], [2, 61, 3, 62, 2, 9, 64]):
        close(run_part(part, rt, x, portions, E, spoil=True), ref, dtype, f"portions {portions}")


@pytest.mark.parametrize("dtype,path", DIFF_PATHS)
@pytest.mark.parametrize("H,G,D,DV,rot,window,keep", [(1, 1, 8, 8, 8, 0, 0), (6, 2, 40, 24, 20, 100, 5), (5, 1, 10, 6, 4, 50, 1), (3, 3, 128, 256, 64, 64, 64), (16, 4, 64, 128, 32, 77, 0),
                                                      (5, 1, 48, 80, 16, 300, 7), (8, 8, 24, 40, 24, 31, 2), (40, 2, 64, 64, 0, 90, 33), (2, 2, 128, 128, 0, 0, 0),
                                                      (4, 2, 128, 64, 128, 65, 3), (3, 1, 64, 200, 0, 128, 70)])
def test_differential_attention_in_other_sizes(dtype, path, H, G, D, DV, rot, window, keep):
    """One head; groups of many heads; widths that are no power of two, values wider and narrower than a map; everything turning, or nothing;
    stretched frequencies."""
    E, T = 40, 150
    m = pd.attention_mixer(H, G, D, DV, window, keep, rot, 300.0, (4.0, 1.0, 4.0, 100), diff=0.6)
    w = weights_of(m, E, H + D)
    x = pd.to_bf16(np.random.default_rng(D).standard_normal((T, E)))
    ref = plain_diff(x, m, w, 1e-6)
    part = diff_part(m, E, 1e-6)
    rt = load_part(part, w, torch_type(dtype))
    if not takes(part, rt, path):
        pytest.skip("these sizes do not take this path")
    for portions in ([T], [70, 40, 2]):
        mostly_close(run_part(part, rt, x, portions, E, spoil=True), ref, dtype, f"portions {portions}")


@pytest.mark.parametrize("splits", [1, 2, 3, 7])
@pytest.mark.parametrize("window,keep", [(0, 0), (130, 5), (64, 70)])
def test_pages_of_single_rows_shared_out_over_blocks(splits, window, keep):
    """More blocks than pages, too: the merge takes what each left, in order, and blocks without a page leave nothing."""
    from borrowed_compute_b200.parts import diff_attention

    E, T = 40, 210
    m = pd.attention_mixer(6, 2, 32, 48, window, keep, 16, 300.0)
    w = weights_of(m, E, 3)
    x = pd.to_bf16(np.random.default_rng(1).standard_normal((T, E)))
    part = diff_part(m, E, 1e-6)
    rt = load_part(part, w, torch.bfloat16)
    diff_attention.force_splits = splits
    close(run_part(part, rt, x, [1, 60], E, spoil=True), plain_diff(x, m, w, 1e-6), "bfloat16")


def test_stretched_frequencies_at_and_between_the_rules_borders():
    from borrowed_compute_b200.parts.rope import inverse_frequencies

    rot = {"dims": 40, "base": 5000.0, "scaling": {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 512}}
    got = inverse_frequencies(40, 5000.0, {"rope_type": "llama3", "factor": 6.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0, "original_max_position_embeddings": 512})
    want, plain = pd.frequencies(rot), pd.frequencies(dict(rot, scaling=None))
    kinds = {"kept": np.isclose(want, plain).sum(), "slowed": np.isclose(want, plain / 6.0).sum()}
    assert kinds["kept"] > 2 and kinds["slowed"] > 2 and kinds["kept"] + kinds["slowed"] < 20
    assert np.allclose(got.numpy(), want, rtol=1e-6)


# ------------------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_the_stream_after_every_layer(name, dtype):
    eng, cfg, w = small(name, dtype)
    toks = tokens_for(cfg, 150, seed=1)
    got = []
    ref, streams = pd.forward(cfg, w, toks)
    eng.model.after_run = lambda i, res: got.append(res.detach().float().cpu().numpy().copy())
    try:
        out = run_whole(eng, toks)
    finally:
        eng.model.after_run = None
    assert len(got) == len(streams)
    for i, (g, s) in enumerate(zip(got, streams)):
        mostly_close(g[: len(toks)], s, dtype, f"the stream after layer {i}")
    mostly_close(out, ref, dtype, "scores")
    for n in (1, 2, 3):            # the first tokens of a sequence, alone
        mostly_close(run_whole(eng, toks[:n]), ref[:n], dtype, f"a prompt of {n}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prefill_against_token_by_token_and_portions(name, dtype):
    """The windows pass over decoded tokens, the kept first positions stay, pages fill and are let go; a layer reads another's pages."""
    eng, cfg, w = small(name, dtype)
    toks = tokens_for(cfg, 200, seed=2)
    ref = pd.logits(cfg, w, toks)
    for cuts in ([], [120], [2, 2, 60, 3, 64, 1, 2, 40], [64, 64], [63, 2, 63], [199]):
        mostly_close(run_cut(eng, toks, cuts), ref, dtype, f"portions {cuts}")
    eng.cache.slots.check()


@pytest.mark.parametrize("name", NAMES)
def test_batches_give_the_same_bits_in_float32(name):
    from borrowed_compute_b200.engine import StepEntry

    eng, cfg, w = small(name, "float32")
    toks = tokens_for(cfg, 140, seed=3)
    whole = run_whole(eng, toks)
    others = [tokens_for(cfg, n, seed=4 + n) for n in (5, 90)]
    slots = [eng.acquire() for _ in range(3)]
    out = eng.step([StepEntry(slots[0], others[0], (4,)), StepEntry(slots[1], toks, tuple(range(len(toks)))), StepEntry(slots[2], others[1], ())]).cpu().numpy()
    for s in slots:
        eng.release(s)
    assert np.array_equal(out[1:], whole)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_against_each_alone_then_decoded_together(name, dtype):
    from borrowed_compute_b200.engine import StepEntry

    eng, cfg, w = small(name, dtype)
    lengths, tail = [1, 37, 130, 66], 40
    seqs = [tokens_for(cfg, n + tail, seed=10 + n) for n in lengths]
    refs = [pd.logits(cfg, w, s) for s in seqs]
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
        wanted = [i for i in live if not (t % 7 == 3 and i == live[0])]          # now and then one asks for nothing
        out = eng.step([StepEntry(slots[i], [seqs[i][lengths[i] + t]], (0,) if i in wanted else ()) for i in live]).cpu().numpy()
        for k, i in enumerate(wanted):
            rows[i].append(out[k:k + 1])
        for i in live:
            if i not in wanted:
                rows[i].append(refs[i][lengths[i] + t][None])
    for i in live:
        eng.release(slots[i])
    for i, r in enumerate(rows):
        got = np.concatenate(r)
        mostly_close(got, refs[i][: len(got)], dtype, f"sequence {i}")
    eng.cache.slots.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_step_that_asks_for_nothing(dtype):
    from borrowed_compute_b200.engine import StepEntry

    eng, cfg, w = small("A", dtype)
    toks = tokens_for(cfg, 60, seed=5)
    ref = pd.logits(cfg, w, toks)
    s = eng.acquire()
    assert eng.step([StepEntry(s, toks[:40], ())]).shape == (0, cfg["vocab"])
    assert eng.step([StepEntry(s, toks[40:41], ())]).shape == (0, cfg["vocab"])
    out = eng.step([StepEntry(s, toks[41:], (0, 18))]).cpu().numpy()
    eng.release(s)
    mostly_close(out, ref[[41, 59]], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_slots_and_pages_used_again(name, dtype):
    """What a sequence left behind (pages, states, the convolutions' last inputs) does not reach the next one in its slot."""
    eng, cfg, w = small(name, dtype)
    a, b = tokens_for(cfg, 190, seed=20), tokens_for(cfg, 75, seed=21)
    ref_a, ref_b = pd.logits(cfg, w, a), pd.logits(cfg, w, b)
    for _ in range(3):
        mostly_close(run_cut(eng, a, [100]), ref_a, dtype, "the long one")
        mostly_close(run_cut(eng, b, [3, 70]), ref_b, dtype, "the short one in the same slot")
    eng.cache.slots.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding_far_past_the_windows(name, dtype):
    eng, cfg, w = small(name, dtype)
    toks = tokens_for(cfg, 420, seed=30)
    mostly_close(run_cut(eng, toks, [20]), pd.logits(cfg, w, toks), dtype)


def test_a_cut_back_is_refused_unless_to_the_start():
    from borrowed_compute_b200.config import CacheError
    from borrowed_compute_b200.engine import StepEntry

    eng, cfg, w = small("A", "float32")
    toks = tokens_for(cfg, 30, seed=31)
    s = eng.acquire()
    first = eng.step([StepEntry(s, toks, (29,))]).cpu().numpy()
    with pytest.raises(CacheError, match="keeps per-sequence"):
        eng.rollback(s, 10)
    eng.rollback(s, 0)
    assert np.array_equal(eng.step([StepEntry(s, toks, (29,))]).cpu().numpy(), first)
    eng.release(s)


@pytest.mark.parametrize("seed", range(14))
def test_drawn_configurations(seed):
    """Sizes, constants and the order of layers drawn at random, in float32: whole, in portions, and token by token."""
    rng = np.random.default_rng(1000 + seed)
    cfg = pd.draw_config(rng)
    w = pd.make_weights(cfg, seed)
    eng = engine_for(cfg, w, "float32", max_tokens=1024, max_slots=2, max_seq=512)
    toks = [int(t) for t in rng.integers(0, cfg["vocab"], 150)]
    ref = pd.logits(cfg, w, toks)
    close(run_whole(eng, toks), ref, "float32", f"whole, {json.dumps(cfg)}")
    close(run_cut(eng, toks, [2, 66, 30]), ref, "float32", f"portions, {json.dumps(cfg)}")


@pytest.mark.parametrize("seed", range(10))
def test_drawn_configurations_in_bfloat16(seed):
    """A drawn model may be badly conditioned (a head whose read-out nearly cancels, normed): it is held to five times what rounding the
    sublayers' inputs alone does to the oracle, if that is more than the usual tolerance."""
    rng = np.random.default_rng(2000 + seed)
    cfg = pd.draw_config(rng)
    w = pd.make_weights(cfg, seed)
    eng = engine_for(cfg, w, "bfloat16", max_tokens=1024, max_slots=2, max_seq=512)
    toks = tokens_for(cfg, 150, seed=seed)
    ref = pd.logits(cfg, w, toks)
    rounded = pd.logits(cfg, w, toks, round_to=lambda a: pd.to_bf16(a).astype(np.float64))
    least = 5.0 * float(np.quantile(np.abs(rounded - ref).max(axis=1), 0.9))
    mostly_close(run_whole(eng, toks), ref, "bfloat16", f"whole, {json.dumps(cfg)}", least)
    mostly_close(run_cut(eng, toks, [2, 66, 30]), ref, "bfloat16", f"portions, {json.dumps(cfg)}", least)


# ------------------------------------------------------------------ the entry points

def folder_for(tmp_path, name, seed):
    from borrowed_compute_b200.weights.safetensors_io import write_safetensors

    cfg = json.loads(json.dumps(pd.SMALL[name]))
    w = pd.make_weights(cfg, seed)
    for layer in cfg["layers"]:                  # a folder leaves the ranks to the tensors
        layer["mixer"].pop("decay_rank", None), layer["mixer"].pop("gate_rank", None)
    folder = str(tmp_path / f"duratar_{name}")
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {n: torch.from_numpy(np.asarray(a)).to(torch.bfloat16) for n, a in w.items()})
    return folder, cfg, w


def test_greedy_generation_through_the_library_and_the_command_line(tmp_path):
    from borrowed_compute_b200 import Local, Sampling

    folder, cfg, w = folder_for(tmp_path, "A", 41)
    prompts = [tokens_for(cfg, n, seed=50 + n) for n in (9, 30)]
    want = [pd.generate(cfg, w, p, 12) for p in prompts]
    local = Local.load(folder, dtype="float32", max_tokens=1024, max_slots=4, max_seq=256)
    out, stats = local.generate(prompts, 12, Sampling(), stop_ids=())
    assert [list(g) for g in out] == want and stats.generated == 24
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "bc-infer"), "generate", folder, ";".join(",".join(map(str, p)) for p in prompts),
                          "--max-tokens", "12", "--dtype", "float32", "--stop-ids", ""], capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [[int(t) for t in line.split(",")] for line in res.stdout.strip().splitlines()] == want
    # bfloat16 decodes through captured graphs: the tokens are the oracle's wherever its two best scores lie well apart
    out16, _ = Local.load(folder, dtype="bfloat16", max_tokens=1024, max_slots=4, max_seq=256).generate(prompts, 12, Sampling(), stop_ids=())
    for p, mine in zip(prompts, out16):
        toks = list(p)
        assert len(mine) == 12
        for t in mine:
            last = pd.logits(cfg, w, toks)[-1]
            best = np.sort(last)
            if best[-1] - best[-2] > 0.1 * (1.0 + np.abs(last).max()):
                assert t == int(last.argmax()), "a clear choice was missed"
            toks.append(int(t))


@pytest.mark.parametrize("dtype", DTYPES)
def test_replaying_steps_with_the_trace_tool(tmp_path, dtype):
    folder, cfg, w = folder_for(tmp_path, "B", 42)
    a, b = tokens_for(cfg, 80, seed=60), tokens_for(cfg, 33, seed=61)
    ref_a, ref_b = pd.logits(cfg, w, a), pd.logits(cfg, w, b)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:70], "want": [0, 69]}, {"id": "y", "tokens": b[:30], "want": [29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[70:71], "want": []}, {"id": "y", "tokens": b[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[71:72], "want": [0]}, {"id": "y", "tokens": b[31:32], "want": [0]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[72:73], "want": [0]}], "end": ["x"]}]
    out = str(tmp_path / "scores")
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out, "--max-tokens", "256"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [line for line in res.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda i: np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])      # noqa: E731
    assert not os.path.exists(os.path.join(out, "1.f32"))
    mostly_close(read(0), np.stack([ref_a[0], ref_a[69], ref_b[29]]), dtype, "step 0")
    mostly_close(read(2), np.stack([ref_a[71], ref_b[31]]), dtype, "step 2")
    mostly_close(read(3), ref_a[72:73], dtype, "step 3")
