"""A plain, slow NumPy restatement of the Duratar decoder, one function a mechanism, in float64.

It shares no code with the package: the tests hold the engine's kernels to it.  A model is a
config.json dictionary and a mapping from tensor names to arrays.  Notation: h [T, E] are the rows of
ONE sequence at positions 0 .. T-1; matrices are stored [out, in]; N(x) = x / sqrt(mean(x^2) + eps).

The stream of a row is a bundle of S copies X [S, E], at first all equal to N(embed[token]) * g0 (g0 one number).
A sublayer f (a mixer or a feed-forward) with connection (a [S], M [S, S], b [S]), norm number g and factors l [E]:
    u = a X,   y = l * f(N(u) * g),   X <- M^T X + b y^T.
At the end the copies are added up; scores = head (N(sum) * g1).

Mixer "attention" (H query heads on G key heads, two maps a head, map width d, value width v):
    q, k: every (head, map) over its own N times a shared weight [d]; the first dims of it rotated, pairs (i, i + dims/2);
    map m of head h:  A_m = softmax(scale q_{h,m} . k_{g,m}) V_g  over j <= i with i - j < size or j < keep_first;
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff;  o = N(A_1 - lambda A_2) (1 - diff);  Wo on the heads side by side.
    With kv_from the keys and values are another layer's.
Mixer "lightning":  q, k, v = silu(W. h);  S_t = c_h S_{t-1} + k v^T,  o = S_t^T q;  Wo (N(all heads) * w * sigmoid(Wg h)).
Mixer "channel_delta":  q, k, v through a causal convolution a channel and silu; q, k to unit length, q / sqrt(d);
    b = sigmoid(Wb h);  c = exp(-exp(A_h) softplus(Wa2 Wa1 h + t)) a key channel;
    S <- diag(c) S;  r = b (v - S^T k);  S <- S + k r^T;  o = S^T q;  Wo (N(o of a head) * w * sigmoid(Wg2 Wg1 h)).
Feed-forward:  Wdown act(Wup h), act(z) = sp(p) z^2 + z/2 above zero, (1/2 + sp(q)) (e^z - 1 - z) + z/2 below, sp = softplus.
"""

from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def over_rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


# ------------------------------------------------------------------------------------ the bundle of streams

def collapse(X, a):
    """X [S, T, E] -> [T, E]."""
    return np.tensordot(np.asarray(a, dtype=np.float64), X, axes=(0, 0))


def spread(X, y, M, b):
    """X_t <- sum_s M[s, t] X_s + b[t] y."""
    out = np.zeros_like(X)
    for t in range(X.shape[0]):
        for s in range(X.shape[0]):
            out[t] += M[s, t] * X[s]
        out[t] += b[t] * y
    return out


# ---------------------------------------------------------------------------------------------- attention

def frequencies(rot):
    """Radians a position for every rotated pair."""
    dims, out = int(rot["dims"]), []
    for i in range(dims // 2):
        f = float(rot["base"]) ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            turns = float(sc["original"]) * f / (2.0 * math.pi)      # how often the wave turns within the original positions
            if turns < sc["low"]:
                f = f / sc["factor"]
            elif turns <= sc["high"]:
                s = (turns - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return np.asarray(out, dtype=np.float64)


def rotate(x, pos, freqs):
    """x [..., T, d]: the first 2 len(freqs) dimensions turn."""
    n = len(freqs)
    ang = np.asarray(pos, dtype=np.float64)[:, None] * freqs[None, :]
    c, s = np.cos(ang), np.sin(ang)
    out = x.copy()
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def visible(T, mask, L=None):
    """[T, L] booleans: which of positions 0 .. L-1 position i sees."""
    i, j = np.arange(T)[:, None], np.arange(T if L is None else L)[None, :]
    see = j <= i
    if mask:
        see &= (i - j < mask["size"]) | (j < mask.get("keep_first", 0))
    return see


def softmax_rows(s, see):
    s = np.where(see, s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return p / p.sum(axis=-1, keepdims=True)


def head_maps(x, heads, dim):
    """[T, heads * 2 * dim] -> [heads, 2, T, dim]."""
    return x.reshape(x.shape[0], heads, 2, dim).transpose(1, 2, 0, 3)


def keys_values(h, m, t, p, eps):
    """The cached keys [G, 2, T, d] (normed and rotated) and values [G, T, v] of a layer."""
    G, d, v = m["kv_heads"], m["dim"], m["vdim"]
    k = over_rms(head_maps(h @ t[p + "k"].T, G, d), eps) * t[p + "k.norm"]
    if m.get("rot"):
        k = rotate(k, np.arange(h.shape[0]), frequencies(m["rot"]))
    return k, (h @ t[p + "v"].T).reshape(h.shape[0], G, v).transpose(1, 0, 2)


def lam(m, t, p):
    return float(np.exp((t[p + "lq1"] * t[p + "lk1"]).sum()) - np.exp((t[p + "lq2"] * t[p + "lk2"]).sum()) + m["diff"])


def combine_maps(a1, a2, lam_, diff, eps):
    return over_rms(a1 - lam_ * a2, eps) * (1.0 - diff)


def attention(h, m, t, p, eps, kv):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = over_rms(head_maps(h @ t[p + "q"].T, H, d), eps) * t[p + "q.norm"]
    if m.get("rot"):
        q = rotate(q, np.arange(T), frequencies(m["rot"]))
    k, v = kv
    see, l, out = visible(T, m.get("mask")), lam(m, t, p), []
    for n in range(H):
        g = n // (H // G)
        a = [softmax_rows(q[n, j] @ k[g, j].T * m["scale"], see) @ v[g] for j in range(2)]
        out.append(combine_maps(a[0], a[1], l, m["diff"], eps))
    return np.concatenate(out, axis=1) @ t[p + "o"].T


# --------------------------------------------------------------------------------------------- recurrences

def lightning_scan(q, k, v, decay, S=None):
    """q, k [T, H, d], v [T, H, P] -> o [T, H, P], S [H, d, P]."""
    S = np.zeros((q.shape[1], q.shape[2], v.shape[2])) if S is None else S.copy()
    c = np.asarray(decay, dtype=np.float64)[:, None, None]
    o = np.zeros(v.shape)
    for i in range(q.shape[0]):
        S = c * S + k[i][:, :, None] * v[i][:, None, :]
        o[i] = np.einsum("hdp,hd->hp", S, q[i])
    return o, S


def lightning(h, m, t, p, eps):
    T, H, d, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(h @ t[p + n].T).reshape(T, H, d) for n in ("q", "k"))
    v = silu(h @ t[p + "v"].T).reshape(T, H, P)
    o, _ = lightning_scan(q, k, v, m["decay"])
    return (over_rms(o.reshape(T, H * P), eps) * t[p + "norm"] * sigmoid(h @ t[p + "g"].T)) @ t[p + "o"].T


def short_conv(x, w, before=None):
    """x [T, C], w [C, taps] -> silu of the causal convolution; ``before``: the taps - 1 rows ahead of x."""
    taps = w.shape[1]
    pad = np.zeros((taps - 1, x.shape[1])) if before is None else np.asarray(before, dtype=np.float64)
    full = np.concatenate([pad, x], axis=0)
    return silu(sum(full[j:j + x.shape[0]] * w[:, j][None, :] for j in range(taps)))


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta_scan(q, k, v, c, b, S=None):
    """q, k, c [T, H, d], v [T, H, P], b [T, H] -> o [T, H, P], S [H, d, P]."""
    S = np.zeros((q.shape[1], q.shape[2], v.shape[2])) if S is None else S.copy()
    o = np.zeros(v.shape)
    for i in range(q.shape[0]):
        S = c[i][:, :, None] * S
        r = b[i][:, None] * (v[i] - np.einsum("hdp,hd->hp", S, k[i]))
        S = S + k[i][:, :, None] * r[:, None, :]
        o[i] = np.einsum("hdp,hd->hp", S, q[i])
    return o, S


def delta_inputs(h, m, t, p):
    """What enters the recurrence: q, k, c [T, H, d], v [T, H, P], b [T, H]."""
    T, H, G, d, P = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (unit(short_conv(h @ t[p + n].T, t[p + n + ".conv"]).reshape(T, G, d)) for n in ("q", "k"))
    v = short_conv(h @ t[p + "v"].T, t[p + "v.conv"]).reshape(T, H, P)
    q, k = (np.repeat(x, H // G, axis=1) for x in (q * d ** -0.5, k))
    c = np.exp(-np.exp(t[p + "A_log"])[None, :, None] * softplus((h @ t[p + "a1"].T) @ t[p + "a2"].T + t[p + "dt_bias"]).reshape(T, H, d))
    return q, k, c, v, sigmoid(h @ t[p + "b"].T)


def channel_delta(h, m, t, p, eps):
    T, H, P = h.shape[0], m["heads"], m["vdim"]
    q, k, c, v, b = delta_inputs(h, m, t, p)
    o, _ = delta_scan(q, k, v, c, b)
    gate = sigmoid((h @ t[p + "g1"].T) @ t[p + "g2"].T)
    return ((over_rms(o, eps) * t[p + "norm"]).reshape(T, H * P) * gate) @ t[p + "o"].T


# --------------------------------------------------------------------------------------------- feed-forward

def xielu(z, pq):
    p, q = float(pq[0]), float(pq[1])
    low = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z + 0.5 * z, (0.5 + softplus(q)) * (np.expm1(low) - low) + 0.5 * z)


def feed_forward(h, t, p):
    return xielu(h @ t[p + "up"].T, t[p + "act"]) @ t[p + "down"].T


# ------------------------------------------------------------------------------------------------ the model

def forward(cfg, tensors, tokens, round_to=None):
    """Scores [T, vocab] and the sum of the streams after every layer [layers, T, E].  ``round_to``: a function that rounds what a
    16-bit engine would keep in 16 bits between its kernels (normed inputs of the sublayers and of the head)."""
    t = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    eps, S = float(cfg["norm"]["eps"]), int(cfg["streams"])
    r = round_to or (lambda a: a)
    x0 = over_rms(t["embed"][np.asarray(tokens)], eps) * float(t["embed.norm"])
    X = np.repeat(x0[None], S, axis=0)
    kept, after = {}, []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = r(over_rms(collapse(X, t[p + "hc1.in"]), eps) * float(t[p + "norm1"]))
        if L["type"] == "attention":
            j = m.get("kv_from")
            if j is None:
                kept[i] = keys_values(h, m, t, p + "mix.", eps)
            y = attention(h, m, t, p + "mix.", eps, kept[i if j is None else j])
        else:
            y = {"lightning": lightning, "channel_delta": channel_delta}[L["type"]](h, m, t, p + "mix.", eps)
        X = spread(X, y * t[p + "ls1"], t[p + "hc1.mix"], t[p + "hc1.out"])
        if L.get("mlp"):
            h = r(over_rms(collapse(X, t[p + "hc2.in"]), eps) * float(t[p + "norm2"]))
            X = spread(X, feed_forward(h, t, p + "mlp.") * t[p + "ls2"], t[p + "hc2.mix"], t[p + "hc2.out"])
        after.append(X.sum(axis=0))
    return r(over_rms(X.sum(axis=0), eps) * float(t["final.norm"])) @ t["head"].T, np.stack(after)


def logits(cfg, tensors, tokens, round_to=None):
    return forward(cfg, tensors, tokens, round_to)[0]


def generate(cfg, tensors, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(np.argmax(logits(cfg, tensors, ids)[-1])))
    return ids[len(prompt):]


# ------------------------------------------------------------------------- small models and their weights

def to_bf16(a):
    """float32 values rounded to the nearest bfloat16 (ties to even)."""
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def attention_mixer(heads, kv_heads, dim, vdim, window=0, keep=0, rot=0, base=10000.0, scaling=None, scale=None, diff=0.5, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.5 / dim ** 0.5 if scale is None else scale, "diff": diff}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def lightning_mixer(heads, dim, vdim, slowest=0.99):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": [float(d) for d in np.linspace(0.5, slowest, heads)]}


def delta_mixer(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank, "gate_rank": gate_rank}


def model(vocab, width, streams, layers, eps=1e-5):
    """``layers``: (mixer, ff) pairs; the mixer's keys tell its type, ff 0 leaves the feed-forward out."""
    kind = lambda m: "lightning" if "decay" in m else "channel_delta" if "conv" in m else "attention"          # noqa: E731
    return {"architecture": "Duratar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "layers": [{"type": kind(m), "mixer": m, "mlp": {"kind": "dense", "ff": f} if f else None} for m, f in layers]}


SMALL = {
    # three streams; shared keys under a wider window than their owner's; shared delta keys; a layer without a feed-forward
    "A": model(131, 72, 3, [
        (attention_mixer(4, 2, 16, 24, 24, 3, 8, 500.0, (3.0, 1.0, 4.0, 60)), 40),
        (delta_mixer(4, 2, 12, 20, 4, 8, 16), 56),
        (attention_mixer(4, 2, 16, 24, 50, 5, 8, 500.0, (3.0, 1.0, 4.0, 60), diff=0.3, kv_from=0), 0),
        (lightning_mixer(3, 16, 12), 40)]),
    # one stream, one head, no mask, no rotation, a convolution of one tap, widths that nothing divides
    "B": model(97, 50, 1, [
        (lightning_mixer(2, 10, 14), 22),
        (attention_mixer(3, 1, 10, 6, diff=0.2), 30),
        (delta_mixer(3, 1, 18, 10, 1, 5, 3), 0),
        (attention_mixer(3, 1, 10, 6, 70, 66, diff=0.7, kv_from=1), 26),
        (delta_mixer(1, 1, 6, 7, 2, 4, 8), 22)], eps=1e-6),
    # widths the tensor-core kernels take
    "C": model(200, 128, 2, [
        (attention_mixer(4, 2, 64, 128, 100, 66, 32, 10000.0), 96),
        (attention_mixer(4, 2, 64, 128, 0, 0, 32, 10000.0, kv_from=0), 64),
        (delta_mixer(2, 2, 64, 64, 3, 16, 24), 96),
        (attention_mixer(2, 1, 48, 40, 65, 2, 48, 300.0), 64),
        (lightning_mixer(2, 128, 64, 0.995), 96)]),
}


def tensor_shapes(cfg):
    E, S, V = cfg["width"], cfg["streams"], cfg["vocab"]
    out = {"embed": (V, E), "embed.norm": (), "final.norm": (), "head": (V, E)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        for n in ("1", "2") if L.get("mlp") else ("1",):
            out.update({p + "norm" + n: (), p + "ls" + n: (E,), p + f"hc{n}.in": (S,), p + f"hc{n}.out": (S,), p + f"hc{n}.mix": (S, S)})
        H, d, v = m["heads"], m["dim"], m["vdim"]
        out[x + "o"] = (E, H * v)
        if L["type"] == "attention":
            out.update({x + "q": (2 * H * d, E), x + "q.norm": (d,), **{x + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")}})
            if m.get("kv_from") is None:
                G = m["kv_heads"]
                out.update({x + "k": (2 * G * d, E), x + "k.norm": (d,), x + "v": (G * v, E)})
        elif L["type"] == "lightning":
            out.update({x + "q": (H * d, E), x + "k": (H * d, E), x + "v": (H * v, E), x + "g": (H * v, E), x + "norm": (H * v,)})
        else:
            G, taps = m["kv_heads"], m["conv"]
            out.update({x + "q": (G * d, E), x + "k": (G * d, E), x + "v": (H * v, E), x + "q.conv": (G * d, taps), x + "k.conv": (G * d, taps),
                        x + "v.conv": (H * v, taps), x + "b": (H, E), x + "A_log": (H,), x + "norm": (v,), x + "dt_bias": (H * d,),
                        x + "a1": (m["decay_rank"], E), x + "a2": (H * d, m["decay_rank"]), x + "g1": (m["gate_rank"], E), x + "g2": (H * v, m["gate_rank"])})
        if L.get("mlp"):
            f = L["mlp"]["ff"]
            out.update({p + "mlp.up": (f, E), p + "mlp.down": (E, f), p + "mlp.act": (2,)})
    return out


def make_weights(cfg, seed):
    """Random weights that bfloat16 holds exactly: matrices of spread 1 / sqrt(inputs), norm numbers around one, connections that mix the
    streams well, channels of the delta rule that forget within a few to a few hundred tokens."""
    rng, t = np.random.default_rng(seed), {}
    S = cfg["streams"]
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if "norm" in name:
            a = 1.0 + 0.3 * rng.uniform(-1, 1, shape)
        elif last in ("ls1", "ls2"):
            a = rng.uniform(0.4, 1.2, shape)
        elif last == "in":
            a = rng.uniform(0.3, 1.4, shape) / S
        elif last == "out":
            a = rng.uniform(0.5, 1.2, shape)
        elif last == "mix":
            a = 0.75 * np.eye(S) + 0.25 * rng.standard_normal((S, S)) / math.sqrt(S)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            a = 0.5 * rng.standard_normal(shape) / shape[0] ** 0.25
        elif last == "A_log":
            a = rng.uniform(-2.0, 1.0, shape)
        elif last == "dt_bias":
            a = rng.uniform(-5.0, -1.0, shape)
        elif last == "act":
            a = rng.uniform(-1.5, 1.5, shape)
        elif last == "conv":
            a = rng.uniform(-0.6, 0.6, shape)
            a[:, -1] += 0.8
        elif name == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / math.sqrt(shape[-1]) * (2.0 if last in ("head", "g", "g2", "a2", "b") else 1.0)
        t[name] = to_bf16(a)
    return t


def draw_config(rng):
    """A configuration whose sizes, constants and order of layers are drawn."""
    E, layers, owners = int(rng.choice([24, 40, 56, 64, 72, 128])), [], []
    for i in range(int(rng.integers(2, 6))):
        u = rng.random()
        if u < 0.45:
            if owners and rng.random() < 0.5:
                j = int(rng.choice(owners))
                m = dict(layers[j][0], kv_from=j, diff=float(rng.choice([0.1, 0.8])))
                m.pop("mask", None)
                if rng.random() < 0.8:
                    m["mask"] = {"size": int(rng.choice([1, 7, 64, 90])), "keep_first": int(rng.choice([0, 2, 65]))}
            else:
                G, d = int(rng.choice([1, 2, 3])), int(rng.choice([8, 10, 16, 40, 48, 64, 128]))
                scaling = (float(rng.choice([2.0, 8.0])), 1.0, float(rng.choice([2.0, 4.0])), int(rng.choice([32, 64, 300]))) if rng.random() < 0.6 else None
                m = attention_mixer(G * int(rng.choice([1, 2, 3, 5])), G, d, int(rng.choice([6, 8, 24, 64, 104, 128])), int(rng.choice([0, 1, 5, 33, 64, 100])),
                                    int(rng.choice([0, 1, 4, 64, 66])), int(rng.choice([0, d // 2 // 2 * 2, d])), float(rng.choice([100.0, 10000.0])), scaling,
                                    diff=float(rng.choice([0.2, 0.5, 0.8])))
                owners.append(i)
        elif u < 0.7:
            m = lightning_mixer(int(rng.choice([1, 2, 5])), int(rng.choice([6, 8, 16, 40, 130])), int(rng.choice([4, 12, 33, 64])), float(rng.choice([0.9, 0.999])))
        else:
            G = int(rng.choice([1, 2]))
            m = delta_mixer(G * int(rng.choice([1, 2, 3])), G, int(rng.choice([6, 8, 16, 20, 64, 100])), int(rng.choice([5, 8, 32, 72])), int(rng.choice([1, 2, 3, 4, 6])),
                            int(rng.choice([3, 8, 24])), int(rng.choice([4, 16, 20])))
        layers.append((m, int(rng.choice([0, 8, 20, 48]))))
    return model(int(rng.choice([50, 131, 200])), E, int(rng.choice([1, 2, 4, 5, 9])), layers, eps=float(rng.choice([1e-6, 1e-5, 1e-3])))
