"""A plain, slow NumPy restatement of the Kodulix decoder, one function a mechanism, in float64.

It shares no code with the package: the tests hold the engine's kernels to it.  A model is a
config.json dictionary and a mapping from tensor names to arrays.  Notation: x is the residual
stream [T, E] of ONE sequence whose rows are positions 0 .. T-1; matrices are stored [out, in].

Entry:     x_p = embed[t_p] + bigram[b_p] + s_p;   b_0 = N (the last row), b_p = (t_{p-1} a + t_p c) mod N for a table of N + 1 rows;
           s_p holds sin(p f_i) at 2i and cos(p f_i) at 2i + 1 with f_i = 10000^(-2i/E).

A layer:   x <- x + m N1(mixer(x));  x <- x + m N2(ff(x)),   N(x) = x / rms(x) * (1 + w): no norm ahead of a sublayer.

Mixer (H query heads on G key heads, widths d and dv):
    q = Nq(Wq x) tau_p, k = Nk(Wk x), v = Wv x   (Nq, Nk: RMS norm of every head, plain weights shared by the heads)
    tau_p = 1 + coef ln(floor((p + 1) / every) + 1)
    s_h(i, j) = scale q_h(i) . k_g(j) + R[beta(i - j), h],  j <= i;  softmax;  Wo on the heads side by side.
    beta(n) over B rows, h = B/2: n below h, then h + floor((B - h) ln(n / h) / ln(D / h)), at most B - 1.

Feed-forward: p = softmax(Wr x) over n experts and e identities; choice scores p + c; neighbours form groups whose score is their
    largest choice score, only the best ``keep`` groups stand; the ``top`` largest choice scores choose; weights p / (sum + 1e-20);
    sum of weight * expert(x), an identity being x itself, plus shared(x).
    expert(x) = Wdown (g sigmoid(1.702 g) (u + 1)), g = min(Wgate x, L), u = clip(Wup x, -L, L).

Output: N(x) with ``final.norm``, scores = embed N(x) * logit_scale.
"""

from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms(x, eps):
    return np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """x over its root mean square, times (1 + w): the weight is stored around zero."""
    return x / rms(x, eps) * (1.0 + w)


def plain_norm(x, w, eps):
    return x / rms(x, eps) * w


# ------------------------------------------------------------------------------- what enters

def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """The table row of every position: a hash of the token before and the token itself; row ``buckets`` opens a sequence."""
    rows = [buckets]
    for before, here in zip(tokens[:-1], tokens[1:]):
        rows.append((int(before) * int(mul_prev) + int(here) * int(mul_cur)) % buckets)
    return np.asarray(rows, dtype=np.int64)


def sinusoid(positions, width):
    out = np.zeros((len(positions), width))
    for r, p in enumerate(positions):
        for c in range(width):
            angle = float(p) * 10000.0 ** (-2.0 * (c // 2) / width)
            out[r, c] = math.sin(angle) if c % 2 == 0 else math.cos(angle)
    return out


def embedded(cfg, t, tokens):
    tokens = np.asarray(tokens, dtype=np.int64)
    x = t["embed"][tokens]
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram:
        x = x + t["bigram"][bigram_rows(tokens, int(bigram["buckets"]), bigram["mul_prev"], bigram["mul_cur"])]
    return x + sinusoid(range(len(tokens)), int(cfg["width"]))


# ---------------------------------------------------------------------------------- attention

def query_temperature(positions, coef, every):
    return np.asarray([1.0 + float(coef) * math.log((int(p) + 1) // int(every) + 1.0) for p in positions])


def distance_bucket(n, rows, reach):
    """Which of ``rows`` entries a distance n falls into: one each below rows/2, then logarithmically wider ones up to ``reach``.

    floor((B - h) ln(n/h) / ln(D/h)) >= k exactly when (n/h)^(B - h) >= (D/h)^k: whole numbers decide, nothing is rounded."""
    half = rows // 2
    if n < half:
        return n
    k = 0
    while half + k + 1 < rows and n ** (rows - half) * half ** (k + 1) >= reach ** (k + 1) * half ** (rows - half):
        k += 1
    return half + k


def bias_matrix(rel, T, reach):
    """[H, T, T]: the bias of query i and key j <= i (0 elsewhere)."""
    by_distance = np.stack([rel[distance_bucket(n, rel.shape[0], reach)] for n in range(T)])      # [T, H]
    n = np.arange(T)[:, None] - np.arange(T)[None, :]
    return np.where(n[None] >= 0, by_distance[np.maximum(n, 0)].transpose(2, 0, 1), 0.0)


def softmax_rows(s, ok):
    s = np.where(ok, s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return p / p.sum(axis=-1, keepdims=True)


def attention(x, m, t, pre, eps):
    T = x.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = plain_norm((x @ t[pre + "q"].T).reshape(T, H, d), t[pre + "q.norm"], eps)
    k = plain_norm((x @ t[pre + "k"].T).reshape(T, G, d), t[pre + "k.norm"], eps)
    v = (x @ t[pre + "v"].T).reshape(T, G, dv)
    temp = m.get("q_temp")
    if temp:
        q = q * query_temperature(range(T), temp["coef"], temp["every"])[:, None, None]
    bias = bias_matrix(t[pre + "rel"], T, int(m["bias_max"]))
    ok = np.arange(T)[None, :] <= np.arange(T)[:, None]
    out = np.zeros((T, H, dv))
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * float(m["scale"]) + bias[h]
        out[:, h] = softmax_rows(s, ok) @ v[:, g]
    return out.reshape(T, H * dv) @ t[pre + "o"].T


# ------------------------------------------------------------------------------- feed-forward

def clipped_glu(x, t, pre, limit):
    g = np.minimum(x @ t[pre + "gate"].T, float(limit))
    u = np.clip(x @ t[pre + "up"].T, -float(limit), float(limit))
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ t[pre + "down"].T


def route(x, router, correction, top, groups=1, keep=1):
    """(choices [T, top], weights [T, top]) of the rows of x; the lower index wins a tie."""
    z = x @ router.T
    p = np.exp(z - z.max(axis=-1, keepdims=True))
    p = p / p.sum(axis=-1, keepdims=True)
    choices, weights = [], []
    for row in p:
        c = row + correction
        size = len(c) // groups
        best = sorted(range(groups), key=lambda g: (-c[g * size:(g + 1) * size].max(), g))[:keep]
        allowed = [e for e in range(len(c)) if e // size in best]
        mine = sorted(allowed, key=lambda e: (-c[e], e))[:top]
        choices.append(mine)
        weights.append(row[mine] / (row[mine].sum() + 1e-20))
    return np.asarray(choices), np.asarray(weights)


def experts(x, mlp, t, pre):
    r = mlp["router"]
    n = int(r["experts"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    choices, weights = route(x, t[pre + "router"], t[pre + "correction"], int(r["top"]), int(groups["count"]), int(groups["keep"]))
    out = np.zeros_like(x)
    for i in range(x.shape[0]):
        for e, w in zip(choices[i], weights[i]):
            y = x[i] if e >= n else clipped_glu(x[i:i + 1], t, f"{pre}e{e}.", mlp["expert"]["limit"])[0]
            out[i] += w * y
    if mlp.get("shared"):
        out = out + clipped_glu(x, t, pre + "shared.", mlp["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------------- whole

def forward(cfg, weights, tokens, routed=None):
    """(scores [T, vocab], streams after every layer [layers, T, E]); ``routed`` (a list) receives (layer, what its feed-forward reads)."""
    t = {n: np.asarray(w, dtype=np.float64) for n, w in weights.items()}
    eps, m = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = embedded(cfg, t, tokens)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + m * offset_norm(attention(x, layer["mixer"], t, p + "mix.", eps), t[p + "norm1"], eps)
        if layer.get("mlp"):
            if routed is not None:
                routed.append((i, x))
            x = x + m * offset_norm(experts(x, layer["mlp"], t, p + "mlp."), t[p + "norm2"], eps)
        after.append(x)
    scores = offset_norm(x, t["final.norm"], eps) @ t["embed"].T * float(cfg.get("logit_scale", 1.0))
    return scores, np.stack(after)


def generate(cfg, weights, prompt, n):
    """Greedy generation, the whole sequence again for every token."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(np.argmax(forward(cfg, weights, tokens)[0][-1])))
    return tokens[len(prompt):]


def choice_margin(scores, top, groups=1, keep=1):
    """How far a row of choice scores is from another choice: the gap between the last group kept and the first left out, and
    between the last expert chosen and the first left out of those groups."""
    size = len(scores) // groups
    best = np.sort(scores.reshape(groups, size).max(axis=1))[::-1]
    order = sorted(range(groups), key=lambda g: -scores[g * size:(g + 1) * size].max())[:keep]
    within = np.sort(np.concatenate([scores[g * size:(g + 1) * size] for g in order]))[::-1]
    gap = best[keep - 1] - best[keep] if keep < groups else math.inf
    return min(gap, within[top - 1] - within[top] if top < len(within) else math.inf)


def row_margins(cfg, weights, tokens):
    """For every position, the smallest choice margin over the layers: a row with a wide one chooses the same experts under rounding."""
    routed = []
    forward(cfg, weights, tokens, routed)
    out = np.full(len(tokens), math.inf)
    for i, x in routed:
        mlp, pre = cfg["layers"][i]["mlp"], f"l{i}.mlp."
        groups = mlp["router"].get("groups") or {"count": 1, "keep": 1}
        z = x @ np.asarray(weights[pre + "router"], dtype=np.float64).T
        p = np.exp(z - z.max(axis=-1, keepdims=True))
        c = p / p.sum(axis=-1, keepdims=True) + np.asarray(weights[pre + "correction"], dtype=np.float64)
        out = np.minimum(out, [choice_margin(row, mlp["router"]["top"], groups["count"], groups["keep"]) for row in c])
    return out


# ----------------------------------------------------------------------- small models for tests

def to_bf16(a):
    """Nearest values that bfloat16 holds (ties to even), as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32).reshape(np.shape(a))


def mixer(heads, kv_heads, dim, vdim, rows, reach, scale=None, temp=(0.5, 7)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "bias_rows": rows, "bias_max": reach}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def moe(experts, top, ff, limit, identity=0, groups=None, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "identity": identity}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        f["shared"] = {"ff": shared[0], "limit": shared[1]}
    return f


def model(vocab, width, layers, eps=1e-5, residual_mult=1.0, logit_scale=1.0, bigram=(101, 13, 5)):
    return {"architecture": "Kodulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": residual_mult, "logit_scale": logit_scale,
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))} if bigram else {},
            "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


# Two small models that differ in every size and constant, in what their layers have and in what they leave out.
SMALL = {
    "A": model(150, 64, [
        (mixer(6, 2, 32, 32, 12, 90, temp=(0.4, 50)), moe(10, 3, 24, 1.5, identity=2, groups=(3, 2), shared=(40, 0.75))),
        (mixer(4, 4, 16, 48, 8, 33, temp=None), None),
        (mixer(3, 1, 64, 32, 32, 200, temp=(0.8, 64)), moe(5, 2, 16, 2.5, identity=1)),
    ], eps=1e-5, residual_mult=0.6, logit_scale=0.5, bigram=(211, 37, 11)),
    "B": model(89, 40, [
        (mixer(2, 1, 20, 12, 2, 3, temp=(0.25, 1)), moe(3, 1, 8, 0.5, identity=3, groups=(2, 1))),
        (mixer(5, 5, 48, 48, 20, 64, scale=0.05), moe(4, 4, 20, 7.0, shared=(12, 7.0))),
        (mixer(8, 1, 16, 16, 6, 400, temp=(1.5, 20)), moe(12, 4, 12, 1.0, identity=4, groups=(8, 5), shared=(8, 3.0))),
    ], eps=1e-3, residual_mult=1.25, logit_scale=2.0, bigram=(7, 100003, 65537)),
}


def tensor_shapes(cfg):
    """name -> shape of every tensor a model of this configuration has."""
    E, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    if cfg["embedding"].get("bigram"):
        out["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, E)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (E,), p + "mix.q": (H * d, E), p + "mix.k": (G * d, E), p + "mix.v": (G * dv, E), p + "mix.o": (E, H * dv),
                    p + "mix.q.norm": (d,), p + "mix.k.norm": (d,), p + "mix.rel": (m["bias_rows"], H)})
        if f:
            n, ff = f["router"]["experts"] + f["router"].get("identity", 0), f["expert"]["ff"]
            out.update({p + "norm2": (E,), p + "mlp.router": (n, E), p + "mlp.correction": (n,)})
            parts = [(f"e{e}", ff) for e in range(f["router"]["experts"])] + ([("shared", f["shared"]["ff"])] if f.get("shared") else [])
            for name, w in parts:
                out.update({f"{p}mlp.{name}.gate": (w, E), f"{p}mlp.{name}.up": (w, E), f"{p}mlp.{name}.down": (E, w)})
    return out


def make_weights(cfg, seed):
    """Random weights that bfloat16 holds exactly: matrices of spread 1 / sqrt(inputs) (gates and routers wider, so that they decide),
    norm weights around zero (around one for the heads'), biases of spread one, corrections that outweigh many scores and make most
    choice scores negative."""
    rng = np.random.default_rng(seed)
    t = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if name.endswith(("q.norm", "k.norm")):
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif "norm" in last:
            a = 0.2 * rng.standard_normal(shape)
        elif last == "rel":
            a = rng.standard_normal(shape)
        elif last == "correction":
            a = 0.2 * rng.standard_normal(shape) - 0.6
        elif name in ("embed", "bigram"):
            a = rng.standard_normal(shape) * (1.5 if name == "embed" else 0.8)
        else:
            a = rng.standard_normal(shape) / math.sqrt(shape[-1]) * {"router": 1.5, "gate": 1.5}.get(last, 1.0)
        t[name] = to_bf16(a)
    return t


def draw_config(rng):
    """A configuration whose sizes, constants and layers are drawn."""
    pick = lambda *a: a[int(rng.integers(len(a)))]                                                        # noqa: E731
    layers = []
    for _ in range(int(rng.integers(1, 4))):
        G = pick(1, 1, 2, 3)
        rows = pick(2, 4, 10, 16, 32)
        m = mixer(G * pick(1, 2, 4, 5), G, pick(8, 20, 32, 64, 128), pick(8, 16, 32, 64, 128), rows, rows // 2 + pick(1, 8, 50, 300), scale=pick(None, 0.02, 0.3),
                  temp=pick(None, (0.5, 1), (0.3, 30), (1.0, 100)))
        f = None
        if rng.random() < 0.8:
            groups, keep = pick((1, 1), (2, 1), (4, 2), (3, 3))
            size = pick(2, 3, 6)
            n = groups * size
            identity = int(rng.integers(0, n // 2 + 1))
            f = moe(n - identity, min(16, int(rng.integers(1, keep * size + 1))), pick(8, 12, 32, 50), pick(0.5, 1.5, 7.0), identity,
                    None if groups == 1 else (groups, keep), pick(None, (16, 1.0), (26, 4.0)))
        layers.append((m, f))
    return model(int(rng.integers(40, 160)), pick(24, 40, 64, 100, 128), layers, eps=pick(1e-6, 1e-4), residual_mult=pick(1.0, 0.3, 0.9),
                 logit_scale=pick(1.0, 0.5, 3.0), bigram=pick(None, (17, 3, 5), (997, 1009, 31), (128, 2147483647, 2147483646)))
