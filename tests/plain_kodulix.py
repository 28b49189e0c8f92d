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
    correction = t.get(pre + "correction")
    correction = np.zeros(len(t[pre + "router"])) if correction is None else correction
    choices, weights = route(x, t[pre + "router"], correction, int(r["top"]), int(groups["count"]), int(groups["keep"]))
    out = np.zeros_like(x)
    for i in range(x.shape[0]):
        for e, w in zip(choices[i], weights[i]):
            y = x[i] if e >= n else clipped_glu(x[i:i + 1], t, f"{pre}e{e}.", mlp["expert"]["limit"])[0]
            out[i] += w * y
    if mlp.get("shared"):
        out = out + clipped_glu(x, t, pre + "shared.", mlp["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------------- whole

def forward(cfg, weights, tokens):
    """(scores [T, vocab], streams after every layer [layers, T, E])."""
    t = {n: np.asarray(w, dtype=np.float64) for n, w in weights.items()}
    eps, m = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = embedded(cfg, t, tokens)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + m * offset_norm(attention(x, layer["mixer"], t, p + "mix.", eps), t[p + "norm1"], eps)
        if layer.get("mlp"):
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
