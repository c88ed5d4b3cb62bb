"""Plain numpy restatement of the Zegelix layer math, one function per mechanism, in float64 and without caches, pages or batches: a sequence
goes in whole and every position comes out.  Slow on purpose; it shares no code with the package.

``weights``: name -> array ([out, in] matrices), ``cfg``: the parsed configuration (a dict)."""
import math

import numpy as np


def sigmoid(v):
    return np.exp(-np.logaddexp(0.0, -v))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps) * w


# ------------------------------------------------------------------ rotation
def turn(x, positions, dims, base):
    """x [T, heads, d]: elements i and i + dims / 2 form a plane that turns by position * base^(-2 i / dims); elements past ``dims`` stay."""
    half = dims // 2
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * float(base) ** (-2.0 * np.arange(half) / dims)
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half], out[..., half:dims] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


# ------------------------------------------------------------------ attention
def window_sees(positions, n_keys, mask):
    """[queries, keys]: the query at position p sees key j when 0 <= p - j < size."""
    gap = np.asarray(positions)[:, None] - np.arange(n_keys)[None, :]
    return (gap >= 0) & (gap < mask["size"]) if mask else gap >= 0


def pooled(x, pool):
    """Means of the whole runs of ``pool`` consecutive rows: [rows // pool, ...]."""
    n = x.shape[0] // pool
    return x[:n * pool].reshape(n, pool, *x.shape[1:]).mean(axis=1)


def block_sees(positions, n_blocks, mask):
    """[queries, blocks]: the query at position p sees a block whose last token has left its window."""
    last = np.arange(n_blocks) * mask["pool"] + mask["pool"] - 1
    return last[None, :] <= np.asarray(positions)[:, None] - mask["size"]


def softmax_with_sink(scores, seen, sink):
    """Weights of the seen scores; exp(sink) joins the denominator (None: no sink)."""
    s = np.where(seen, scores, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + (np.exp(sink - m) if sink is not None else 0.0))


def capped(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def attend(q, k, v, scale, mask, cap=0.0, sinks=None, temp=None, positions=None):
    """q [queries, H, dim] at ``positions`` (default 0 ..), k and v [keys, G, ...] as cached -> [queries, H, vdim]."""
    H, G = q.shape[1], k.shape[1]
    positions = np.arange(q.shape[0]) if positions is None else np.asarray(positions)
    seen = window_sees(positions, k.shape[0], mask)
    if mask and mask.get("pool"):
        kb, vb = pooled(k, mask["pool"]), pooled(v, mask["pool"])
        seen = np.concatenate([seen, block_sees(positions, kb.shape[0], mask)], axis=1)
        k, v = np.concatenate([k, kb]), np.concatenate([v, vb])
    out = np.zeros((q.shape[0], H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale * (1.0 if temp is None else temp[h])
        out[:, h] = softmax_with_sink(capped(s, cap), seen, None if sinks is None else sinks[h]) @ v[:, g]
    return out


def attention(W, p, m, h):
    T, base = h.shape[0], m["rot"]["base"]
    proj = lambda n, heads, d: (h @ W[f"{p}.{n}"].T + W[f"{p}.{n}.b"]).reshape(T, heads, d)
    at = np.arange(T)
    q = turn(proj("q", m["heads"], m["dim"]), at, m["rot"]["dims"], base)
    k = turn(proj("k", m["kv_heads"], m["dim"]), at, m["rot"]["dims"], base)
    v = turn(proj("v", m["kv_heads"], m["vdim"]), at, m["vdim"], base)
    o = attend(q, k, v, m["scale"], m.get("mask"), m.get("softcap") or 0.0, W[f"{p}.sink"], W[f"{p}.temp"])
    o = turn(o, -at, m["vdim"], base).reshape(T, -1)
    return (o * sigmoid(h @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


# ------------------------------------------------------------------ recurrence
def causal_conv(x, w, b):
    """x [T, channels], w [channels, taps] (last column: the current token)."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(padded[j:j + x.shape[0]] * w[:, j] for j in range(taps)) + b


def block_linear(u, w, b):
    """u [T, channels] in as many equal parts as w has matrices [out, in]."""
    n, size = w.shape[0], w.shape[1]
    parts = u.reshape(u.shape[0], n, size)
    return (np.einsum("tni,noi->tno", parts, w) + b).reshape(u.shape)


def gated_recurrence(u, r, i, lam):
    """S <- a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), from S = 0."""
    log_a = -8.0 * r * np.logaddexp(0.0, lam)
    a, b = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a)) * i * u
    S, out = np.zeros(u.shape[1]), np.zeros(u.shape)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return out


def rglru(W, p, m, h):
    y = gelu_tanh(h @ W[f"{p}.y"].T + W[f"{p}.y.b"])
    u = causal_conv(h @ W[f"{p}.x"].T + W[f"{p}.x.b"], W[f"{p}.conv"], W[f"{p}.conv.b"])
    gate = lambda n: sigmoid(block_linear(u, W[f"{p}.{n}"], W[f"{p}.{n}.b"]))
    return (gated_recurrence(u, gate("ra"), gate("ri"), W[f"{p}.lam"]) * y) @ W[f"{p}.o"].T


# ------------------------------------------------------------------ feed-forward
def clamped_ffn(W, p, h, limit):
    g, u = np.minimum(h @ W[f"{p}.gate"].T, limit), np.clip(h @ W[f"{p}.up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[f"{p}.down"].T


def route(z, top):
    """Largest ``top`` of each row and their softmax."""
    best = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    s = np.take_along_axis(z, best, axis=-1)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return best, e / e.sum(axis=-1, keepdims=True)


def experts(W, p, mlp, h):
    best, weight = route(h @ W[f"{p}.router"].T + W[f"{p}.router.b"], mlp["router"]["top"])
    out = np.zeros(h.shape)
    for e in range(mlp["router"]["experts"]):
        rows, slot = np.nonzero(best == e)
        if rows.size:
            out[rows] += weight[rows, slot][:, None] * clamped_ffn(W, f"{p}.e{e}", h[rows], mlp["expert"]["limit"])
    if mlp.get("shared"):
        out += sigmoid(h @ W[f"{p}.shared.sg"].T) * clamped_ffn(W, f"{p}.shared", h, mlp["shared"]["limit"])
    return out


# ------------------------------------------------------------------ the model
MIXERS = {"attention": attention, "rglru": rglru}


def layer(W, p, e, x, eps):
    x = x + MIXERS[e["type"]](W, f"{p}.mix", e["mixer"], rms_norm(x, W[f"{p}.norm1"], eps))
    if e.get("mlp") is not None:
        x = x + experts(W, f"{p}.mlp", e["mlp"], rms_norm(x, W[f"{p}.norm2"], eps))
    return x


def runs(cfg):
    """(layer, does a pass of the loop begin with it) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(l, False) for l in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(l, False) for l in range(a)] + [(l, l == a) for _ in range(loop["times"]) for l in range(a, b)] + [(l, False) for l in range(b, n)]


def forward(cfg, weights, tokens, layers_out=None):
    W = {n: np.asarray(a, dtype=np.float64) for n, a in weights.items()}
    eps = cfg["norm"]["eps"]
    first = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    x = first
    for l, begins in runs(cfg):
        if begins:
            x = np.concatenate([x, first], axis=1) @ W["loop.in"].T
        x = layer(W, f"l{l}", cfg["layers"][l], x, eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, weights, toks)[-1])))
    return toks[len(prompt):]
