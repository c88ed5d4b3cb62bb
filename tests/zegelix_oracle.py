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


# ------------------------------------------------------------------ small configurations with random weights
def feed_forward(mlp):
    """None, or (experts, top, expert width, limit, width of the shared expert or 0, its limit)."""
    if mlp is None:
        return None
    experts, top, ff, limit, shared, shared_limit = mlp
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    return {**f, "shared": {"ff": shared, "limit": shared_limit}} if shared else f


def attention_layer(mlp, heads, kv_heads, dim, vdim, window, pool, rot_dims, base=10000.0, cap=30.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims}, "scale": scale or 1.0 / math.sqrt(dim)}
    if cap:
        m["softcap"] = cap
    if window:
        m["mask"] = {"size": window, "pool": pool} if pool else {"size": window}
    return {"type": "attention", "mlp": feed_forward(mlp), "mixer": m}


def rglru_layer(mlp, width, blocks, taps):
    return {"type": "rglru", "mlp": feed_forward(mlp), "mixer": {"width": width, "blocks": blocks, "conv": taps}}


def random_config(layers, vocab=96, width=64, eps=1e-6, scale=3.0, logit_scale=1.0, loop=None):
    c = {"architecture": "Zegelix", "embedding": {"scale": scale}, "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def round_bf16(a):
    """float array -> float32 values that bfloat16 represents (round to nearest even)."""
    u = np.array(a, dtype=np.float32, order="C").view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16 << 16).astype(np.uint32)
    return u.view(np.float32)


CODES = 8            # columns that hold a code of the token and that no layer writes to, read by the routers alone


def random_weights(cfg, seed=0):
    """Every tensor the configuration asks for, as float32 arrays that hold bfloat16 values.  The routers read a code of the token, so that no choice of
    experts is within rounding of another."""
    g = np.random.default_rng(seed)
    H, W = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        W[name] = round_bf16(g.standard_normal((n, k)) * gain / math.sqrt(k))

    def vec(name, n, mean=0.0, std=0.2):
        W[name] = round_bf16(mean + std * g.standard_normal(n))

    def gated(name, f):
        for n, shape in (("gate", (f, H)), ("up", (f, H)), ("down", (H, f))):
            mat(f"{name}.{n}", *shape)

    W["embed"] = round_bf16(g.standard_normal((cfg["vocab"], H)) / cfg["embedding"]["scale"])
    vec("final.norm", H, 1.0)
    if cfg.get("loop"):
        mat("loop.in", H, 2 * H)
    for i, layer in enumerate(cfg["layers"]):
        l, p, m, f = f"l{i}", f"l{i}.mix", layer["mixer"], layer["mlp"]
        vec(f"{l}.norm1", H, 1.0)
        if layer["type"] == "attention":
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                mat(f"{p}.{n}", rows, H)
                vec(f"{p}.{n}.b", rows, 0.0, 0.5)
            vec(f"{p}.temp", m["heads"], 1.2, 0.4)
            vec(f"{p}.sink", m["heads"], 0.5, 1.0)
            mat(f"{p}.g", m["heads"] * m["vdim"], H)
            mat(f"{p}.o", H, m["heads"] * m["vdim"], 1.2)
        else:
            w, b = m["width"], m["blocks"]
            for n in "yx":
                mat(f"{p}.{n}", w, H, 1.3)
                vec(f"{p}.{n}.b", w, 0.0, 0.4)
            W[f"{p}.conv"] = round_bf16(g.standard_normal((w, m["conv"])) / math.sqrt(m["conv"]))
            vec(f"{p}.conv.b", w)
            for n in ("ra", "ri"):
                W[f"{p}.{n}"] = round_bf16(g.standard_normal((b, w // b, w // b)) / math.sqrt(w // b))
                W[f"{p}.{n}.b"] = round_bf16(0.5 * g.standard_normal((b, w // b)))
            W[f"{p}.lam"] = round_bf16(g.uniform(-7.0, 1.0, w))          # from memories of hundreds of tokens to almost none
            mat(f"{p}.o", H, w, 1.5)
        if f is None:
            continue
        vec(f"{l}.norm2", H, 1.0)
        mat(f"{l}.mlp.router", f["router"]["experts"], H)
        vec(f"{l}.mlp.router.b", f["router"]["experts"], 0.0, 0.1)
        for e in range(f["router"]["experts"]):
            gated(f"{l}.mlp.e{e}", f["expert"]["ff"])
        if f.get("shared"):
            gated(f"{l}.mlp.shared", f["shared"]["ff"])
            mat(f"{l}.mlp.shared.sg", 1, H)
    _settle_routing(cfg, W, g)
    return W


def _settle_routing(cfg, W, g, gap=0.1):
    moe = [(i, layer["mlp"]["router"]) for i, layer in enumerate(cfg["layers"]) if layer["mlp"] is not None]
    if not moe:
        return
    for n in W:                                          # no branch writes to the code's columns, a pass of the loop hands them on
        if n.endswith(".mix.o") or n.endswith(".down"):
            W[n][:CODES] = 0.0
    if cfg.get("loop"):
        W["loop.in"][:CODES] = 0.0
        W["loop.in"][:CODES, :CODES] = np.eye(CODES)
    scale = cfg["embedding"]["scale"]
    for i, r in moe:
        z = g.standard_normal((r["experts"], CODES)) * 0.5
        W[f"l{i}.mlp.router"] = round_bf16(np.pad(z, ((0, 0), (0, cfg["width"] - CODES))))
        W[f"l{i}.norm2"][:CODES] = 1.0
    for t in range(cfg["vocab"]):
        for _ in range(3000):
            code = round_bf16(2.0 * g.choice([-1.0, 1.0], CODES) / scale)
            gaps = [np.inf]
            for i, r in moe:
                for rms in (0.7, 1.0, 1.5, 2.5, 4.0):            # what the norm in front of the router may divide by
                    z = np.float64(W[f"l{i}.mlp.router"])[:, :CODES] @ (np.float64(code) * scale) / rms + W[f"l{i}.mlp.router.b"]
                    z = np.sort(z)[::-1]
                    if r["top"] < len(z):
                        gaps.append(z[r["top"] - 1] - z[r["top"]])
            if min(gaps) > gap:
                break
        else:
            raise ValueError("no code of this token settles its routing")
        W["embed"][t, :CODES] = code
