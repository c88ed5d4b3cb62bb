"""Plain numpy restatement of the Beputar layer math, one function per mechanism, in float64 and without caches, pages or batches: a sequence
goes in whole and every position comes out.  Slow on purpose; it shares no code with the package.

``weights``: name -> array ([out, in] matrices), ``cfg``: the parsed configuration (a dict)."""
import math

import numpy as np


def sigmoid(v):
    return np.exp(-np.logaddexp(0.0, -v))


def silu(v):
    return v * sigmoid(v)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps) * w


# ------------------------------------------------------------------ rotation
def frequencies(rot):
    """(angle per position of every pair, factor on cos and sin); ``scaling`` is YaRN."""
    dims, base, y = rot["dims"], float(rot["base"]), rot.get("scaling")
    i = np.arange(dims // 2)
    f = base ** (-2.0 * i / dims)
    if y is None:
        return f, 1.0
    pair_of = lambda turns: dims * math.log(y["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair_of(y["fast"])), 0), min(math.ceil(pair_of(y["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / y["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(y["factor"]) + 1.0


def rotate(x, positions, rot, interleaved):
    """x [T, heads, dim]; pair i holds elements (2i, 2i + 1) or (i, i + dims / 2); elements past ``dims`` stay."""
    f, mag = frequencies(rot)
    d = rot["dims"]
    a = (np.asarray(positions, dtype=np.float64)[:, None] * f)[:, None, :]
    c, s = np.cos(a) * mag, np.sin(a) * mag
    first, second = (np.arange(0, d, 2), np.arange(1, d, 2)) if interleaved else (np.arange(d // 2), np.arange(d // 2, d))
    out = x.copy()
    u, v = x[..., first], x[..., second]
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------ attention
def visible(nq, nk, mask, first_query=0):
    """[queries, keys]: the query in row r stands at position first_query + r and sees the last ``size`` keys and the first ``keep_first``."""
    gap = (first_query + np.arange(nq))[:, None] - np.arange(nk)[None, :]
    if not mask:
        return gap >= 0
    return (gap >= 0) & ((gap < mask["size"]) | (np.arange(nk)[None, :] < mask.get("keep_first", 0)))


def softmax(scores, seen, sink=False):
    """``sink``: one more score of 0 in the denominator, without a value."""
    s = np.where(seen, scores, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0) if sink else s.max(axis=-1, keepdims=True)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + (np.exp(-m) if sink else 0.0))


def attend(q, k, v, scale, mask, sink=False, first_query=0):
    """q [queries, H, dim], k and v [keys, G, ...] -> [queries, H, vdim]."""
    H, G = q.shape[1], k.shape[1]
    seen = visible(q.shape[0], k.shape[0], mask, first_query)
    out = np.zeros((q.shape[0], H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax(q[:, h] @ k[:, g].T * scale, seen, sink) @ v[:, g]
    return out


def biased_attention(W, p, m, h, eps):
    T, d = h.shape[0], m["dim"]
    q = (h @ W[f"{p}.q"].T + W[f"{p}.q.b"]).reshape(T, m["heads"], d)
    v = (h @ W[f"{p}.k"].T + W[f"{p}.k.b"]).reshape(T, m["kv_heads"], d)
    turn = lambda x: rms_norm(rotate(x, np.arange(T), m["rot"], True), 1.0, eps)
    return attend(turn(q), turn(v), v, m["scale"], m.get("mask")).reshape(T, -1) @ W[f"{p}.o"].T


def gated_attention(W, p, m, h, eps):
    T, d = h.shape[0], m["dim"]
    q = (h @ W[f"{p}.q"].T).reshape(T, m["heads"], d)
    v = (h @ W[f"{p}.k"].T).reshape(T, m["kv_heads"], d)
    turn = lambda x, w: rotate(rms_norm(x, w, eps), np.arange(T), m["rot"], False)
    a = attend(turn(q, W[f"{p}.q.norm"]), turn(v, W[f"{p}.k.norm"]), v, m["scale"], m.get("mask"), sink=True)
    return (a * sigmoid(h @ W[f"{p}.g"].T)[:, :, None]).reshape(T, -1) @ W[f"{p}.o"].T


# ------------------------------------------------------------------ recurrences
def decayed_sum(q, k, v, decay):
    """q, k [T, H, dim], v [T, H, vdim], decay [H]: S <- decay S + k v^T, o = S^T q."""
    T, H, d = q.shape
    S, out = np.zeros((H, d, v.shape[2])), np.zeros(v.shape)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hd,hdv->hv", q[t], S)
    return out


def lightning_attention(W, p, m, h, eps):
    T, H = h.shape[0], m["heads"]
    proj = lambda n, d: silu(h @ W[f"{p}.{n}"].T).reshape(T, H, d)
    o = decayed_sum(proj("q", m["dim"]), proj("k", m["dim"]), proj("v", m["vdim"]), np.asarray(m["decay"], dtype=np.float64)).reshape(T, -1)
    return (rms_norm(o, W[f"{p}.norm"], eps) * sigmoid(h @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


def token_shift(h, mu):
    before = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]])
    return h + (before - h) * mu


def wkv_recurrence(r, k, v, w, u):
    """r, k, w [T, H, dim], v [T, H, vdim], u [H, dim]: o = (S + (u k) v^T)^T r, then S <- w S + k v^T."""
    T, H, d = r.shape
    S, out = np.zeros((H, d, v.shape[2])), np.zeros(v.shape)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hd,hdv->hv", r[t], S + u[:, :, None] * kv)
        S = w[t][:, :, None] * S + kv
    return out


def wkv(W, p, m, h, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    mix = {n: token_shift(h, W[f"{p}.mu.{n}"]) for n in "rkvgw"}
    r, k, v = ((mix[n] @ W[f"{p}.{n}"].T).reshape(T, H, d) for n in "rkv")
    z = np.tanh(mix["w"] @ W[f"{p}.w1"].T) @ W[f"{p}.w2"].T + W[f"{p}.w0"]
    o = wkv_recurrence(r, k, v, np.exp(-np.exp(z)).reshape(T, H, d), W[f"{p}.u"])
    o = rms_norm(o, 1.0, eps).reshape(T, -1) * W[f"{p}.norm"] * silu(mix["g"] @ W[f"{p}.g"].T)
    return o @ W[f"{p}.o"].T


def parallel(W, p, m, h, eps):
    sides = (gated_attention(W, f"{p}.left", m["left"], h, eps), lightning_attention(W, f"{p}.right", m["right"], h, eps))
    return 0.5 * sum(rms_norm(y, W[f"{p}.{n}.out"], eps) for y, n in zip(sides, ("left", "right")))


MIXERS = {"wkv": wkv, "parallel": parallel, "attention": biased_attention}


# ------------------------------------------------------------------ feed-forward
def dense_mlp(W, p, f, h):
    return gelu_tanh(h @ W[f"{p}.up"].T) @ W[f"{p}.down"].T


def route(z, top):
    """Router logits [T, experts] -> chosen experts [T, top] (best first) and their sigmoid scores."""
    idx = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return idx, sigmoid(np.take_along_axis(z, idx, axis=-1))


def expert(W, p, h):
    return (silu(h @ W[f"{p}.gate"].T) * (h @ W[f"{p}.up"].T)) @ W[f"{p}.down"].T


def moe_mlp(W, p, f, h):
    """The score of a chosen expert scales what it reads."""
    idx, w = route(h @ W[f"{p}.router"].T, f["router"]["top"])
    out = expert(W, f"{p}.shared", h) if f.get("shared") else np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t], w[t]):
            out[t] += expert(W, f"{p}.e{e}", we * h[t])
    return out


FEED_FORWARD = {"dense": dense_mlp, "moe": moe_mlp}


# ------------------------------------------------------------------ model
def forward(weights, cfg, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        l, f = f"l{i}", layer["mlp"]
        x = x + rms_norm(MIXERS[layer["type"]](W, f"{l}.mix", layer["mixer"], x, eps), W[f"{l}.norm1"], eps) * W[f"{l}.ls1"]
        if f is not None:
            x = x + rms_norm(FEED_FORWARD[f["kind"]](W, f"{l}.mlp", f, x), W[f"{l}.norm2"], eps) * W[f"{l}.ls2"]
        after.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T, np.stack(after)


# ------------------------------------------------------------------ configurations and weights of tests
def _rot(dims, base, scaling):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def feed_forward(mlp):
    """None, a width (dense), or (experts, top, expert width, width of the shared expert or 0)."""
    if not isinstance(mlp, tuple):
        return None if mlp is None else {"kind": "dense", "ff": mlp}
    f = {"kind": "moe", "expert": {"ff": mlp[2]}, "router": {"experts": mlp[0], "top": mlp[1]}}
    return {**f, "shared": {"ff": mlp[3]}} if mlp[3] else f


def attention_sizes(heads, kv_heads, dim, window, rot_dims, base=10000.0, scaling=None, keep_first=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": _rot(rot_dims, base, scaling), "scale": scale or 1.0 / math.sqrt(dim)}
    if window:
        m["mask"] = {"size": window} if keep_first is None else {"size": window, "keep_first": keep_first}
    return m


def attention_layer(mlp, *sizes, **kw):
    return {"type": "attention", "mlp": feed_forward(mlp), "mixer": attention_sizes(*sizes, **kw)}


def wkv_layer(mlp, heads, dim):
    return {"type": "wkv", "mlp": feed_forward(mlp), "mixer": {"heads": heads, "dim": dim}}


def parallel_layer(mlp, left, heads, dim, vdim, decay):
    return {"type": "parallel", "mlp": feed_forward(mlp), "mixer": {"left": left, "right": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}}


def random_config(layers, vocab=96, width=64, eps=1e-6, scale=3.0):
    return {"architecture": "Beputar", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def round_bf16(a):
    """float array -> float32 values that bfloat16 represents (round to nearest even)."""
    u = np.array(a, dtype=np.float32, order="C").view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16 << 16).astype(np.uint32)
    return u.view(np.float32)


CODES = 8            # columns that hold a code of the token and that no layer writes to, read by the routers alone


def random_weights(cfg, seed=0, rank=12):
    """Every tensor the configuration asks for, as float32 arrays that hold bfloat16 values.  The routers read a code of the token, so that no choice of
    experts is within rounding of another.  ``rank``: inner width of the decay's projection."""
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
    for i, layer in enumerate(cfg["layers"]):
        l, p, m, f = f"l{i}", f"l{i}.mix", layer["mixer"], layer["mlp"]
        vec(f"{l}.norm1", H, 1.0)
        vec(f"{l}.ls1", H, 0.5, 0.1)
        if layer["type"] == "attention":
            for n, k in (("q", m["heads"]), ("k", m["kv_heads"])):
                mat(f"{p}.{n}", k * m["dim"], H, 1.5)
                vec(f"{p}.{n}.b", k * m["dim"], 0.0, 0.5)
            mat(f"{p}.o", H, m["heads"] * m["dim"])
        elif layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for k in "rkvg":
                mat(f"{p}.{k}", n, H)
            for k in "rkvgw":
                W[f"{p}.mu.{k}"] = round_bf16(g.uniform(0.0, 1.0, H))
            mat(f"{p}.w1", rank, H)
            mat(f"{p}.w2", n, rank)
            W[f"{p}.w0"] = round_bf16(g.uniform(-5.0, 0.5, n))
            W[f"{p}.u"] = round_bf16(0.5 * g.standard_normal((m["heads"], m["dim"])))
            vec(f"{p}.norm", n, 1.0)
            mat(f"{p}.o", H, n)
        else:
            a, b = m["left"], m["right"]
            for n, k in (("q", a["heads"]), ("k", a["kv_heads"])):
                mat(f"{p}.left.{n}", k * a["dim"], H, 1.5)
                vec(f"{p}.left.{n}.norm", a["dim"], 1.3)
            mat(f"{p}.left.g", a["heads"], H)
            mat(f"{p}.left.o", H, a["heads"] * a["dim"])
            nk, nv = b["heads"] * b["dim"], b["heads"] * b["vdim"]
            for n, k in (("q", nk), ("k", nk), ("v", nv), ("g", nv)):
                mat(f"{p}.right.{n}", k, H)
            vec(f"{p}.right.norm", nv, 1.0)
            mat(f"{p}.right.o", H, nv)
            vec(f"{p}.left.out", H, 1.0)
            vec(f"{p}.right.out", H, 1.0)
        if f is None:
            continue
        vec(f"{l}.norm2", H, 1.0)
        vec(f"{l}.ls2", H, 0.5, 0.1)
        if f["kind"] == "dense":
            mat(f"{l}.mlp.up", f["ff"], H)
            mat(f"{l}.mlp.down", H, f["ff"])
        else:
            for e in range(f["router"]["experts"]):
                gated(f"{l}.mlp.e{e}", f["expert"]["ff"])
            if f.get("shared"):
                gated(f"{l}.mlp.shared", f["shared"]["ff"])
    _settle_routing(cfg, W, g)
    return W


def _settle_routing(cfg, W, g, gap=0.3):
    moe = [(i, layer["mlp"]["router"]) for i, layer in enumerate(cfg["layers"]) if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe"]
    if not moe:
        return
    for i, _ in enumerate(cfg["layers"]):
        for n in (f"l{i}.ls1", f"l{i}.ls2"):
            if n in W:
                W[n][:CODES] = 0.0
    scale = cfg["embedding"]["scale"]
    for i, r in moe:
        z = g.standard_normal((r["experts"], CODES)) * 0.5
        W[f"l{i}.mlp.router"] = round_bf16(np.pad(z, ((0, 0), (0, cfg["width"] - CODES))))
    for t in range(cfg["vocab"]):
        for _ in range(2000):
            code = round_bf16(2.0 * g.choice([-1.0, 1.0], CODES) / scale)
            gaps = [np.inf]
            for i, r in moe:
                z = np.sort(np.float64(W[f"l{i}.mlp.router"])[:, :CODES] @ (np.float64(code) * scale))[::-1]
                if r["top"] < len(z):
                    gaps.append(z[r["top"] - 1] - z[r["top"]])
            if min(gaps) > gap:
                break
        else:
            raise ValueError("no code of this token settles its routing")
        W["embed"][t, :CODES] = code
