"""Plain numpy restatement of the Pubodra layer math, one function per mechanism, in float64 and without caches, pages or batches: a
sequence goes in whole and every position comes out.  Slow on purpose; it shares no code with the package.

``weights``: name -> array ([out, in] matrices), ``cfg``: the parsed configuration (a dict)."""
import math

import numpy as np


def sigmoid(v):
    return np.exp(-np.logaddexp(0.0, -v))


def dynamic_tanh(x, alpha, w, b):
    """Element-wise squashing in the place of a norm: no mean, no variance."""
    return np.tanh(alpha * x) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


# ------------------------------------------------------------------ rotation
def frequencies(dims, base, scaling=None):
    """(angle per position of every pair, factor on cos and sin).  ``scaling``: YaRN -- pairs that turn often within the original context keep
    their frequency, slow ones are divided by the factor, a ramp lies between."""
    i = np.arange(dims // 2)
    f = float(base) ** (-2.0 * i / dims)
    if scaling is None:
        return f, 1.0
    pair_of = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, positions, rot):
    """x [T, ..., >= dims]: elements 2i and 2i + 1 form pair i, turned by position * frequency i; elements past ``dims`` stay."""
    f, mag = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    a = np.asarray(positions, dtype=np.float64)[:, None] * f
    a = a.reshape(a.shape[0], *([1] * (x.ndim - 2)), a.shape[1])
    c, s = np.cos(a) * mag, np.sin(a) * mag
    out = x.copy()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * c - v * s
    out[..., 1:rot["dims"]:2] = v * c + u * s
    return out


# ------------------------------------------------------------------ attention
def windowed_softmax(scores, window, first_query=0):
    """scores [..., queries, keys]; the query in row r stands at position first_query + r and sees itself and the window - 1 keys before it."""
    nq, nk = scores.shape[-2:]
    gap = (first_query + np.arange(nq))[:, None] - np.arange(nk)[None, :]
    seen = (gap >= 0) & ((gap < window) if window else True)
    s = np.where(seen, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_heads(q, c, k_rot, uk, uv, scale, window, first_query=0):
    """q [queries, H, dim + rot_dim] (rotated), latents c [keys, rank] (normed), shared rotated key part [keys, rot_dim], uk [H, dim, rank],
    uv [H, vdim, rank] -> [queries, H, vdim]."""
    H, dim, _ = uk.shape
    out = np.zeros((q.shape[0], H, uv.shape[1]))
    for h in range(H):
        keys, values = c @ uk[h].T, c @ uv[h].T
        s = (q[:, h, :dim] @ keys.T + q[:, h, dim:] @ k_rot.T) * scale
        out[:, h] = windowed_softmax(s, window, first_query) @ values
    return out


def latent_attention_mixer(W, name, m, h, eps):
    T, H, dim, rd, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    pos = np.arange(T)
    q = (h @ W[f"{name}.q"].T).reshape(T, H, dim + rd)
    q = np.concatenate([q[..., :dim], rotate_pairs(q[..., dim:], pos, m["rot"])], axis=-1)
    down = h @ W[f"{name}.dkv"].T
    c = rms_norm(down[:, :rank], W[f"{name}.dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, rank:], pos, m["rot"])
    window = m["mask"]["size"] if m.get("mask") else 0
    a = latent_heads(q, c, k_rot, W[f"{name}.uk"].reshape(H, dim, rank), W[f"{name}.uv"].reshape(H, m["vdim"], rank), m["scale"], window)
    return (a.reshape(T, -1) * sigmoid(h @ W[f"{name}.g"].T)) @ W[f"{name}.o"].T


# ------------------------------------------------------------------ feed-forward
def dense_mlp(W, name, f, h):
    return gelu_tanh(h @ W[f"{name}.up"].T) @ W[f"{name}.down"].T


def route(z, top):
    """Router logits [T, experts] -> chosen experts [T, top] (best first) and their softmax scores scaled to sum to one."""
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    s /= s.sum(axis=-1, keepdims=True)
    idx = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    w = np.take_along_axis(s, idx, axis=-1)
    return idx, w / (w.sum(axis=-1, keepdims=True) + 1e-20)


def expert(W, name, h):
    return squared_relu(h @ W[f"{name}.up"].T) @ W[f"{name}.down"].T


def moe_mlp(W, name, f, h):
    idx, w = route(h @ W[f"{name}.router"].T, f["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t], w[t]):
            out[t] += we * expert(W, f"{name}.e{e}", h[t])
    return out


FEED_FORWARD = {"dense": dense_mlp, "moe": moe_mlp}


# ------------------------------------------------------------------ model
def layer_runs(cfg):
    """(layer, vector added to the residual before it or None) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    looped = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + looped + [(i, None) for i in range(b, n)]


def forward(weights, cfg, tokens):
    """(logits [T, vocab], residual stream after every layer run [runs, T, width])."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in weights.items()}
    norm = lambda x, name: dynamic_tanh(x, W[f"{name}.alpha"], W[name], W[f"{name}.b"])
    x = W["embed"][np.asarray(tokens)]
    after = []
    for i, t in layer_runs(cfg):
        if t is not None:
            x = x + W["loop.step"][t]
        layer, l = cfg["layers"][i], f"l{i}"
        x = x + latent_attention_mixer(W, f"{l}.mix", layer["mixer"], norm(x, f"{l}.norm1"), cfg["norm"]["eps"])
        f = layer["mlp"]
        if f is not None:
            x = x + FEED_FORWARD[f["kind"]](W, f"{l}.mlp", f, norm(x, f"{l}.norm2"))
        after.append(x)
    return norm(x, "final.norm") @ W["embed"].T, np.stack(after)


# ------------------------------------------------------------------ configurations and weights of tests
def latent_layer(heads, dim, rot_dim, vdim, kv_rank, window, mlp, base=10000.0, scaling=None, scale=None):
    """``mlp``: None, a width (dense), or (experts, top, expert width)."""
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if isinstance(mlp, tuple):
        f = {"kind": "moe", "expert": {"ff": mlp[2]}, "router": {"experts": mlp[0], "top": mlp[1]}}
    else:
        f = None if mlp is None else {"kind": "dense", "ff": mlp}
    return {"type": "latent_attention", "mlp": f,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window}, "rot": rot,
                      "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)}}


def random_config(layers, vocab=96, width=64, eps=1e-6, loop=None):
    c = {"architecture": "Pubodra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def round_bf16(a):
    """float array -> float32 values that bfloat16 represents (round to nearest even)."""
    u = np.array(a, dtype=np.float32, order="C").view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16 << 16).astype(np.uint32)
    return u.view(np.float32)


def random_weights(cfg, seed=0, clear_routing=False):
    """Every tensor the configuration asks for, as float32 arrays that hold bfloat16 values.  ``clear_routing``: the routers read a few columns
    that hold a code of the token and that no layer writes to, so that no choice of experts is within rounding of another."""
    g = np.random.default_rng(seed)
    H, W = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        W[name] = round_bf16(g.standard_normal((n, k)) * gain / math.sqrt(k))

    def norm(name):
        W[name], W[f"{name}.b"] = round_bf16(1.0 + 0.2 * g.standard_normal(H)), round_bf16(0.1 * g.standard_normal(H))
        W[f"{name}.alpha"] = round_bf16(np.float32(g.uniform(0.4, 0.9)))

    W["embed"] = round_bf16(g.standard_normal((cfg["vocab"], H)))
    if cfg.get("loop"):
        W["loop.step"] = round_bf16(0.5 * g.standard_normal((cfg["loop"]["times"], H)))
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        l, m, f = f"l{i}", layer["mixer"], layer["mlp"]
        norm(f"{l}.norm1")
        mat(f"{l}.mix.q", m["heads"] * (m["dim"] + m["rot_dim"]), H, 1.5)
        mat(f"{l}.mix.dkv", m["kv_rank"] + m["rot_dim"], H, 1.5)
        W[f"{l}.mix.dkv.norm"] = round_bf16(1.0 + 0.2 * g.standard_normal(m["kv_rank"]))
        mat(f"{l}.mix.uk", m["heads"] * m["dim"], m["kv_rank"])
        mat(f"{l}.mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(f"{l}.mix.g", m["heads"] * m["vdim"], H)
        mat(f"{l}.mix.o", H, m["heads"] * m["vdim"])
        if f is None:
            continue
        norm(f"{l}.norm2")
        if f["kind"] == "dense":
            mat(f"{l}.mlp.up", f["ff"], H)
            mat(f"{l}.mlp.down", H, f["ff"])
        else:
            mat(f"{l}.mlp.router", f["router"]["experts"], H, 1.5)
            for e in range(f["router"]["experts"]):
                mat(f"{l}.mlp.e{e}.up", f["expert"]["ff"], H)
                mat(f"{l}.mlp.e{e}.down", H, f["expert"]["ff"])
    if clear_routing:
        _settle_routing(cfg, W, g)
    return W


def _settle_routing(cfg, W, g, codes=8, gap=0.3):
    for n in list(W):
        if n.endswith(".mix.o") or n.endswith(".down"):
            W[n][:codes] = 0.0
        elif n == "loop.step":
            W[n][:, :codes] = 0.0
    layers = [i for i, layer in enumerate(cfg["layers"]) if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe"]
    for i in layers:
        W[f"l{i}.mlp.router"] = round_bf16(np.pad(g.standard_normal((cfg["layers"][i]["mlp"]["router"]["experts"], codes)), ((0, 0), (0, cfg["width"] - codes))))
    for t in range(cfg["vocab"]):
        for _ in range(2000):
            x = np.zeros(cfg["width"])
            x[:codes] = 2.0 * g.choice([-1.0, 1.0], codes)
            gaps = [np.inf]
            for i in layers:
                l, top = f"l{i}", cfg["layers"][i]["mlp"]["router"]["top"]
                h = dynamic_tanh(x, *(np.float64(W[f"{l}.norm2{s}"]) for s in (".alpha", "", ".b")))
                z = np.sort(np.float64(W[f"{l}.mlp.router"])[:, :codes] @ h[:codes])[::-1]
                if top < len(z):
                    gaps.append(z[top - 1] - z[top])
            if min(gaps) > gap:
                break
        else:
            raise ValueError("no code of this token settles its routing")
        W["embed"][t, :codes] = x[:codes]
