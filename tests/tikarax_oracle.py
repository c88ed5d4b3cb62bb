"""Plain numpy restatement of the Tikarax layer math, one function per mechanism, in float64 and without caches, pages or batches: a
sequence goes in whole and every position comes out.  Slow on purpose; it shares no code with the package.

``weights``: name -> array ([out, in] matrices), ``cfg``: the parsed configuration (a dict)."""
import math

import numpy as np


def softplus(v):
    return np.logaddexp(0.0, v)


def sigmoid(v):
    return np.exp(-np.logaddexp(0.0, -v))


def silu(v):
    return v * sigmoid(v)


def grouped_norm(x, w, eps, groups):
    """Every one of ``groups`` equal parts of the last axis over its own root mean square, the whole times w."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    rms = np.sqrt((parts ** 2).mean(axis=-1, keepdims=True) + eps)
    return (parts / rms).reshape(x.shape) * w


def xielu(z, p, q):
    """Squared above zero, exponential below; both branches carry z / 2."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions) + 1) / every) + 1.0)


def causal_softmax_attention(q, k, v, scale):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; query head h reads key / value head h // (H / G)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].T * scale
        s[np.triu_indices(T, 1)] = -np.inf
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, h // rep]
    return out


def attention_mixer(W, name, m, h):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    lin = lambda t: h @ W[f"{name}.{t}"].T + W[f"{name}.{t}.b"]
    q, k, v = lin("q").reshape(T, H, m["dim"]), lin("k").reshape(T, G, m["dim"]), lin("v").reshape(T, G, m["vdim"])
    q = q * query_temperature(np.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    a = causal_softmax_attention(q, k, v, m["scale"]).reshape(T, H * m["vdim"])
    return (a * sigmoid(h @ W[f"{name}.g"].T)) @ W[f"{name}.o"].T


def mingru_recurrence(zpre, u, state):
    """S_t = (1 - z) S_(t-1) + z * candidate, token by token; returns every S and the last one."""
    z = sigmoid(zpre)
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    out = np.zeros_like(u)
    for t in range(u.shape[0]):
        state = (1.0 - z[t]) * state + z[t] * cand[t]
        out[t] = state
    return out, state


def mingru_mixer(W, name, m, h):
    S, _ = mingru_recurrence(h @ W[f"{name}.z"].T + W[f"{name}.z.b"], h @ W[f"{name}.x"].T + W[f"{name}.x.b"], np.zeros(m["width"]))
    return (S * silu(h @ W[f"{name}.g"].T)) @ W[f"{name}.o"].T


def dense_mlp(W, name, h):
    p, q = W[f"{name}.act"]
    return xielu(h @ W[f"{name}.up"].T, p, q) @ W[f"{name}.down"].T


MIXERS = {"attention": attention_mixer, "mingru": mingru_mixer}


def forward(weights, cfg, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in weights.items()}
    norm = lambda x, name: grouped_norm(x, W[name], cfg["norm"]["eps"], cfg["norm"]["groups"])
    x = norm(W["embed"][np.asarray(tokens)], "embed.norm")
    after = []
    for i, layer in enumerate(cfg["layers"]):
        l = f"l{i}"
        x = x + norm(MIXERS[layer["type"]](W, f"{l}.mix", layer["mixer"], norm(x, f"{l}.norm1")), f"{l}.norm1b")
        if layer["mlp"] is not None:
            x = x + norm(dense_mlp(W, f"{l}.mlp", norm(x, f"{l}.norm2")), f"{l}.norm2b")
        after.append(x)
    return norm(x, "final.norm") @ W["head"].T, np.stack(after)


def random_config(layers, vocab=96, width=64, groups=2, eps=1e-6):
    return {"architecture": "Tikarax", "layers": layers, "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}


def attention_layer(heads, kv_heads, dim, vdim, ff, coef=0.5, every=16, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "q_temp": {"coef": coef, "every": every},
                                           "scale": scale if scale is not None else 1.0 / math.sqrt(dim)},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mingru_layer(width, ff):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def round_bf16(a):
    """float array -> float32 values that bfloat16 represents (round to nearest even)."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16 << 16).astype(np.uint32)
    return u.view(np.float32)


def random_weights(cfg, seed=0):
    """Every tensor the configuration asks for, as float32 arrays that hold bfloat16 values."""
    g = np.random.default_rng(seed)
    H = cfg["width"]
    W = {}

    def mat(name, n, k, gain=1.0):
        W[name] = round_bf16(g.standard_normal((n, k)) * gain / math.sqrt(k))

    def vec(name, n, mean, std):
        W[name] = round_bf16(mean + std * g.standard_normal(n))

    W["embed"] = round_bf16(g.standard_normal((cfg["vocab"], H)))
    for n in ("embed.norm", "final.norm"):
        vec(n, H, 1.0, 0.2)
    mat("head", cfg["vocab"], H, 2.0)
    for i, layer in enumerate(cfg["layers"]):
        l, m = f"l{i}", layer["mixer"]
        for n in ["norm1", "norm1b"] + (["norm2", "norm2b"] if layer["mlp"] is not None else []):
            vec(f"{l}.{n}", H, 0.5 if n.endswith("b") else 1.0, 0.2)
        if layer["type"] == "attention":
            rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for t, n in rows.items():
                mat(f"{l}.mix.{t}", n, H, 1.5)
                vec(f"{l}.mix.{t}.b", n, 0.0, 0.3)
            mat(f"{l}.mix.g", m["heads"] * m["vdim"], H)
            mat(f"{l}.mix.o", H, m["heads"] * m["vdim"])
        else:
            for t in ("z", "x"):
                mat(f"{l}.mix.{t}", m["width"], H)
                vec(f"{l}.mix.{t}.b", m["width"], -2.5 if t == "z" else 0.0, 1.0)
            mat(f"{l}.mix.g", m["width"], H)
            mat(f"{l}.mix.o", H, m["width"])
        if layer["mlp"] is not None:
            mat(f"{l}.mlp.up", layer["mlp"]["ff"], H)
            mat(f"{l}.mlp.down", H, layer["mlp"]["ff"])
            W[f"{l}.mlp.act"] = round_bf16([g.uniform(-1, 1), g.uniform(-1, 1)])
    return W
