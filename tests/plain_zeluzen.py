"""A plain, slow implementation of the Zeluzen decoder in float64 numpy: one function per mechanism, the recurrence a
literal loop over tokens and every attention row a literal walk over the keys it may see.  It shares nothing with the
library; the GPU tests compare the engine with it.

A model is (cfg, W): cfg the config.json object, W a dict name -> float64 array.  Everything runs on one
sequence: x is [n, width], the first token has position 0.
"""
import math

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, np.float64)))


def silu(z):
    return z * sigmoid(z)


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


# ---------------------------------------------------------------- the time-mixing recurrence


def shifted(x):
    """Row t is row t - 1 of x; row 0 is zeros."""
    return np.concatenate([np.zeros((1, x.shape[1])), x[:-1]])


def blend(x, mu):
    """Every channel between the token's own row (mu 0) and the previous token's (mu 1)."""
    return (1.0 - mu) * x + mu * shifted(x)


def channel_decay(mix, w1, w2, w0):
    """In (0, 1), one number per token, head and key channel (flat over heads and channels)."""
    return np.exp(-np.exp(np.tanh(mix @ w1.T) @ w2.T + w0))


def wkv_scan(r, k, v, w, u):
    """r, k, w [n, heads, d], v [n, heads, dv], u [heads, d].  A token reads the state that its predecessors left, plus its own
    outer product weighted by u; then the state's rows decay and the outer product joins it unweighted."""
    n, H, dv = v.shape
    d = r.shape[2]
    out = np.zeros((n, H, dv))
    for a in range(H):
        S = np.zeros((d, dv))
        for t in range(n):
            own = np.outer(k[t, a], v[t, a])
            out[t, a] = r[t, a] @ (S + u[a][:, None] * own)
            S = w[t, a][:, None] * S + own
    return out


def wkv(x, W, pre, m, eps):
    H, d = m["heads"], m["dim"]
    n = x.shape[0]
    mixed = {s: blend(x, W[pre + "mu." + s]) for s in "rkvgw"}
    r, k, v = [(mixed[s] @ W[pre + s].T).reshape(n, H, d) for s in "rkv"]
    w = channel_decay(mixed["w"], W[pre + "w1"], W[pre + "w2"], W[pre + "w0"]).reshape(n, H, d)
    o = rms_unit(wkv_scan(r, k, v, w, W[pre + "u"]), eps).reshape(n, H * d)
    return (o * W[pre + "norm"] * silu(mixed["g"] @ W[pre + "g"].T)) @ W[pre + "o"].T


# ---------------------------------------------------------------- attention


def row_softmax_with_zero_sink(s):
    """exp(s_j) / (1 + sum exp(s)): an extra score of 0 that has no value."""
    top = max(s.max(), 0.0)
    e = np.exp(s - top)
    return e / (math.exp(-top) + e.sum())


def chunk_start(p, size):
    return (p // size) * size if size else 0


def frequencies(rot):
    """One angle per position for each of the dims / 2 pairs: slow waves stretched, fast ones kept, a linear passage between."""
    dims, sc = rot["dims"], rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = rot["base"] ** (-2.0 * i / dims)
        if sc:
            turns = sc["original"] * f / (2.0 * math.pi)       # full turns within the original length
            if turns <= sc["high"]:
                keep = max(0.0, (turns - sc["low"]) / (sc["high"] - sc["low"])) if turns >= sc["low"] else 0.0
                f = keep * f + (1.0 - keep) * f / sc["factor"]
        out.append(f)
    return out


def rotate_pairs(x, p, rot):
    """Neighbouring channels (2i, 2i + 1) of the first `dims` channels turn together."""
    y = np.array(x, np.float64)
    for i, f in enumerate(frequencies(rot)):
        c, s = math.cos(p * f), math.sin(p * f)
        a, b = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = a * c - b * s
        y[..., 2 * i + 1] = b * c + a * s
    return y


def keys_and_values(x, W, pre, m, eps):
    """What a layer with projections of its own keeps per token: keys [n, G, d], normed and rotated, and values [n, G, dv]."""
    G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
    n = x.shape[0]
    k = rms_norm((x @ W[pre + "k"].T).reshape(n, G, d), W[pre + "k.norm"], eps)
    k = np.stack([rotate_pairs(k[t], t, m["rot"]) for t in range(n)])
    return k, (x @ W[pre + "v"].T).reshape(n, G, dv)


def attend(x, W, pre, m, eps, kv):
    H, G, d, dv, scale = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"]
    size = m["mask"]["size"] if m.get("mask") else 0
    n = x.shape[0]
    k, v = kv
    q = rms_norm((x @ W[pre + "q"].T).reshape(n, H, d), W[pre + "q.norm"], eps)
    out = np.zeros((n, H, dv))
    for i in range(n):
        lo = chunk_start(i, size)
        qi = rotate_pairs(q[i], i, m["rot"])
        for a in range(H):
            g = a // (H // G)
            out[i, a] = row_softmax_with_zero_sink((k[lo:i + 1, g] @ qi[a]) * scale) @ v[lo:i + 1, g]
    return out.reshape(n, H * dv) @ W[pre + "o"].T


# ---------------------------------------------------------------- feed-forward


def dense(x, W, pre):
    return (silu(x @ W[pre + "gate"].T) * (x @ W[pre + "up"].T)) @ W[pre + "down"].T


def route(x, W, pre, router):
    """(scores [n, experts], choices [n, top]): the choice looks at the corrected scores, the weights do not."""
    z = x @ W[pre + "router"].T
    s = np.exp(z - z.max(-1, keepdims=True))
    s = s / s.sum(-1, keepdims=True)
    return s, np.argsort(-(s + W[pre + "correction"]), axis=-1, kind="stable")[:, :router["top"]]


def expert(x, W, pre):
    return np.maximum(x @ W[pre + "up"].T, 0.0) ** 2 @ W[pre + "down"].T


def routed(x, W, pre, mlp):
    s, chosen = route(x, W, pre, mlp["router"])
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        for e in chosen[t]:
            own = expert(x[t], W, pre + "e%d." % e) if e < mlp["router"]["experts"] else x[t]
            y[t] += s[t, e] * own
    return y


# ---------------------------------------------------------------- the model


def forward(cfg, W, tokens, layers_out=None, margins=None):
    """Logits [n, vocab] of one sequence from its first token.  layers_out (a list) receives the stream after every layer;
    margins (a list) how far the last chosen and the first refused expert of every routed token are apart."""
    eps = cfg["norm"]["eps"]
    x = rms_norm(W["embed"][np.asarray(tokens)], W["embed.norm"], eps)
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        pre, m = "l%d." % i, L["mixer"]
        if L["type"] == "wkv":
            y = wkv(x, W, pre + "mix.", m, eps)
        elif L["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = keys_and_values(x, W, pre + "mix.", m, eps)
            y = attend(x, W, pre + "mix.", m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            raise ValueError(L["type"])
        x = x + rms_norm(y, W[pre + "norm1"], eps)
        if L.get("mlp"):
            if L["mlp"]["kind"] == "dense":
                y = dense(x, W, pre + "mlp.")
            else:
                y = routed(x, W, pre + "mlp.", L["mlp"])
                if margins is not None:
                    s, _ = route(x, W, pre + "mlp.", L["mlp"]["router"])
                    c, top = np.sort(s + W[pre + "mlp.correction"], axis=-1)[:, ::-1], L["mlp"]["router"]["top"]
                    if top < c.shape[1]:
                        margins.append(c[:, top - 1] - c[:, top])
            x = x + rms_norm(y, W[pre + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T


def greedy_generate(cfg, W, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(np.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]


# ---------------------------------------------------------------- test infrastructure: configurations and weights


def wkv_mixer(heads=3, dim=16):
    return {"heads": heads, "dim": dim}


def attn_mixer(heads=6, kv_heads=2, dim=24, vdim=16, size=20, scale=0.3, base=500.0, dims=12, scaling=(4.0, 1.0, 3.0, 60), kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if size:
        m["mask"] = {"size": size}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense_mlp(ff=40):
    return {"kind": "dense", "ff": ff}


def moe_mlp(ff=24, experts=5, identity=2, top=3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}


def make_config(layers, width=48, vocab=97, eps=1e-5, max_positions=2048):
    """layers: a list of (type, mixer, mlp or None)."""
    return {"architecture": "Zeluzen", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers], "max_positions": max_positions}


def tensor_shapes(cfg, rank=7):
    """name -> (shape, kind); kind says how random_weights draws the tensor.  `rank`: the inner size of the decay's map."""
    width = cfg["width"]
    out = {"embed": ((cfg["vocab"], width), "embed"), "embed.norm": ((width,), "norm"), "final.norm": ((width,), "norm"),
           "head": ((cfg["vocab"], width), "mat")}
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        x, H, d = p + "mix.", m["heads"], m["dim"]
        out[p + "norm1"] = ((width,), "norm")
        if L["type"] == "wkv":
            for s in "rkvgw":
                out[x + "mu." + s] = ((width,), "mu")
            for s in "rkvg":
                out[x + s] = ((H * d, width), "mat")
            out.update({x + "w1": ((rank, width), "mat"), x + "w2": ((H * d, rank), "mat"), x + "w0": ((H * d,), "w0"), x + "u": ((H, d), "u"),
                        x + "norm": ((H * d,), "norm"), x + "o": ((width, H * d), "mat")})
        else:
            G, dv = m["kv_heads"], m["vdim"]
            out.update({x + "q": ((H * d, width), "mat"), x + "q.norm": ((d,), "norm"), x + "o": ((width, H * dv), "mat")})
            if m.get("kv_from") is None:
                out.update({x + "k": ((G * d, width), "mat"), x + "k.norm": ((d,), "norm"), x + "v": ((G * dv, width), "mat")})
        if L.get("mlp"):
            f, mlp = p + "mlp.", L["mlp"]
            out[p + "norm2"] = ((width,), "norm")
            if mlp["kind"] == "dense":
                out.update({f + "gate": ((mlp["ff"], width), "mat"), f + "up": ((mlp["ff"], width), "mat"), f + "down": ((width, mlp["ff"]), "mat")})
            else:
                ff, r = mlp["expert"]["ff"], mlp["router"]
                for e in range(r["experts"]):
                    out[f + "e%d.up" % e] = ((ff, width), "mat")
                    out[f + "e%d.down" % e] = ((width, ff), "mat")
                n = r["experts"] + r.get("identity", 0)
                out.update({f + "router": ((n, width), "router"), f + "correction": ((n,), "correction")})
    return out


def bf16_round(a):
    """float32 array rounded to the nearest bfloat16 value (ties to even), still float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def random_weights(cfg, seed, gain=1.0, rank=7):
    """Random weights, rounded to bfloat16 values.  Drawn so that faults show: norm weights far from 1, blends all over (0, 1),
    decays spread from quick to slow, a bonus far from 1, corrections that change many choices."""
    rng, w = np.random.default_rng(seed), {}
    for name, (shape, kind) in tensor_shapes(cfg, rank).items():
        z = rng.standard_normal(shape)
        if kind == "mat":
            a = z * gain / math.sqrt(shape[-1])
        elif kind == "embed":
            a = z
        elif kind == "router":
            a = z * 1.5 / math.sqrt(shape[-1])
        elif kind == "norm":
            a = 1.0 + 0.3 * z
        elif kind == "mu":
            a = 0.5 + 0.25 * z
        elif kind == "w0":
            a = 1.5 * z - 2.0
        elif kind == "u":
            a = 0.8 * z + 0.5
        elif kind == "correction":
            a = 0.15 * z
        else:
            raise ValueError(kind)
        w[name] = bf16_round(np.asarray(a, np.float32))
    return w


def steady_routing(cfg, w, channels=8, margin=0.01):
    """Edits the weights so that rounding cannot turn a router's choice: the routers read the first few channels alone, which
    hold the embedding as it is (no sublayer writes there).  Returns the tokens whose choices all have at least this margin."""
    eps, good = cfg["norm"]["eps"], np.ones(cfg["vocab"], bool)
    for i, L in enumerate(cfg["layers"]):
        for role in ("norm1", "norm2"):
            if "l%d.%s" % (i, role) in w:
                w["l%d.%s" % (i, role)][:channels] = 0.0
    x = rms_norm(np.asarray(w["embed"], np.float64), np.asarray(w["embed.norm"], np.float64), eps)
    for i, L in enumerate(cfg["layers"]):
        if L.get("mlp") and L["mlp"]["kind"] == "moe":
            r = w["l%d.mlp.router" % i]
            r[:, channels:] = 0.0
            r[:, :channels] *= bf16_round(np.float32(math.sqrt(r.shape[1] / channels)))
            w["l%d.mlp.router" % i] = bf16_round(r)
            W = {k: np.asarray(w["l%d.mlp.%s" % (i, k)], np.float64) for k in ("router", "correction")}
            s, _ = route(x, W, "", L["mlp"]["router"])
            c, top = np.sort(s + W["correction"], axis=-1)[:, ::-1], L["mlp"]["router"]["top"]
            if top < c.shape[1]:
                good &= c[:, top - 1] - c[:, top] > margin
    return np.flatnonzero(good).tolist()


def write_model(folder, cfg, w):
    """config.json and model.safetensors (bfloat16) of (cfg, w) in `folder`."""
    import json
    import os
    import struct
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, off = {}, [], 0
    for name, a in w.items():
        blob = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [off, off + len(blob)]}
        blobs.append(blob)
        off += len(blob)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)))
        f.write(hj)
        for b in blobs:
            f.write(b)
