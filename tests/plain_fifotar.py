"""A plain, slow implementation of the Fifotar decoder in float64 numpy: one function per mechanism, the recurrence a
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


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ---------------------------------------------------------------- the gated delta rule


def causal_conv(x, taps):
    """y_t[c] = sum_j taps[c, K - 1 - j] x_{t - j}[c], zeros before the first token."""
    n, K = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for t in range(n):
        for j in range(min(K, t + 1)):
            y[t] += taps[:, K - 1 - j] * x[t - j]
    return y


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def head_decay(a, a_log, dt_bias):
    """One decay per head and token, in (0, 1)."""
    return np.exp(-np.exp(a_log) * softplus(a + dt_bias))


def delta_scan(q, k, v, g, beta, share):
    """q, k [n, kv heads, d], v [n, heads, dv], g and beta [n, heads]; query/key head of head a: a // share.  The state of
    every head decays, is corrected towards the token's value along its key, and is read afterwards."""
    n, H, dv = v.shape
    d = q.shape[2]
    out = np.zeros((n, H, dv))
    for a in range(H):
        S = np.zeros((d, dv))
        for t in range(n):
            kt, qt = k[t, a // share], q[t, a // share]
            S = g[t, a] * S
            u = beta[t, a] * (v[t, a] - S.T @ kt)
            S = S + np.outer(kt, u)
            out[t, a] = S.T @ qt
    return out


def delta(h, W, pre, m, eps):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q = silu(causal_conv(h @ W[pre + "q"].T, W[pre + "q.conv"])).reshape(n, G, d)
    k = silu(causal_conv(h @ W[pre + "k"].T, W[pre + "k.conv"])).reshape(n, G, d)
    v = silu(causal_conv(h @ W[pre + "v"].T, W[pre + "v.conv"])).reshape(n, H, dv)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = sigmoid(h @ W[pre + "b"].T)
    g = head_decay(h @ W[pre + "a"].T, W[pre + "A_log"], W[pre + "dt_bias"])
    o = delta_scan(q, k, v, g, beta, H // G)
    o = rms_norm(o, W[pre + "norm"], eps).reshape(n, H * dv) * silu(h @ W[pre + "g"].T)
    return o @ W[pre + "o"].T


# ---------------------------------------------------------------- attention


def row_softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def row_softmax_with_zero_sink(s):
    """exp(s_j) / (1 + sum exp(s)): an extra score of 0 that has no value."""
    top = max(s.max(), 0.0)
    e = np.exp(s - top)
    return e / (math.exp(-top) + e.sum())


def chunk_start(p, size):
    return (p // size) * size if size else 0


def chunked_attention(h, W, pre, m, v_first):
    """Attention without positions inside chunks of the sequence, capped scores, a sink of score 0, an element-wise gate.
    v_first: the values of the first layer that mixes values (None in that layer itself, and where nothing is mixed).
    Returns the output and this layer's own values."""
    H, G, d, dv, scale = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"]
    size = m["mask"]["size"] if m.get("mask") else 0
    n = h.shape[0]
    q = (h @ W[pre + "q"].T).reshape(n, H, d)
    k = (h @ W[pre + "k"].T).reshape(n, G, d)
    v = h @ W[pre + "v"].T
    own = v
    if v_first is not None:
        lam = float(np.asarray(W[pre + "vmix"]).reshape(-1)[0])
        v = (1.0 - lam) * v + lam * v_first
    v = v.reshape(n, G, dv)
    out = np.zeros((n, H, dv))
    for i in range(n):
        lo = chunk_start(i, size)
        for a in range(H):
            g = a // (H // G)
            s = np.array([q[i, a] @ k[j, g] for j in range(lo, i + 1)]) * scale
            if m.get("softcap"):
                s = soft_cap(s, m["softcap"])
            out[i, a] = row_softmax_with_zero_sink(s) @ v[lo:i + 1, g]
    out = out.reshape(n, H * dv) * sigmoid(h @ W[pre + "g"].T)
    return out @ W[pre + "o"].T, own


def yarn_frequencies(rot):
    """(frequencies of the dims / 2 pairs, the factor on cos and sin)."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    def dim(t): return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x, p, rot):
    """Channel i of the first `dims` channels of x is turned together with channel i + dims / 2."""
    f, mag = yarn_frequencies(rot)
    half = rot["dims"] // 2
    y = np.array(x, np.float64)
    for i in range(half):
        c, s = mag * math.cos(p * f[i]), mag * math.sin(p * f[i])
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


def latent_attention(h, W, pre, m, eps):
    """Attention whose queries come out of a normed latent and whose keys and values are maps of a second one, beside one
    rotated key part that all heads share; all earlier positions; a sigmoid gate per head."""
    H, d, dr, dv, rank, scale = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"]
    n = h.shape[0]
    cq = rms_norm(h @ W[pre + "dq"].T, W[pre + "dq.norm"], eps)
    q = (cq @ W[pre + "uq"].T).reshape(n, H, d + dr)
    down = h @ W[pre + "dkv"].T
    c = rms_norm(down[:, :rank], W[pre + "dkv.norm"], eps)
    kr = np.stack([rotate_halves(down[t, rank:], t, m["rot"]) for t in range(n)])
    k = (c @ W[pre + "uk"].T).reshape(n, H, d)
    v = (c @ W[pre + "uv"].T).reshape(n, H, dv)
    gate = sigmoid(h @ W[pre + "g"].T)
    out = np.zeros((n, H, dv))
    for i in range(n):
        for a in range(H):
            qr = rotate_halves(q[i, a, d:], i, m["rot"])
            s = np.array([q[i, a, :d] @ k[j, a] + qr @ kr[j] for j in range(i + 1)]) * scale
            out[i, a] = (row_softmax(s) @ v[:i + 1, a]) * gate[i, a]
    return out.reshape(n, H * dv) @ W[pre + "o"].T


# ---------------------------------------------------------------- the model


def clamped_mlp(h, W, pre, limit):
    g = np.minimum(h @ W[pre + "gate"].T, limit)
    u = np.clip(h @ W[pre + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[pre + "down"].T


def forward(cfg, W, tokens, layers_out=None):
    """Logits [n, vocab] of one sequence from its first token; layers_out (a list) receives the stream after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    v_first = None
    for i, L in enumerate(cfg["layers"]):
        pre, m = "l%d." % i, L["mixer"]
        h = rms_norm(x, W[pre + "norm1"], eps)
        if L["type"] == "delta":
            y = delta(h, W, pre + "mix.", m, eps)
        elif L["type"] == "latent_attention":
            y = latent_attention(h, W, pre + "mix.", m, eps)
        elif L["type"] == "attention":
            y, own = chunked_attention(h, W, pre + "mix.", m, v_first if m.get("v_mix") else None)
            if m.get("v_mix") and v_first is None:
                v_first = own
        else:
            raise ValueError(L["type"])
        x = x + mult * rms_norm(y, W[pre + "norm1b"], eps)
        if L.get("mlp"):
            y = clamped_mlp(rms_norm(x, W[pre + "norm2"], eps), W, pre + "mlp.", L["mlp"]["limit"])
            x = x + mult * rms_norm(y, W[pre + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return soft_cap(rms_norm(x, W["final.norm"], eps) @ W["embed"].T, cfg["logit_softcap"])


def greedy_generate(cfg, W, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(np.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]


# ---------------------------------------------------------------- test infrastructure: configurations and weights


def delta_mixer(heads=6, kv_heads=2, dim=12, vdim=20, conv=4):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def chunk_mixer(heads=4, kv_heads=2, dim=24, vdim=16, size=20, scale=0.3, softcap=9.0, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap, "v_mix": v_mix}
    if size:
        m["mask"] = {"size": size}
    return m


def latent_mixer(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=28, kv_rank=40, scale=0.25, base=100.0, scaling=(3.0, 64, 4.0, 1.0)):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return m


def dense(ff=40, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def make_config(layers, width=48, vocab=97, eps=1e-5, scale=3.0, mult=0.6, logit_softcap=20.0, max_positions=2048):
    """layers: a list of (type, mixer, mlp or None)."""
    return {"architecture": "Fifotar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "residual_mult": mult,
            "logit_softcap": logit_softcap, "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers], "max_positions": max_positions}


def tensor_shapes(cfg):
    """name -> (shape, kind); kind says how random_weights draws the tensor."""
    width = cfg["width"]
    out = {"embed": ((cfg["vocab"], width), "embed"), "final.norm": ((width,), "norm")}
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        x = p + "mix."
        out[p + "norm1"] = out[p + "norm1b"] = ((width,), "norm")
        H, dv = m["heads"], m["vdim"]
        if L["type"] == "delta":
            G, d, K = m["kv_heads"], m["dim"], m["conv"]
            for t, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                out[x + t] = ((rows, width), "mat")
                out[x + t + ".conv"] = ((rows, K), "conv")
            out.update({x + "b": ((H, width), "mat"), x + "A_log": ((H,), "a_log"), x + "norm": ((dv,), "norm"), x + "a": ((H, width), "mat"),
                        x + "dt_bias": ((H,), "dt"), x + "g": ((H * dv, width), "mat"), x + "o": ((width, H * dv), "mat")})
        elif L["type"] == "attention":
            G, d = m["kv_heads"], m["dim"]
            out.update({x + "q": ((H * d, width), "mat"), x + "k": ((G * d, width), "mat"), x + "v": ((G * dv, width), "mat"),
                        x + "g": ((H * dv, width), "mat"), x + "o": ((width, H * dv), "mat")})
            if m.get("v_mix"):
                out[x + "vmix"] = ((), "lambda")
        else:
            d, dr, qr, rank = m["dim"], m["rot_dim"], m["q_rank"], m["kv_rank"]
            out.update({x + "dq": ((qr, width), "mat"), x + "dq.norm": ((qr,), "norm"), x + "uq": ((H * (d + dr), qr), "mat"),
                        x + "dkv": ((rank + dr, width), "mat"), x + "dkv.norm": ((rank,), "norm"), x + "uk": ((H * d, rank), "mat"),
                        x + "uv": ((H * dv, rank), "mat"), x + "g": ((H, width), "mat"), x + "o": ((width, H * dv), "mat")})
        if L.get("mlp"):
            f, ff = p + "mlp.", L["mlp"]["ff"]
            out[p + "norm2"] = out[p + "norm2b"] = ((width,), "norm")
            out.update({f + "gate": ((ff, width), "gate"), f + "up": ((ff, width), "gate"), f + "down": ((width, ff), "mat")})
    return out


def bf16_round(a):
    """float32 array rounded to the nearest bfloat16 value (ties to even), still float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def random_weights(cfg, seed, gain=1.0):
    """Random weights, rounded to bfloat16 values.  Drawn so that faults show: norm weights far from 1, convolution taps of
    like size, decays spread over (0, 1), gate and up maps that reach the feed-forward's limit, a mixing factor far from 0."""
    rng, w = np.random.default_rng(seed), {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        n_in = shape[-1] if shape else 1
        z = rng.standard_normal(shape)
        if kind == "mat":
            a = z * gain / math.sqrt(n_in)
        elif kind == "gate":
            a = z * 1.5 * gain / math.sqrt(n_in)
        elif kind == "embed":
            a = z
        elif kind == "norm":
            a = 1.0 + 0.3 * z
        elif kind == "conv":
            a = 0.8 * z / math.sqrt(n_in) + 0.3
        elif kind == "a_log":
            a = 0.5 * z - 1.0
        elif kind == "dt":
            a = z - 1.0
        elif kind == "lambda":
            a = 0.5 + 0.15 * z
        else:
            raise ValueError(kind)
        w[name] = bf16_round(np.asarray(a, np.float32))
    return w


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
