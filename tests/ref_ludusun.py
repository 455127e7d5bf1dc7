"""Float64 oracle of the Ludusun design (layer-list family), written from its equations, one function per mechanism.  It shares no code
with the engine.  Shapes: a sequence is [T, width]; weights are stored [out, in] and applied as W x.

The design: the stream starts as embed[token] * scale; every layer is x <- x + mixer(norm x), x <- x + ff(norm x) with an RMS norm whose
weight is stored around zero (factor 1 + w).  Mixers:
  "attention"         causal softmax attention; rotate-half partial rotation with the long-context frequency blend and its magnitude on cos
                      and sin; every query / key head divided by its own root mean square AFTER the rotation; a learned sink per head.  A layer
                      may read another layer's keys and values instead of having its own
  "latent_attention"  queries and keys / values through normed low-rank latents, no positions, a sliding window, a sigmoid gate per head
  "parallel"          left: causal attention whose values are its keys, biases on q and k, a query temperature that grows with the position,
                      a sigmoid gate per output element; right: gated delta rule with a decay per head and key channel from a low-rank map,
                      short convolutions, heads normed one by one, a sigmoid gate from another low-rank map; a * left + b * right
Feed-forward: W_down (silu(W_gate h) * (W_up h)).  Logits: norm, the embedding table itself, tanh soft-cap."""
import numpy as np


# ---------------------------------------------------------------------------------------------------------------- small pieces
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_unit(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def zero_centred_norm(x, w, eps):
    return rms_unit(x, eps) * (1.0 + w)


def unit_vector(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def frequencies(rot):
    """Frequency per pair and the magnitude that cos and sin carry."""
    dims, base = rot["dims"], rot["base"]
    i = np.arange(dims // 2)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def place(turns):
        return dims * np.log(sc["original"] / (2 * np.pi * turns)) / (2 * np.log(base))
    lo = max(np.floor(place(sc["fast"])), 0.0)
    hi = min(np.ceil(place(sc["slow"])), dims - 1.0)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """x [T, heads, d]: entry i of the first half of the leading `dims` turns together with entry i of their second half."""
    y = x.copy()
    if not rot or rot["dims"] <= 0:
        return y
    f, mag = frequencies(rot)
    half = rot["dims"] // 2
    a = np.asarray(pos, dtype=np.float64)[:, None, None] * f[None, None, :]
    c, s = np.cos(a) * mag, np.sin(a) * mag
    u, v = x[..., :half], x[..., half:2 * half]
    y[..., :half] = u * c - v * s
    y[..., half:2 * half] = v * c + u * s
    return y


def visible(i, j, window=None):
    """Does position i see position j?  Every earlier one and itself; with a window only the last `window` of them."""
    i, j = np.asarray(i), np.asarray(j)
    return (j <= i) & (True if window is None else i - j < window)


def softmax_heads(scores, see, sink=None):
    """Rows of weights over the visible keys; sink: a number whose exponential joins the denominator."""
    s = np.where(see, scores, -np.inf)
    top = s.max(axis=1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    den = e.sum(axis=1, keepdims=True)
    if sink is not None:
        den = den + np.exp(sink - top)
    return e / den


def query_temperature(pos, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(pos) + 1.0) / every) + 1.0)


def causal_conv(u, w):
    """u [T, C], w [C, taps], last column for the current token; zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(pad[j:j + T] * w[None, :, j] for j in range(taps))


def delta_recurrence(q, k, v, g, beta, S=None):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H]: S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if S is None else S.copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hnp,hn->hp", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hnp,hn->hp", S, q[t])
    return o, S


# ---------------------------------------------------------------------------------------------------------------- mixers
def own_keys(cfg, c, W, p, h, pos):
    """Keys (rotated, then normed) and values of a layer that has its own."""
    T = h.shape[0]
    G = c.get("kv_heads", c["heads"])
    k = rms_unit(rotate((h @ W[p + "k"].T).reshape(T, G, c["dim"]), pos, c.get("rot")), cfg["norm"]["eps"])
    return k, (h @ W[p + "v"].T).reshape(T, G, c.get("vdim", c["dim"]))


def attention(cfg, c, W, p, h, pos, kept, i):
    T = h.shape[0]
    H, G, d, dv = c["heads"], c.get("kv_heads", c["heads"]), c["dim"], c.get("vdim", c["dim"])
    if c.get("kv_from") is None:
        kept[i] = own_keys(cfg, c, W, p, h, pos)
    k, v = kept[i if c.get("kv_from") is None else c["kv_from"]]
    q = rms_unit(rotate((h @ W[p + "q"].T).reshape(T, H, d), pos, c.get("rot")), cfg["norm"]["eps"])
    see = visible(np.asarray(pos)[:, None], np.asarray(pos)[None, :])
    out = np.zeros((T, H, dv))
    for n in range(H):
        g = n // (H // G)
        out[:, n] = softmax_heads((q[:, n] @ k[:, g].T) * c["scale"], see, W[p + "sink"][n]) @ v[:, g]
    return out.reshape(T, H * dv) @ W[p + "o"].T


def latent_attention(cfg, c, W, p, h, pos, kept, i):
    T = h.shape[0]
    eps = cfg["norm"]["eps"]
    H, d, dv = c["heads"], c["dim"], c.get("vdim", c["dim"])
    cq = rms_unit(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"][None, :]
    lat = rms_unit(h @ W[p + "dkv"].T, eps) * W[p + "dkv.norm"][None, :]
    q = (cq @ W[p + "uq"].T).reshape(T, H, d)
    k = (lat @ W[p + "uk"].T).reshape(T, H, d)
    v = (lat @ W[p + "uv"].T).reshape(T, H, dv)
    see = visible(np.asarray(pos)[:, None], np.asarray(pos)[None, :], c["mask"]["size"] if c.get("mask") else None)
    gate = sigmoid(h @ W[p + "g"].T)
    out = np.zeros((T, H, dv))
    for n in range(H):
        out[:, n] = (softmax_heads((q[:, n] @ k[:, n].T) * c["scale"], see) @ v[:, n]) * gate[:, n:n + 1]
    return out.reshape(T, H * dv) @ W[p + "o"].T


def keys_as_values_attention(cfg, c, W, p, h, pos):
    T = h.shape[0]
    H, G, d = c["heads"], c.get("kv_heads", c["heads"]), c["dim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"][None, :]).reshape(T, H, d)
    k = (h @ W[p + "k"].T + W[p + "k.b"][None, :]).reshape(T, G, d)
    if c.get("q_temp"):
        q = q * query_temperature(pos, c["q_temp"]["coef"], c["q_temp"]["every"])[:, None, None]
    see = visible(np.asarray(pos)[:, None], np.asarray(pos)[None, :])
    out = np.zeros((T, H, d))
    for n in range(H):
        g = n // (H // G)
        out[:, n] = softmax_heads((q[:, n] @ k[:, g].T) * c["scale"], see) @ k[:, g]
    return (out.reshape(T, H * d) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def delta_decay(W, p, h, H, d):
    a = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"][None, :]
    return np.exp(-np.exp(W[p + "A_log"])[None, :, None] * softplus(a).reshape(-1, H, d))


def gated_delta(cfg, c, W, p, h):
    T = h.shape[0]
    H, G, d, dv = c["heads"], c.get("kv_heads", c["heads"]), c["dim"], c.get("vdim", c["dim"])
    q, k, v = (silu(causal_conv(h @ W[p + s].T, W[p + s + ".conv"])) for s in "qkv")
    spread = np.arange(H) // (H // G)
    q = (unit_vector(q.reshape(T, G, d)) / np.sqrt(d))[:, spread]
    k = unit_vector(k.reshape(T, G, d))[:, spread]
    o, _ = delta_recurrence(q, k, v.reshape(T, H, dv), delta_decay(W, p, h, H, d), sigmoid(h @ W[p + "b"].T))
    o = rms_unit(o, cfg["norm"]["eps"]) * W[p + "norm"][None, None, :]
    return (o.reshape(T, H * dv) * sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)) @ W[p + "o"].T


def parallel(cfg, c, W, p, h, pos, kept, i):
    return (c.get("left_scale", 1.0) * keys_as_values_attention(cfg, c["left"], W, p + "left.", h, pos)
            + c.get("right_scale", 1.0) * gated_delta(cfg, c["right"], W, p + "right.", h))


MIXERS = {"attention": attention, "latent_attention": latent_attention, "parallel": parallel}


def feed_forward(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ---------------------------------------------------------------------------------------------------------------- the model
def forward(cfg, W, toks):
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    eps = cfg["norm"]["eps"]
    pos = np.arange(len(toks))
    x = W["embed"][np.asarray(toks)] * cfg.get("embedding", {}).get("scale", 1.0)
    taps, kept = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](cfg, layer["mixer"], W, p + "mix.", zero_centred_norm(x, W[p + "norm1"], eps), pos, kept, i)
        if layer.get("mlp"):
            x = x + feed_forward(W, p + "mlp.", zero_centred_norm(x, W[p + "norm2"], eps))
        taps.append(x.copy())
    y = zero_centred_norm(x, W["final.norm"], eps) @ W["embed"].T
    cap = cfg.get("logit_softcap", 0.0)
    return cap * np.tanh(y / cap) if cap else y, np.stack(taps)


# ---------------------------------------------------------------------------------------------------------------- weights for tests
def tensor_shapes(cfg, rank=8):
    """name -> shape of every tensor of a configuration.  rank: inner size of the two low-rank maps of a parallel mixer (a number, a pair
    (decay, gate), or a dictionary of either by layer)."""
    Wd, V = cfg["width"], cfg["vocab"]
    sh = {"embed": (V, Wd), "final.norm": (Wd,)}
    for i, layer in enumerate(cfg["layers"]):
        p, c, kind = f"l{i}.", layer["mixer"], layer["type"]
        a = p + "mix."
        sh[p + "norm1"] = (Wd,)
        if kind == "attention":
            H, d = c["heads"], c["dim"]
            G, dv = c.get("kv_heads", H), c.get("vdim", d)
            sh[a + "q"], sh[a + "sink"], sh[a + "o"] = (H * d, Wd), (H,), (Wd, H * dv)
            if c.get("kv_from") is None:
                sh[a + "k"], sh[a + "v"] = (G * d, Wd), (G * dv, Wd)
        elif kind == "latent_attention":
            H, d, R, Rq = c["heads"], c["dim"], c["kv_rank"], c["q_rank"]
            dv = c.get("vdim", d)
            sh[a + "dq"], sh[a + "dq.norm"], sh[a + "uq"] = (Rq, Wd), (Rq,), (H * d, Rq)
            sh[a + "dkv"], sh[a + "dkv.norm"] = (R, Wd), (R,)
            sh[a + "uk"], sh[a + "uv"], sh[a + "g"], sh[a + "o"] = (H * d, R), (H * dv, R), (H, Wd), (Wd, H * dv)
        else:
            lc, rc = c["left"], c["right"]
            l, r = a + "left.", a + "right."
            H, d = lc["heads"], lc["dim"]
            G = lc.get("kv_heads", H)
            sh[l + "q"], sh[l + "q.b"], sh[l + "k"], sh[l + "k.b"] = (H * d, Wd), (H * d,), (G * d, Wd), (G * d,)
            sh[l + "g"], sh[l + "o"] = (H * d, Wd), (Wd, H * d)
            H, d, taps = rc["heads"], rc["dim"], rc["conv"]
            G, dv = rc.get("kv_heads", H), rc.get("vdim", d)
            k = rank.get(i, 8) if isinstance(rank, dict) else rank
            ka, kg = k if isinstance(k, (tuple, list)) else (k, k)
            for s, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                sh[r + s], sh[r + s + ".conv"] = (n, Wd), (n, taps)
            sh[r + "b"], sh[r + "A_log"], sh[r + "dt_bias"], sh[r + "norm"] = (H, Wd), (H,), (H * d,), (dv,)
            sh[r + "a1"], sh[r + "a2"], sh[r + "g1"], sh[r + "g2"] = (ka, Wd), (H * d, ka), (kg, Wd), (H * dv, kg)
            sh[r + "o"] = (Wd, H * dv)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            sh[p + "norm2"], sh[p + "mlp.gate"], sh[p + "mlp.up"], sh[p + "mlp.down"] = (Wd,), (ff, Wd), (ff, Wd), (Wd, ff)
    return sh


def to_bf16_bits(a):
    """Round-to-nearest-even bfloat16 bit patterns (uint16) of a float array."""
    b = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    b = (b + 0x7FFF + ((b >> 16) & 1)) >> 16
    return b.astype(np.uint16)


def from_bf16_bits(b):
    return (b.astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def random_weights(cfg, seed=0, gain=1.0, rank=8):
    """Random weights that bfloat16 holds exactly: (bits for the engine, float64 values for the oracle)."""
    rng = np.random.default_rng(seed)
    bits, W = {}, {}
    for name, shape in tensor_shapes(cfg, rank).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            a = rng.normal(0, gain / np.sqrt(shape[-1]), shape)
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            a = rng.uniform(-0.4, 0.4, shape)
        elif leaf == "norm":
            a = rng.uniform(0.6, 1.5, shape)
        elif leaf == "sink":
            a = rng.normal(0, 1.5, shape)
        elif leaf == "A_log":
            a = rng.uniform(-2.0, 1.0, shape)
        elif leaf == "dt_bias":
            a = rng.uniform(-3.0, 0.5, shape)
        elif leaf == "conv":
            a = rng.normal(0, 0.6, shape)
        elif name.endswith((".q.b", ".k.b")):
            a = rng.normal(0, 0.8, shape)
        else:
            a = rng.normal(0, 1.0 / np.sqrt(shape[-1]), shape)
        b = to_bf16_bits(np.asarray(a))
        bits[name] = b
        W[name] = from_bf16_bits(b).reshape(shape)
    return bits, W


def set_weight(bits, W, name, value):
    b = to_bf16_bits(np.asarray(value))
    bits[name] = b
    W[name] = from_bf16_bits(b).reshape(np.shape(value))


def write_model_dir(path, cfg, bits, shapes):
    """config.json and model.safetensors (an 8-byte header length, a JSON table, then the bfloat16 data)."""
    import json
    import os
    import struct
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    table, blobs, at = {}, [], 0
    for name, b in bits.items():
        raw = np.ascontiguousarray(b).tobytes()
        table[name] = {"dtype": "BF16", "shape": list(shapes[name]), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    head = json.dumps(table).encode()
    head += b" " * (-len(head) % 8)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        f.write(b"".join(blobs))


def rel_err(got, want):
    """Per row: rms of the difference (mean removed) over the rms spread of the wanted row."""
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    s = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / np.maximum(np.sqrt((s * s).mean(axis=-1)), 1e-30)
