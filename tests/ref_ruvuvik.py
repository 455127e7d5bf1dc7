"""Float64 oracle of the Ruvuvik design (layer-list family), written from its equations, one function per mechanism.  It shares no code
with the engine.  Shapes: a sequence is [T, width]; weights are stored [out, in] and applied as W x.

The design: the stream starts as norm(embed[token]); every layer is x <- x + mixer(norm(x)), x <- x + ff(norm(x)) with an RMS norm whose
weight is stored around zero (factor 1 + w); a layer may borrow all its tensors from another layer and still has a cache or state of its
own.  Mixers:
  "attention"         softmax attention inside fixed chunks of positions; RMS norm with weight over the whole q / k projection, interleaved
                      partial rotation, a temperature per head, soft-capped scores, a sigmoid gate per head
  "latent_attention"  keys and values expanded from a normed low-rank latent, one rotated key part shared by all heads, a learned sink per
                      head in the softmax denominator
  "wkv"               token shift with a blend per input, a decay per channel from a low-rank map of the token, a matrix state per head read
                      before the token's own write with a bonus for the current token; heads normed one by one, weight, SiLU gate
Feed-forward: W_down xIELU(W_up h) with two learned numbers."""
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


def xielu(z, p, q):
    """z > 0: softplus(p) z^2 + z / 2;  z <= 0: (1/2 + softplus(q)) (e^z - 1 - z) + z / 2."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def rotate(x, pos, dims, base):
    """x [T, heads, d]: the pairs (2i, 2i+1) of the first `dims` entries of every head turn by pos * base^(-2i/dims)."""
    y = x.copy()
    if dims <= 0:
        return y
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    a = np.asarray(pos, dtype=np.float64)[:, None, None] * f[None, None, :]
    c, s = np.cos(a), np.sin(a)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * c - v * s
    y[..., 1:dims:2] = v * c + u * s
    return y


def visible(i, j, chunk):
    """Does position i see position j?  chunk None: every earlier position and itself; otherwise only those of its own chunk of positions."""
    i, j = np.asarray(i), np.asarray(j)
    return (j <= i) & (True if chunk is None else i // chunk == j // chunk)


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


def wkv_recurrence(r, k, v, w, u, S=None):
    """r, k, w [T, H, d], v [T, H, d], u [H, d]: o = (S + diag(u) k v^T)^T r with the state before the token's write, then
    S <- diag(w) S + k v^T."""
    T, H, d = r.shape
    S = np.zeros((H, d, v.shape[2])) if S is None else S.copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        o[t] = np.einsum("hnp,hn->hp", S, r[t]) + np.sum(r[t] * u * k[t], axis=-1, keepdims=True) * v[t]
        S = w[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
    return o, S


# ---------------------------------------------------------------------------------------------------------------- mixers
def attention(cfg, c, W, p, h, pos):
    T = h.shape[0]
    eps = cfg["norm"]["eps"]
    H, G, d, dv = c["heads"], c.get("kv_heads", c["heads"]), c["dim"], c.get("vdim", c["dim"])
    q = rms_unit(h @ W[p + "q"].T, eps) * W[p + "q.norm"][None, :]
    k = rms_unit(h @ W[p + "k"].T, eps) * W[p + "k.norm"][None, :]
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), (h @ W[p + "v"].T).reshape(T, G, dv)
    rot = c.get("rot")
    if rot:
        q, k = rotate(q, pos, rot["dims"], rot["base"]), rotate(k, pos, rot["dims"], rot["base"])
    chunk = c["mask"]["size"] if c.get("mask") else None
    see = visible(np.asarray(pos)[:, None], np.asarray(pos)[None, :], chunk)
    gate = sigmoid(h @ W[p + "g"].T)
    out = np.zeros((T, H, dv))
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T) * c["scale"] * W[p + "temp"][n]
        cap = c.get("softcap", 0.0)
        if cap:
            s = cap * np.tanh(s / cap)
        out[:, n] = (softmax_heads(s, see) @ v[:, g]) * gate[:, n:n + 1]
    return out.reshape(T, H * dv) @ W[p + "o"].T


def latent_attention(cfg, c, W, p, h, pos):
    T = h.shape[0]
    eps = cfg["norm"]["eps"]
    H, d, dr, dv, R = c["heads"], c["dim"], c["rot_dim"], c.get("vdim", c["dim"]), c["kv_rank"]
    q = (h @ W[p + "q"].T).reshape(T, H, d + dr)
    down = h @ W[p + "dkv"].T
    lat = rms_unit(down[:, :R], eps) * W[p + "dkv.norm"][None, :]
    rot = c.get("rot") or {"dims": 0, "base": 1.0}
    kr = rotate(down[:, None, R:], pos, rot["dims"], rot["base"])[:, 0]
    qr = rotate(q[:, :, d:], pos, rot["dims"], rot["base"])
    k = (lat @ W[p + "uk"].T).reshape(T, H, d)
    v = (lat @ W[p + "uv"].T).reshape(T, H, dv)
    see = visible(np.asarray(pos)[:, None], np.asarray(pos)[None, :], None)
    out = np.zeros((T, H, dv))
    for n in range(H):
        s = (q[:, n, :d] @ k[:, n].T + qr[:, n] @ kr.T) * c["scale"]
        out[:, n] = softmax_heads(s, see, W[p + "sink"][n]) @ v[:, n]
    return out.reshape(T, H * dv) @ W[p + "o"].T


def token_mix(h, mu, before=None):
    """h + (h' - h) mu with h' the previous token's h (zeros before the first one)."""
    prev = np.concatenate([np.zeros((1, h.shape[1])) if before is None else before[None, :], h[:-1]])
    return h + (prev - h) * mu[None, :]


def wkv_decay(W, p, mix_w):
    return np.exp(-np.exp(np.tanh(mix_w @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"][None, :]))


def wkv(cfg, c, W, p, h, pos):
    T = h.shape[0]
    H, d = c["heads"], c["dim"]
    mix = {s: token_mix(h, W[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = (mix[s] @ W[p + s].T for s in "rkv")
    w = wkv_decay(W, p, mix["w"])
    o, _ = wkv_recurrence(r.reshape(T, H, d), k.reshape(T, H, d), v.reshape(T, H, d), w.reshape(T, H, d), W[p + "u"])
    o = rms_unit(o, cfg["norm"]["eps"]).reshape(T, H * d)
    return (o * W[p + "norm"][None, :] * silu(mix["g"] @ W[p + "g"].T)) @ W[p + "o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "wkv": wkv}


def feed_forward(W, p, h):
    return xielu(h @ W[p + "up"].T, *W[p + "act"]) @ W[p + "down"].T


# ---------------------------------------------------------------------------------------------------------------- the model
def weights_layer(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, W, toks):
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    eps = cfg["norm"]["eps"]
    pos = np.arange(len(toks))
    x = zero_centred_norm(W["embed"][np.asarray(toks)], W["embed.norm"], eps)
    taps = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{weights_layer(cfg, i)}."
        x = x + MIXERS[layer["type"]](cfg, layer["mixer"], W, p + "mix.", zero_centred_norm(x, W[p + "norm1"], eps), pos)
        if layer.get("mlp"):
            x = x + feed_forward(W, p + "mlp.", zero_centred_norm(x, W[p + "norm2"], eps))
        taps.append(x.copy())
    return zero_centred_norm(x, W["final.norm"], eps) @ W["head"].T, np.stack(taps)


# ---------------------------------------------------------------------------------------------------------------- weights for tests
def tensor_shapes(cfg, rank=8):
    """name -> shape of every tensor of a configuration.  rank: inner size of the decay's low-rank map (a number, or one per layer)."""
    Wd, V = cfg["width"], cfg["vocab"]
    sh = {"embed": (V, Wd), "embed.norm": (Wd,), "head": (V, Wd), "final.norm": (Wd,)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, c, kind = f"l{i}.", layer["mixer"], layer["type"]
        a = p + "mix."
        sh[p + "norm1"] = (Wd,)
        H, d = c["heads"], c["dim"]
        if kind == "attention":
            G, dv = c.get("kv_heads", H), c.get("vdim", d)
            sh[a + "q"], sh[a + "k"], sh[a + "v"], sh[a + "o"] = (H * d, Wd), (G * d, Wd), (G * dv, Wd), (Wd, H * dv)
            sh[a + "q.norm"], sh[a + "k.norm"], sh[a + "temp"], sh[a + "g"] = (H * d,), (G * d,), (H,), (H, Wd)
        elif kind == "latent_attention":
            dr, dv, R = c["rot_dim"], c.get("vdim", d), c["kv_rank"]
            sh[a + "q"], sh[a + "dkv"], sh[a + "dkv.norm"] = (H * (d + dr), Wd), (R + dr, Wd), (R,)
            sh[a + "uk"], sh[a + "uv"], sh[a + "sink"], sh[a + "o"] = (H * d, R), (H * dv, R), (H,), (Wd, H * dv)
        else:
            k = rank[i] if isinstance(rank, (list, tuple, dict)) else rank
            for s in "rkvgw":
                sh[a + "mu." + s] = (Wd,)
            for s in "rkvg":
                sh[a + s] = (H * d, Wd)
            sh[a + "w1"], sh[a + "w2"], sh[a + "w0"] = (k, Wd), (H * d, k), (H * d,)
            sh[a + "u"], sh[a + "norm"], sh[a + "o"] = (H, d), (H * d,), (Wd, H * d)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            sh[p + "norm2"], sh[p + "mlp.up"], sh[p + "mlp.down"], sh[p + "mlp.act"] = (Wd,), (ff, Wd), (Wd, ff), (2,)
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
            a = rng.normal(0, 1.0, shape)
        elif leaf in ("norm1", "norm2") or name in ("embed.norm", "final.norm"):
            a = rng.uniform(-0.4, 0.4, shape)
        elif leaf == "norm":
            a = rng.uniform(0.6, 1.5, shape)
        elif ".mu." in name:
            a = rng.uniform(0.0, 1.0, shape)
        elif leaf == "temp":
            a = rng.uniform(0.5, 2.0, shape)
        elif leaf == "sink":
            a = rng.normal(0, 1.5, shape)
        elif leaf == "act":
            a = rng.uniform(-1.0, 1.0, shape)
        elif leaf == "w0":
            a = rng.uniform(-5.0, 0.5, shape)
        elif leaf == "u":
            a = rng.normal(0, 0.7, shape)
        else:
            a = rng.normal(0, (gain if name == "head" else 1.0) / np.sqrt(shape[-1]), shape)
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
