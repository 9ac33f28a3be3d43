"""Plain restatement, in numpy and double precision, of models whose layers are listed one by one. Pabovik: latent
attention, lightning attention and RWKV-style time mixing between sandwich norms. Nozurax: retention and grouped-query
attention with a sink, in parallel with the feed-forward behind one norm. One function per
mechanism, whole sequences at a time, no cache and no chunks. Test infrastructure only: nothing of the product
path is imported, and nothing of this file is used by it.

`W` is a dict name -> float array, `p` a layer's prefix such as "l3.".
"""
import numpy as np


def rms_norm(x, w, eps):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotate_interleaved(x, positions, dims, base):
    """x [T, ..., D]: the pairs (2i, 2i + 1) of the first `dims` entries turn by position * base^(-2i / dims)."""
    out = np.array(x, dtype=np.float64)
    for i in range(dims // 2):
        a = np.asarray(positions, dtype=np.float64) * float(base) ** (-2.0 * i / dims)
        a = a.reshape((-1,) + (1,) * (x.ndim - 2))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def rotate_half(x, positions, dims, base):
    """x [T, ..., D]: the pairs (i, i + dims / 2) of the first `dims` entries turn by position * base^(-2i / dims)."""
    out = np.array(x, dtype=np.float64)
    half = dims // 2
    for i in range(half):
        a = np.asarray(positions, dtype=np.float64) * float(base) ** (-2.0 * i / dims)
        a = a.reshape((-1,) + (1,) * (x.ndim - 2))
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * np.cos(a) - v * np.sin(a)
        out[..., i + half] = v * np.cos(a) + u * np.sin(a)
    return out


def causal_softmax_attention(q, k, v, scale, sink=None):
    """q, k [T, H, D], v [T, H, Dv] -> [T, H, Dv]. sink [H]: one more term exp(sink) of the denominator, without a value."""
    T = q.shape[0]
    s = np.einsum("thd,shd->hts", q, k) * scale
    s = np.where(np.tril(np.ones((T, T), dtype=bool))[None], s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, np.asarray(sink)[:, None, None])
    e = np.exp(s - top)
    total = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(np.asarray(sink)[:, None, None] - top)
    return np.einsum("hts,shd->thd", e / total, v)


def latent_attention(h, W, p, c, eps):
    T, H = h.shape[0], c["heads"]
    dim, rd, vd, rank = c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    pos = np.arange(T)
    q = rms_norm(h @ W[p + "mix.dq"].T, W[p + "mix.dq.norm"], eps) @ W[p + "mix.uq"].T
    q = q.reshape(T, H, dim + rd)
    kv = h @ W[p + "mix.dkv"].T
    lat = rms_norm(kv[:, :rank], W[p + "mix.dkv.norm"], eps)
    rot = c["rot"]
    k_rot = rotate_interleaved(kv[:, rank:], pos, rot["dims"], rot["base"])
    q_rot = rotate_interleaved(q[..., dim:], pos, rot["dims"], rot["base"])
    k = np.concatenate([(lat @ W[p + "mix.uk"].T).reshape(T, H, dim), np.repeat(k_rot[:, None], H, axis=1)], axis=-1)
    v = (lat @ W[p + "mix.uv"].T).reshape(T, H, vd)
    o = causal_softmax_attention(np.concatenate([q[..., :dim], q_rot], axis=-1), k, v, c["scale"])
    return (o.reshape(T, H * vd) * sigmoid(h @ W[p + "mix.g"].T)) @ W[p + "mix.o"].T


def lightning_scan(q, k, v, decay):
    """q, k [T, H, D], v [T, H, Dv], decay [H]: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]))
    out = np.empty((T, H, v.shape[2]))
    for t in range(T):
        S = S * np.asarray(decay)[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def lightning(h, W, p, c, eps):
    T, H = h.shape[0], c["heads"]
    q = silu(h @ W[p + "mix.q"].T).reshape(T, H, c["dim"])
    k = silu(h @ W[p + "mix.k"].T).reshape(T, H, c["dim"])
    v = silu(h @ W[p + "mix.v"].T).reshape(T, H, c["vdim"])
    o = lightning_scan(q, k, v, c["decay"]).reshape(T, H * c["vdim"])
    o = rms_norm(o, W[p + "mix.norm"], eps) * sigmoid(h @ W[p + "mix.g"].T)
    return o @ W[p + "mix.o"].T


def wkv_scan(r, k, v, w, u):
    """r, k, v, w [T, H, D], u [H, D]: the current token enters with the bonus u, the state afterwards without."""
    T, H, D = r.shape
    S = np.zeros((H, D, D))
    out = np.empty((T, H, D))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = S * w[t][:, :, None] + kv
    return out


def token_shift_mix(h, mu):
    prev = np.concatenate([np.zeros_like(h[:1]), h[:-1]], axis=0)
    return h + (prev - h) * mu


def wkv_decay(mix_w, W, p):
    return np.exp(-np.exp(np.tanh(mix_w @ W[p + "mix.w1"].T) @ W[p + "mix.w2"].T + W[p + "mix.w0"]))


def wkv(h, W, p, c, eps):
    T, H, D = h.shape[0], c["heads"], c["dim"]
    mix = {s: token_shift_mix(h, W[p + "mix.mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[p + "mix." + s].T).reshape(T, H, D) for s in "rkv")
    w = wkv_decay(mix["w"], W, p).reshape(T, H, D)
    o = wkv_scan(r, k, v, w, W[p + "mix.u"].reshape(H, D))
    o = rms_norm(o, None, eps).reshape(T, H * D) * W[p + "mix.norm"] * silu(mix["g"] @ W[p + "mix.g"].T)
    return o @ W[p + "mix.o"].T


def retention(h, W, p, c, eps):
    """Linear attention with a fixed decay per head, rotated queries and keys, every head's output normed and gated."""
    T, H, D = h.shape[0], c["heads"], c["dim"]
    pos, rot = np.arange(T), c["rot"]
    q = rotate_half((h @ W[p + "mix.q"].T).reshape(T, H, D), pos, rot["dims"], rot["base"])
    k = rotate_half((h @ W[p + "mix.k"].T).reshape(T, H, D), pos, rot["dims"], rot["base"]) * D ** -0.5
    v = (h @ W[p + "mix.v"].T).reshape(T, H, c["vdim"])
    o = rms_norm(lightning_scan(q, k, v, c["decay"]), None, eps).reshape(T, H * c["vdim"])
    return (o * silu(h @ W[p + "mix.g"].T)) @ W[p + "mix.o"].T


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions) + 1) / every) + 1.0)


def sink_attention(h, W, p, c, eps):
    """Grouped-query attention without rotation: biases, q and k normed over all their heads at once, queries scaled with
    the logarithm of the position, a learned sink per head in the denominator."""
    T, H, G, D = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q = rms_norm(h @ W[p + "mix.q"].T + W[p + "mix.q.b"], W[p + "mix.q.norm"], eps).reshape(T, H, D)
    k = rms_norm(h @ W[p + "mix.k"].T + W[p + "mix.k.b"], W[p + "mix.k.norm"], eps).reshape(T, G, D)
    v = (h @ W[p + "mix.v"].T + W[p + "mix.v.b"]).reshape(T, G, c["vdim"])
    q = q * query_temperature(np.arange(T), c["q_temp"]["coef"], c["q_temp"]["every"])[:, None, None]
    shared = np.arange(H) // (H // G)
    o = causal_softmax_attention(q, k[:, shared], v[:, shared], c["scale"], W[p + "mix.sink"])
    return o.reshape(T, H * c["vdim"]) @ W[p + "mix.o"].T


def relu(z):
    return np.maximum(z, 0.0)


def dense_ff(h, W, p, act=silu):
    return (act(h @ W[p + "mlp.gate"].T) * (h @ W[p + "mlp.up"].T)) @ W[p + "mlp.down"].T


MIXERS = {"latent_attention": latent_attention, "lightning": lightning, "wkv": wkv, "retention": retention,
          "attention": sink_attention}


def weights_layer(layers, i):
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def sandwich_layer(x, layer, W, p, eps):
    y = MIXERS[layer["type"]](rms_norm(x, W[p + "norm1"], eps), W, p, layer["mixer"], eps)
    x = x + rms_norm(y, W[p + "norm1b"], eps)
    if layer.get("mlp"):
        y = dense_ff(rms_norm(x, W[p + "norm2"], eps), W, p)
        x = x + rms_norm(y, W[p + "norm2b"], eps)
    return x


def parallel_layer(x, layer, W, p, eps):
    """One norm, its weight stored around zero; mixer and feed-forward read the same input."""
    h = rms_norm(x, 1.0 + W[p + "norm1"], eps)
    y = MIXERS[layer["type"]](h, W, p, layer["mixer"], eps)
    return x + (y + dense_ff(h, W, p, relu) if layer.get("mlp") else y)


def forward(cfg, W, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in W.items()}
    eps = cfg["norm"]["eps"]
    parallel = cfg["architecture"] == "Nozurax"
    x = W["embed"][np.asarray(tokens)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{weights_layer(cfg['layers'], i)}."
        x = (parallel_layer if parallel else sandwich_layer)(x, layer, W, p, eps)
        after.append(x)
    final = 1.0 + W["final.norm"] if parallel else W["final.norm"]
    return rms_norm(x, final, eps) @ W["head"].T, np.stack(after)
