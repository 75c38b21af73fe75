"""Plain NumPy statement of the mixer-built decoders (the Sizilorn, Kunonex, Tevanex and Mamivik designs and their parts), test infrastructure only.

One function per mechanism, whole sequences at once, float64 unless the caller passes other arrays; recurrences are written
token by token.  Nothing here is shared with the CUDA path.  Shapes: x, h [T, width]; a head-wise array [T, heads, dim].
"""
from __future__ import annotations

import numpy as np


# ------------------------------------------------------------------------------------------------ elementwise

def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


# ------------------------------------------------------------------------------------------------ norms

def rms(x, eps):
    """Division by the root mean square over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dyn_tanh(x, alpha, w, b):
    return np.tanh(alpha * x) * w + b


def layer_norm(x, w, eps):
    """Mean taken off, divided by the standard deviation (eps inside the root), times w."""
    c = x - np.mean(x, axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * w


# ------------------------------------------------------------------------------------------------ absolute positions

def sinusoid(positions, width):
    """[positions, width]: sine in the even columns and cosine in the odd ones, column pair i turning at 10000^(-2i / width)."""
    out = np.zeros((len(positions), width))
    for c in range(width):
        a = np.asarray(positions, np.float64) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = np.cos(a) if c % 2 else np.sin(a)
    return out


# ------------------------------------------------------------------------------------------------ rotation

def rope_frequencies(dims, base, scaling=None):
    """One frequency per pair; `scaling` = dict(factor, low, high, original) stretches the long wavelengths."""
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    if not scaling:
        return f
    out = []
    for fi in f:
        wavelength = 2.0 * np.pi / fi
        turns = scaling["original"] / wavelength
        if turns > scaling["high"]:
            out.append(fi)
        elif turns < scaling["low"]:
            out.append(fi / scaling["factor"])
        else:
            s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
            out.append((1.0 - s) * fi / scaling["factor"] + s * fi)
    return np.array(out)


def rotate_interleaved(x, positions, dims, freqs):
    """x [T, heads, dim]: the pairs (2i, 2i + 1) of the first `dims` dimensions turn by position * freqs[i]."""
    a = np.asarray(positions, np.float64)[:, None] * freqs[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def yarn_frequencies(dims, base, factor, original, fast, slow):
    """Frequencies stretched by `factor` where a pair turns less than `slow` times over the original context, kept where it
    turns more than `fast` times, blended linearly in between; and the factor of cosine and sine."""
    f = base ** (-2.0 * np.arange(dims // 2) / dims)

    def pair_that_turns(t):
        return dims * np.log(original / (2.0 * np.pi * t)) / (2.0 * np.log(base))

    lo, hi = max(np.floor(pair_that_turns(fast)), 0.0), min(np.ceil(pair_that_turns(slow)), dims - 1.0)
    stretched = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * stretched + f * (1.0 - stretched), 0.1 * np.log(factor) + 1.0


def rotate_half(x, positions, dims, freqs):
    """x [T, heads, dim]: the pairs (i, i + dims / 2) of the first `dims` dimensions turn by position * freqs[i]."""
    a = np.asarray(positions, np.float64)[:, None] * freqs[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    out, n = x.copy(), dims // 2
    u, v = x[..., :n], x[..., n:dims]
    out[..., :n] = u * c - v * s
    out[..., n:dims] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------ attention

def causal_attention(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e]; query head h reads key/value head h // (H // G)."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    mask = np.tril(np.ones((T, T), bool))
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T) * scale
        s = np.where(mask, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // group]
    return out


def gated_attention(h, W, cfg, eps):
    """Grouped-query attention with per-head query/key norms, interleaved rotation and a per-head output gate."""
    T = h.shape[0]
    H, G, d, e = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = rms((h @ W["q"].T).reshape(T, H, d), eps) * W["q.norm"]
    k = rms((h @ W["k"].T).reshape(T, G, d), eps) * W["k.norm"]
    v = (h @ W["v"].T).reshape(T, G, e)
    rot = cfg.get("rot")
    if rot:
        f = rope_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        pos = np.arange(T)
        q, k = rotate_interleaved(q, pos, rot["dims"], f), rotate_interleaved(k, pos, rot["dims"], f)
    o = causal_attention(q, k, v, cfg["scale"])
    o = o * sigmoid(h @ W["g"].T)[:, :, None]
    return o.reshape(T, H * e) @ W["o"].T


def chunked_attention(q, k, v, scale, chunk, softcap=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, e]; a position sees the keys of its own chunk up to itself.  softcap: scores pass
    through softcap * tanh(. / softcap); sink [H]: one more term exp(sink) in every denominator."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        for t in range(T):
            lo = t // chunk * chunk
            s = k[lo:t + 1, h // group] @ q[t, h] * scale
            if softcap is not None:
                s = softcap * np.tanh(s / softcap)
            top = s.max() if sink is None else max(s.max(), sink[h])
            p = np.exp(s - top)
            den = p.sum() + (0.0 if sink is None else np.exp(sink[h] - top))
            out[t, h] = p @ v[lo:t + 1, h // group] / den
    return out


def projected_heads(h, W, cfg, eps):
    """q, k, v with biases; the RMS norm of q and k runs over all heads at once."""
    T = h.shape[0]
    q = rms(h @ W["q"].T + W["q.b"], eps) * W["q.norm"]
    k = rms(h @ W["k"].T + W["k.b"], eps) * W["k.norm"]
    v = h @ W["v"].T + W["v.b"]
    return q.reshape(T, cfg["heads"], cfg["dim"]), k.reshape(T, cfg["kv_heads"], cfg["dim"]), v.reshape(T, cfg["kv_heads"], cfg["vdim"])


def sink_attention(h, W, cfg, eps):
    """Chunked attention with a sink per head and half-split rotation."""
    q, k, v = projected_heads(h, W, cfg, eps)
    rot, pos = cfg["rot"], np.arange(h.shape[0])
    f = rope_frequencies(rot["dims"], rot["base"])
    q, k = rotate_half(q, pos, rot["dims"], f), rotate_half(k, pos, rot["dims"], f)
    o = chunked_attention(q, k, v, cfg["scale"], cfg["mask"]["size"], sink=W["sink"])
    return o.reshape(len(pos), -1) @ W["o"].T + W["o.b"]


def capped_attention(h, W, cfg, eps):
    """Chunked attention with capped scores, adjacent-pair rotation stretched to a longer context, and an element-wise gate."""
    q, k, v = projected_heads(h, W, cfg, eps)
    rot, pos = cfg["rot"], np.arange(h.shape[0])
    f, m = yarn_frequencies(rot["dims"], rot["base"], **rot["scaling"])

    def turn(x):
        r = rotate_interleaved(x, pos, rot["dims"], f)
        r[..., :rot["dims"]] *= m
        return r

    o = chunked_attention(turn(q), turn(k), v, cfg["scale"], cfg["mask"]["size"], softcap=cfg["softcap"])
    return (o.reshape(len(pos), -1) * sigmoid(h @ W["g"].T)) @ W["o"].T + W["o.b"]


def latent_attention(h, W, cfg, eps):
    """Attention whose keys and values are projections of one small vector per token; no positions; a gate per head."""
    T, H = h.shape[0], cfg["heads"]
    q = (rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T
    c = rms(h @ W["dkv"].T, eps) * W["dkv.norm"]
    k, v = c @ W["uk"].T, c @ W["uv"].T
    o = causal_attention(q.reshape(T, H, cfg["dim"]), k.reshape(T, H, cfg["dim"]), v.reshape(T, H, cfg["vdim"]), cfg["scale"])
    o = o * sigmoid(h @ W["g"].T)[:, :, None]
    return o.reshape(T, H * cfg["vdim"]) @ W["o"].T


def windowed_attention(q, k, v, scale, window, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, e]; a position sees itself and the window - 1 keys before it.  sink [H]: one more term
    exp(sink) in every denominator."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        for t in range(T):
            lo = max(0, t - window + 1)
            s = k[lo:t + 1, h // group] @ q[t, h] * scale
            top = s.max() if sink is None else max(s.max(), sink[h])
            p = np.exp(s - top)
            den = p.sum() + (0.0 if sink is None else np.exp(sink[h] - top))
            out[t, h] = p @ v[lo:t + 1, h // group] / den
    return out


def shared_kv_attention(h, W, cfg):
    """Windowed grouped-query attention whose values are the keys before their rotation; biases on queries and keys."""
    T, rot = h.shape[0], cfg["rot"]
    q = (h @ W["q"].T + W["q.b"]).reshape(T, cfg["heads"], cfg["dim"])
    k = (h @ W["k"].T + W["k.b"]).reshape(T, cfg["kv_heads"], cfg["dim"])
    f = rope_frequencies(rot["dims"], rot["base"])

    def turn(x):
        return rotate_half(x, np.arange(T), rot["dims"], f)

    o = windowed_attention(turn(q), turn(k), k, cfg["scale"], cfg["mask"]["size"])
    return o.reshape(T, -1) @ W["o"].T


def rotated_latent_attention(h, W, cfg, eps):
    """Windowed latent attention with a second, rotated key part that all heads share, a sink per head and a gate per value."""
    T, H, d, r, rank = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["kv_rank"]
    q = ((rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T).reshape(T, H, d + r)
    down = h @ W["dkv"].T
    c, turned = rms(down[:, :rank], eps) * W["dkv.norm"], down[:, None, rank:]
    f, m = yarn_frequencies(r, cfg["rot"]["base"], **cfg["rot"]["scaling"]) if cfg["rot"].get("scaling") else (rope_frequencies(r, cfg["rot"]["base"]), 1.0)

    def turn(x):
        return m * rotate_half(x, np.arange(T), r, f)

    k = np.concatenate([(c @ W["uk"].T).reshape(T, H, d), np.repeat(turn(turned), H, axis=1)], axis=2)
    q = np.concatenate([q[..., :d], turn(q[..., d:])], axis=2)
    o = windowed_attention(q, k, (c @ W["uv"].T).reshape(T, H, cfg["vdim"]), cfg["scale"], cfg["mask"]["size"], W["sink"])
    return (o.reshape(T, -1) * sigmoid(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ gated delta rule

def causal_conv(x, taps):
    """Depthwise convolution over time, x [T, C], taps [C, K], last tap = the current token, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, x.shape[1]), x.dtype), x])
    return sum(padded[j:j + T] * taps[:, j] for j in range(K))


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_decay(alpha, a_log, dt_bias):
    return np.exp(-np.exp(a_log) * softplus(alpha + dt_bias))


def delta_rule(q, k, v, g, beta, state=None):
    """q, k [T, G, d], v [T, H, e], g, beta [T, H]; head h reads q/k head h // (H // G).  Returns (o [T, H, e], state)."""
    T, H, e = v.shape
    group = H // q.shape[1]
    S = np.zeros((H, q.shape[2], e), v.dtype) if state is None else state.copy()
    o = np.empty_like(v)
    for t in range(T):
        qt, kt = np.repeat(q[t], group, axis=0), np.repeat(k[t], group, axis=0)
        S *= g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hde,hd->he", S, kt))
        S += kt[:, :, None] * u[:, None, :]
        o[t] = np.einsum("hde,hd->he", S, qt)
    return o, S


def gated_delta(h, W, cfg, eps):
    T = h.shape[0]
    H, G, d, e = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = silu(causal_conv(h @ W["q"].T, W["q.conv"])).reshape(T, G, d)
    k = silu(causal_conv(h @ W["k"].T, W["k.conv"])).reshape(T, G, d)
    v = silu(causal_conv(h @ W["v"].T, W["v.conv"])).reshape(T, H, e)
    q, k = unit(q) / np.sqrt(d), unit(k)
    beta = sigmoid(h @ W["b"].T)
    g = delta_decay(h @ W["a"].T, W["A_log"], W["dt_bias"])
    o, _ = delta_rule(q, k, v, g, beta)
    o = rms(o, eps) * W["norm"] * silu(h @ W["g"].T).reshape(T, H, e)
    return o.reshape(T, H * e) @ W["o"].T


def parallel_mixer(h, W, cfg, eps):
    """Half the sum of the two branches' RMS-normed outputs."""
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    left = gated_attention(h, sub("left."), cfg["left"], eps)
    right = gated_delta(h, sub("right."), cfg["right"], eps)
    return 0.5 * (rms(left, eps) * W["left.out"] + rms(right, eps) * W["right.out"])


# ------------------------------------------------------------------------------------------------ delta rule with channel gates

def bounded_decay(h, w1, w2, w0):
    """A decay per channel between exp(-exp(-1/2)) and 1."""
    return np.exp(-np.exp(-0.5) * sigmoid(np.tanh(h @ w1.T) @ w2.T + w0))


def channel_delta_rule(r, k, v, w, a, state=None):
    """r, k, v, w, a [T, H, d]: decay w and removal rate a per key channel; the removal reads along the unit key, the write takes
    the key as it is, and both see the old state.  Returns (o [T, H, d], state)."""
    T, H, d = k.shape
    S = np.zeros((H, d, v.shape[2]), k.dtype) if state is None else state.copy()
    o = np.empty_like(v)
    for t in range(T):
        u = unit(k[t])
        seen = np.einsum("hkv,hk->hv", S, u)
        S = w[t][:, :, None] * S - (a[t] * u)[:, :, None] * seen[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, r[t])
    return o, S


def channel_delta_mixer(h, W, cfg, eps):
    T = h.shape[0]
    H, d = cfg["heads"], cfg["dim"]
    r, k, v = ((h @ W[s].T).reshape(T, H, d) for s in "rkv")
    w = bounded_decay(h, W["w1"], W["w2"], W["w0"]).reshape(T, H, d)
    a = sigmoid(h @ W["a"].T + W["a.b"]).reshape(T, H, d)
    o, _ = channel_delta_rule(r, k, v, w, a)
    return (rms(o, eps).reshape(T, H * d) * W["norm"] * sigmoid(h @ W["g"].T)) @ W["o"].T


def scaled_parallel_mixer(h, W, cfg, eps):
    """Two branches over one input, each times its own constant."""
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    return cfg["left_scale"] * shared_kv_attention(h, sub("left."), cfg["left"]) + cfg["right_scale"] * channel_delta_mixer(h, sub("right."), cfg["right"], eps)


# ------------------------------------------------------------------------------------------------ WKV time mixing

def token_shift(h, mu):
    prev = np.concatenate([np.zeros((1, h.shape[1]), h.dtype), h[:-1]])
    return h + (prev - h) * mu


def wkv_decay(mix_w, w1, w2, w0):
    return np.exp(-np.exp(np.tanh(mix_w @ w1.T) @ w2.T + w0))


def wkv_rule(r, k, v, w, u, state=None):
    """r, k, v, w [T, H, d], u [H, d].  Returns (o [T, H, d], state)."""
    T, H, d = r.shape
    S = np.zeros((H, d, d), r.dtype) if state is None else state.copy()
    o = np.empty_like(r)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return o, S


def wkv_mixer(h, W, cfg, eps):
    T = h.shape[0]
    H, d = cfg["heads"], cfg["dim"]
    mix = {s: token_shift(h, W["mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[s].T).reshape(T, H, d) for s in "rkv")
    w = wkv_decay(mix["w"], W["w1"], W["w2"], W["w0"]).reshape(T, H, d)
    o, _ = wkv_rule(r, k, v, w, W["u"])
    return (rms(o, eps).reshape(T, H * d) * W["norm"] * silu(mix["g"] @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ mLSTM

def mlstm_gates(zi, zf, cap):
    """Log input gate and log forget gate from their projections (biases included)."""
    return cap * np.tanh(zi / cap), -softplus(-cap * np.tanh(zf / cap))


def mlstm_rule(q, k, v, i, f, state=None):
    """q, k [T, H, d], v [T, H, e], i, f [T, H].  State (S [H, d, e], n [H, d], m [H]) is kept times exp(-m), m the running
    maximum of the logarithms, 0 at the start.  Returns (o [T, H, e], state)."""
    T, H, d = k.shape
    S, n, m = (np.zeros((H, d, v.shape[2]), v.dtype), np.zeros((H, d), v.dtype), np.zeros(H, v.dtype)) if state is None else [a.copy() for a in state]
    o = np.empty_like(v)
    for t in range(T):
        top = np.maximum(f[t] + m, i[t])
        keep, write = np.exp(f[t] + m - top), np.exp(i[t] - top)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = top
        den = np.maximum(np.abs(np.einsum("hd,hd->h", n, q[t])), np.exp(-m)) + 1e-6
        o[t] = np.einsum("hde,hd->he", S, q[t]) / den[:, None]
    return o, (S, n, m)


def mlstm_mixer(h, W, cfg, eps):
    T = h.shape[0]
    H, d, e = cfg["heads"], cfg["dim"], cfg["vdim"]
    q, k = (h @ W["q"].T).reshape(T, H, d) / np.sqrt(d), (h @ W["k"].T).reshape(T, H, d)
    i, f = mlstm_gates(h @ W["i"].T + W["i.b"], h @ W["f"].T + W["f.b"], cfg["gate_cap"])
    o, _ = mlstm_rule(q, k, (h @ W["v"].T).reshape(T, H, e), i, f)
    return (rms(o, eps).reshape(T, H * e) * W["norm"] * sigmoid(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ minGRU

def min_gru(z, u, state=None):
    """z (gate, in 0..1) and u (candidate before its activation), [T, n].  Returns (S [T, n], last S)."""
    S = np.zeros(z.shape[1], z.dtype) if state is None else state.copy()
    out = np.empty_like(z)
    for t in range(z.shape[0]):
        cand = np.where(u[t] >= 0, u[t] + 0.5, sigmoid(u[t]))
        S = (1.0 - z[t]) * S + z[t] * cand
        out[t] = S
    return out, S


def mingru_mixer(h, W, cfg, eps):
    S, _ = min_gru(sigmoid(h @ W["z"].T + W["z.b"]), h @ W["x"].T + W["x.b"])
    return (S * silu(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ feed-forward, token input

def poly_norm(z, act, eps):
    """A cubic of z whose powers are each divided by their own root mean square first."""
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def poly_mlp(h, W, eps):
    return poly_norm(h @ W["up"].T + W["up.b"], W["act"], eps) @ W["down"].T + W["down.b"]


def gated_mlp(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def gelu_mlp(h, W):
    return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def clamped_mlp(h, W, limit):
    """Gate and up rows held within a limit, the gate through z * sigmoid(1.702 z), the up rows plus one."""
    g = np.minimum(h @ W["gate"].T, limit)
    u = np.clip(h @ W["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W["down"].T


def routed(h, W, top):
    """Chosen experts and their weights [T, top]: the largest sigmoid scores, as they are."""
    s = sigmoid(h @ W["router"].T)
    chosen = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def moe_mlp(h, W, cfg):
    """Every chosen expert reads its weight times the row; a shared expert with a gate per token runs beside them."""
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    chosen, weight = routed(h, W, cfg["router"]["top"])
    out = np.zeros_like(h)
    if cfg.get("shared"):
        out = sigmoid(h @ W["shared.sg"].T) * clamped_mlp(h, sub("shared."), cfg["shared"]["limit"])
    for e in range(cfg["router"]["experts"]):
        t, j = np.nonzero(chosen == e)
        if len(t):
            out[t] += clamped_mlp(weight[t, j][:, None] * h[t], sub(f"e{e}."), cfg["expert"]["limit"])
    return out


def token_side(x, e, W, eps):
    """The per-layer token input: e [T, dim] is the layer's slice of the side embedding."""
    y = (gelu_tanh(x @ W["gate"].T) * e) @ W["proj"].T
    return x + rms(y, eps) * W["norm"]


# ------------------------------------------------------------------------------------------------ the decoder

class MixerDecoder:
    """config: the parsed config.json; tensors: name -> array."""

    def __init__(self, config, tensors, dtype=np.float64):
        self.cfg = config
        self.w = {k: np.asarray(v, dtype) for k, v in tensors.items()}

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def _norm(self, name, x):
        return dyn_tanh(x, self.w[name + ".alpha"], self.w[name], self.w[name + ".b"])

    def embedding_output(self, tokens):
        return self.w["embed"][tokens]

    def residuals(self, tokens):
        """The residual stream after every layer: [layers, T, width]."""
        tokens = np.asarray(tokens)
        eps = self.cfg["norm"]["eps"]
        side = self.cfg.get("token_side")
        x = self.embedding_output(tokens)
        out = []
        for i, layer in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            mixer = {"wkv": wkv_mixer, "parallel": parallel_mixer}[layer["type"]]
            x = x + mixer(self._norm(p + "norm1", x), self._sub(p + "mix."), layer["mixer"], eps)
            if layer.get("mlp"):
                x = x + gated_mlp(self._norm(p + "norm2", x), self._sub(p + "mlp."))
            if side:
                e = self.w["side.embed"][tokens][:, i * side["dim"]:(i + 1) * side["dim"]]
                x = token_side(x, e, self._sub(p + "side."), eps)
            out.append(x)
        return np.stack(out)

    def logits(self, tokens):
        return self._norm("final.norm", self.residuals(tokens)[-1]) @ self.w["head"].T


class KunonexDecoder(MixerDecoder):
    """Sinusoidal positions, layers whose mixer and feed-forward read one layer norm side by side, a token shift in front of
    every mixer, and a run of layers that is passed through several times."""

    def _norm(self, name, x):
        return layer_norm(x, self.w[name], self.cfg["norm"]["eps"])

    def schedule(self):
        """(layer, pass) in the order of execution; pass is None outside of the loop."""
        n, loop = len(self.cfg["layers"]), self.cfg.get("loop")
        if not loop:
            return [(i, None) for i in range(n)]
        a, b = loop["start"], loop["stop"]
        return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)] + [(i, None) for i in range(b, n)])

    def embedding_output(self, tokens):
        return self._norm("embed.norm", self.w["embed"][tokens] + sinusoid(np.arange(len(tokens)), self.cfg["width"]))

    def residuals(self, tokens):
        """The residual stream after every layer run: [layer runs, T, width]."""
        eps = self.cfg["norm"]["eps"]
        x0 = x = self.embedding_output(np.asarray(tokens))
        out = []
        for i, t in self.schedule():
            if t is not None and i == self.cfg["loop"]["start"]:
                x = np.concatenate([x, x0], axis=1) @ self.w["loop.in"].T + self.w["loop.step"][t]
            p, layer = f"l{i}.", self.cfg["layers"][i]
            h = self._norm(p + "norm1", x)
            mixer = {"mingru": mingru_mixer, "latent_attention": latent_attention}[layer["type"]]
            y = mixer(token_shift(h, self.w[p + "shift"]), self._sub(p + "mix."), layer["mixer"], eps)
            if layer.get("mlp"):
                y = y + poly_mlp(h, self._sub(p + "mlp."), eps)
            x = x + y
            out.append(x)
        return np.stack(out)

    def logits(self, tokens):
        return super().logits(tokens) * self.cfg["logit_scale"]


class TevanexDecoder(MixerDecoder):
    """mLSTM layers and two kinds of chunked attention over a mixture of experts; norms on what a sublayer gives, not on what it
    reads; layers that run another one's tensors again."""

    def _norm(self, name, x):
        return rms(x, self.cfg["norm"]["eps"]) * self.w[name]

    def embedding_output(self, tokens):
        return self.w["embed"][tokens] * self.cfg["embedding"]["scale"]

    def residuals(self, tokens):
        """The residual stream after every layer: [layers, T, width]."""
        eps, m = self.cfg["norm"]["eps"], self.cfg["residual_mult"]
        x = self.embedding_output(np.asarray(tokens))
        out = []
        for i, layer in enumerate(self.cfg["layers"]):
            while self.cfg["layers"][i].get("weights_of") is not None:
                i = self.cfg["layers"][i]["weights_of"]
            p = f"l{i}."
            mixer = {"mlstm": mlstm_mixer, "attention": sink_attention, "attention_2": capped_attention}[layer["type"]]
            x = x + m * self._norm(p + "norm1", mixer(x, self._sub(p + "mix."), layer["mixer"], eps))
            if layer.get("mlp"):
                x = x + m * self._norm(p + "norm2", moe_mlp(x, self._sub(p + "mlp."), layer["mlp"]))
            out.append(x)
        return np.stack(out)

    def logits(self, tokens):
        cap = self.cfg["logit_softcap"]
        return cap * np.tanh(super().logits(tokens) * self.cfg["logit_scale"] / cap)


class MamivikDecoder(MixerDecoder):
    """RMS norms with one number each; a short convolution in front of every mixer; windowed attention beside a delta rule with a
    decay and a removal rate per channel, and windowed latent attention with a rotated part."""

    def _norm(self, name, x):
        return rms(x, self.cfg["norm"]["eps"]) * self.w[name]

    def residuals(self, tokens):
        """The residual stream after every layer: [layers, T, width]."""
        eps = self.cfg["norm"]["eps"]
        x = self.embedding_output(np.asarray(tokens))
        out = []
        for i, layer in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            h = self._norm(p + "norm1", x)
            h = h + causal_conv(h, self.w[p + "canon1"])
            mixer = {"parallel": scaled_parallel_mixer, "latent_attention": rotated_latent_attention}[layer["type"]]
            x = x + mixer(h, self._sub(p + "mix."), layer["mixer"], eps)
            if layer.get("mlp"):
                x = x + gelu_mlp(self._norm(p + "norm2", x), self._sub(p + "mlp."))
            out.append(x)
        return np.stack(out)


def decoder(config, tensors, dtype=np.float64):
    return {"Sizilorn": MixerDecoder, "Kunonex": KunonexDecoder, "Tevanex": TevanexDecoder, "Mamivik": MamivikDecoder}[config["architecture"]](config, tensors, dtype)


def read_safetensors(path):
    """name -> float32 / int32 array (bfloat16 widened)."""
    import json
    import struct
    raw = open(path, "rb").read()
    (n,) = struct.unpack("<Q", raw[:8])
    head = json.loads(raw[8:8 + n])
    out = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        b = raw[8 + n + lo:8 + n + hi]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(b, np.uint16).astype(np.uint32) << 16).view(np.float32)
        else:
            a = np.frombuffer(b, {"F32": np.float32, "F16": np.float16, "I32": np.int32}[t["dtype"]])
        out[name] = a.reshape(t["shape"])
    return out


def write_safetensors(path, tensors):
    """Writes float arrays as bfloat16 (rounded to nearest even) and int32 arrays as they are."""
    import json
    import struct
    head, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.asarray(a)
        if a.dtype == np.int32:
            b, kind = a.tobytes(), "I32"
        else:
            b, kind = to_bf16_bits(a).tobytes(), "BF16"
        head[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    j = json.dumps(head).encode()
    j += b" " * (-len(j) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(j)) + j + b"".join(blobs))


def to_bf16_bits(a):
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16(a):
    """The nearest bfloat16 values, as float32."""
    return (to_bf16_bits(a).astype(np.uint32) << 16).view(np.float32).reshape(np.shape(a))
