"""Plain, slow restatement of the Getizen decoder, used only as a test oracle.

Whole sequences, no cache, one function per mechanism, float64 throughout, no code shared with the product
package.  Notation: h is a sublayer's input [T, width]; p the positions 0..T-1; a weight matrix is [out, in] and
acts as h @ W.T; cfg is the config.json object, W a dict name -> array.

  embedding      x = gn(E[tok])
  norm           gn(x): every one of `groups` equal parts of x over its own rms, then all of it times w
  layer          x <- gn1(alpha x + mixer(x));  x <- gn2(alpha x + ff(x))
  parallel       (rms(left(h)) * wl + rms(right(h)) * wr) / 2
    left         q, k <- rms over the whole projection * gain;  the first n dimensions of every head turned in pairs
                 (i, i + n/2) by p * f_i (f rescaled by wavelength);  score q . k * scale * temp_head;  p sees t <= p of
                 the same chunk floor(p / size);  softmax;  times sigmoid(Wg h) per element;  Wo
    right        y = gelu_tanh(Wy h + by), u = causal convolution per channel of (Wx h + bx);  per block b of channels
                 r, i = sigmoid(R_b u_b + .), sigmoid(I_b u_b + .);  a = exp(-8 r softplus(lam));
                 S <- a S + sqrt(1 - a^2) i u;  Wo (S y)
  retention      q, k turned as above, k / sqrt(d);  S <- decay S + k v^T;  o = S^T q;  o / rms(o) per head;
                 times silu(Wg h);  Wo
  feed-forward   g = min(Wgate h, L), u = clip(Wup h, -L, L);  Wdown (g sigmoid(1.702 g) (u + 1))
  output         E gn(x)
"""
from __future__ import annotations

import math

import numpy as np

F64 = np.float64


def linear(x, w, b=None):
    y = np.asarray(x, F64) @ np.asarray(w, F64).T
    return y if b is None else y + np.asarray(b, F64)


def sigmoid(z):
    z = np.asarray(z, F64)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, F64))


def gelu_tanh(z):
    z = np.asarray(z, F64)
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, gain, eps):
    x = np.asarray(x, F64)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if gain is None else y * np.asarray(gain, F64)


def group_norm(x, gain, eps, groups):
    x = np.asarray(x, F64)
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms_norm(parts, None, eps).reshape(x.shape) * np.asarray(gain, F64)


# ---------------------------------------------------------------------------------------------- rotation
def frequencies(rot):
    n, base = rot["dims"], float(rot["base"])
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)], F64)
    sc = rot.get("scaling")
    if not sc:
        return f
    out = []
    for v in f:
        wave = 2.0 * math.pi / v
        if wave < sc["original"] / sc["high"]:
            out.append(v)
        elif wave > sc["original"] / sc["low"]:
            out.append(v / sc["factor"])
        else:
            s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * v / sc["factor"] + s * v)
    return np.array(out, F64)


def rotate(x, rot):
    """x [T, heads, d]: pairs (i, i + n/2) of the first n dimensions turned by p * f_i; the rest as they are."""
    if not rot or not rot.get("dims"):
        return np.asarray(x, F64)
    n = rot["dims"]
    ang = np.arange(x.shape[0], dtype=F64)[:, None] * frequencies(rot)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., n:]], axis=-1)


# ---------------------------------------------------------------------------------------------- mixers
def visible(T, size):
    """[query, key]: whether the query's position sees the key's.  size None or 0: every earlier key."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    ok = j <= i
    return ok & (i // size == j // size) if size else ok


def chunked_attention(m, eps, W, h, p):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(linear(h, W[p + "q"]), W[p + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(linear(h, W[p + "k"]), W[p + "k.norm"], eps).reshape(T, G, d)
    v = linear(h, W[p + "v"]).reshape(T, G, dv)
    q, k = rotate(q, m.get("rot")), rotate(k, m.get("rot"))
    mask = visible(T, (m.get("mask") or {}).get("size"))
    out = np.zeros((T, H, dv), F64)
    for j in range(H):
        g = j // (H // G)
        s = np.where(mask, q[:, j] @ k[:, g].T * m["scale"] * float(W[p + "temp"][j]), -np.inf)
        e = np.exp(s - s.max(axis=-1, keepdims=True))
        out[:, j] = e / e.sum(axis=-1, keepdims=True) @ v[:, g]
    o = out.reshape(T, H * dv) * sigmoid(linear(h, W[p + "g"]))
    return linear(o, W[p + "o"])


def causal_conv(x, w, b):
    """x [T, C], w [C, taps] (the last column is the current token's), b [C]."""
    T, taps = x.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1]), F64), x])
    out = np.tile(np.asarray(b, F64), (T, 1))
    for n in range(taps):
        out += padded[n:n + T] * np.asarray(w, F64)[:, n]
    return out


def linear_recurrence(u, blocks, W, p):
    """S of every token, [T, width]."""
    T, width = u.shape
    ub = u.reshape(T, blocks, width // blocks)
    r = sigmoid(np.einsum("tbi,boi->tbo", ub, np.asarray(W[p + "ra"], F64)) + np.asarray(W[p + "ra.b"], F64)).reshape(T, width)
    i = sigmoid(np.einsum("tbi,boi->tbo", ub, np.asarray(W[p + "ri"], F64)) + np.asarray(W[p + "ri.b"], F64)).reshape(T, width)
    log_a = -8.0 * r * softplus(W[p + "lam"])
    a, b = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a)) * i * u
    S, out = np.zeros(width, F64), np.zeros((T, width), F64)
    for t in range(T):
        S = a[t] * S + b[t]
        out[t] = S
    return out


def recurrent_block(m, W, h, p):
    y = gelu_tanh(linear(h, W[p + "y"], W[p + "y.b"]))
    u = causal_conv(linear(h, W[p + "x"], W[p + "x.b"]), W[p + "conv"], W[p + "conv.b"])
    return linear(linear_recurrence(u, m["blocks"], W, p) * y, W[p + "o"])


def parallel(m, eps, W, h, p):
    left = chunked_attention(m["left"], eps, W, h, p + "left.")
    right = recurrent_block(m["right"], W, h, p + "right.")
    return 0.5 * (rms_norm(left, W[p + "left.out"], eps) + rms_norm(right, W[p + "right.out"], eps))


def retention(m, eps, W, h, p):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = rotate(linear(h, W[p + "q"]).reshape(T, H, d), m.get("rot"))
    k = rotate(linear(h, W[p + "k"]).reshape(T, H, d), m.get("rot")) / math.sqrt(d)
    v = linear(h, W[p + "v"]).reshape(T, H, dv)
    S, o = np.zeros((H, d, dv), F64), np.zeros((T, H, dv), F64)
    decay = np.asarray(m["decay"], F64)[:, None, None]
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    g = linear(h, W[p + "g"])
    return linear(rms_norm(o, None, eps).reshape(T, H * dv) * g * sigmoid(g), W[p + "o"])


# ---------------------------------------------------------------------------------------------- the rest
def feed_forward(f, W, h, p):
    g = np.minimum(linear(h, W[p + "gate"]), f["limit"])
    u = np.clip(linear(h, W[p + "up"]), -f["limit"], f["limit"])
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), W[p + "down"])


def mixer(layer, eps, W, h, p):
    return (parallel if layer["type"] == "parallel" else retention)(layer["mixer"], eps, W, h, p)


def forward(cfg, W, tokens, stream=None):
    """Logits [T, vocab] of a whole sequence; stream: a list that receives the residual stream behind every layer."""
    eps, groups, alpha = cfg["norm"]["eps"], cfg["norm"].get("groups", 1), cfg.get("postln_alpha", 1.0)
    table = np.asarray(W["embed"], F64)
    x = group_norm(table[np.asarray(tokens)], W["embed.norm"], eps, groups)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = group_norm(alpha * x + mixer(layer, eps, W, x, p + "mix."), W[p + "norm1"], eps, groups)
        if layer.get("mlp") is not None:
            x = group_norm(alpha * x + feed_forward(layer["mlp"], W, x, p + "mlp."), W[p + "norm2"], eps, groups)
        if stream is not None:
            stream.append(x.copy())
    return group_norm(x, W["final.norm"], eps, groups) @ table.T
