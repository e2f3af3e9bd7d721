"""Plain, slow restatement of the Memipel decoder, used only as a test oracle.

Whole sequences, no cache, one function per mechanism, float64 throughout, no code shared with the product
package.  Notation: h is a sublayer's input [T, width]; p, t positions 0..T-1; a weight matrix is [out, in] and
acts as h @ W.T; cfg is the config.json object, W a dict name -> array.

  layer             h = rms(x) (1 + w);  x <- x + mixer(h) + ff(h)
  attention         q, k, v = conv(W h + b);  score q . k * scale - 2^(-8 (head + 1) / H) (p - t) over 0 <= p - t < size;
                    softmax;  v is (1 - l) v + l v1, v1 the values of the first layer that mixes;  Wo . + bo
  latent attention  q = Wuq rms(Wdq h);  c = rms(Wdkv h);  k = Wuk c, v = Wuv c;  score q . k * scale over
                    0 <= p - t < size;  the softmax's denominator has one more term exp(sink_head);  Wo
  lightning         q, k, v = silu(W h);  S <- decay S + k v^T;  o = S^T q;  rms over all heads together * w
                    * sigmoid(Wg h);  Wo
  dense             Wdown gelu(Wup h), gelu(z) = z Phi(z)
  experts           s = softmax(Wr h);  groups of neighbours by their largest s, the best `keep` stay;  the `top`
                    largest s there;  sum of s_e E_e(h), and the shared expert's output;
                    E(h) = Wdown (g sigmoid(1.702 g) (u + 1)), g = min(Wgate h, L), u = clip(Wup h, -L, L)
  output            E rms(x) (1 + w)
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


def silu(z):
    return np.asarray(z, F64) * sigmoid(z)


def gelu(z):
    z = np.asarray(z, F64)
    return z * 0.5 * (1.0 + np.vectorize(math.erf, otypes=[F64])(z / math.sqrt(2.0)))


def rms_norm(x, gain, eps):
    x = np.asarray(x, F64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * np.asarray(gain, F64)


def stored_around_zero_norm(x, w, eps):
    return rms_norm(x, 1.0 + np.asarray(w, F64), eps)


def short_conv(u, w):
    """y_p = sum over j of w[:, j] u_(p - taps + 1 + j), channel by channel; nothing stands in front of position 0."""
    u, w = np.asarray(u, F64), np.asarray(w, F64)
    taps = w.shape[1]
    past = np.concatenate([np.zeros((taps - 1, u.shape[1])), u], axis=0)
    return sum(past[j:j + u.shape[0]] * w[:, j] for j in range(taps))


def visible(T, window):
    """[p, t]: t is not ahead of p and, with a window, among the `window` last tokens up to p itself."""
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (back >= 0) & ((back < window) if window else True)


def slopes(heads):
    return 2.0 ** (-8.0 * (np.arange(heads) + 1) / heads)


def softmax_read(scores, vis, v, sink=None):
    """[T, T] scores, [T, dv] values -> [T, dv]; sink: the logarithm of one more term of every denominator."""
    s = np.where(vis, scores, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    den = e.sum(axis=-1, keepdims=True) + (0.0 if sink is None else np.exp(sink - top))
    return (e / den) @ v


def attention_values(m, W, h, pre):
    v = linear(h, W[pre + "v"], W[pre + "v.b"])
    return short_conv(v, W[pre + "v.conv"]) if m.get("conv") else v


def attention(m, W, h, pre, v_first=None):
    """v_first: the values to mix in (None: none)."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (linear(h, W[pre + n], W[pre + n + ".b"]) for n in ("q", "k"))
    if m.get("conv"):
        q, k = short_conv(q, W[pre + "q.conv"]), short_conv(k, W[pre + "k.conv"])
    v = attention_values(m, W, h, pre)
    if v_first is not None:
        lam = float(np.asarray(W[pre + "vmix"]).reshape(()))
        v = (1.0 - lam) * v + lam * v_first
    q, k, v = q.reshape(T, H, D), k.reshape(T, G, D), v.reshape(T, G, V)
    vis = visible(T, (m.get("mask") or {}).get("size", 0))
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, V))
    for j in range(H):
        g = j // (H // G)
        out[:, j] = softmax_read(q[:, j] @ k[:, g].T * m["scale"] - slopes(H)[j] * back, vis, v[:, g])
    return linear(out.reshape(T, H * V), W[pre + "o"], W[pre + "o.b"])


def latent_attention(m, eps, W, h, pre):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(rms_norm(linear(h, W[pre + "dq"]), W[pre + "dq.norm"], eps), W[pre + "uq"]).reshape(T, H, D)
    c = rms_norm(linear(h, W[pre + "dkv"]), W[pre + "dkv.norm"], eps)
    k, v = linear(c, W[pre + "uk"]).reshape(T, H, D), linear(c, W[pre + "uv"]).reshape(T, H, V)
    vis = visible(T, (m.get("mask") or {}).get("size", 0))
    out = np.zeros((T, H, V))
    for j in range(H):
        out[:, j] = softmax_read(q[:, j] @ k[:, j].T * m["scale"], vis, v[:, j], W[pre + "sink"][j])
    return linear(out.reshape(T, H * V), W[pre + "o"])


def lightning_read(q, k, v, decay):
    """q, k [T, H, D], v [T, H, V] -> o [T, H, V] and the last state [H, D, V]."""
    T, H, D = q.shape
    S, out = np.zeros((H, D, v.shape[2])), np.zeros((T, H, v.shape[2]))
    decay = np.asarray(decay, F64)[:, None, None]
    for p in range(T):
        S = decay * S + k[p][:, :, None] * v[p][:, None, :]
        out[p] = np.einsum("hdv,hd->hv", S, q[p])
    return out, S


def lightning(m, eps, W, h, pre):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(linear(h, W[pre + n])).reshape(T, H, D) for n in ("q", "k"))
    v = silu(linear(h, W[pre + "v"])).reshape(T, H, V)
    o = lightning_read(q, k, v, m["decay"])[0].reshape(T, H * V)
    return linear(rms_norm(o, W[pre + "norm"], eps) * sigmoid(linear(h, W[pre + "g"])), W[pre + "o"])


def dense(W, h, pre):
    return linear(gelu(linear(h, W[pre + "up"])), W[pre + "down"])


def clamped_expert(W, h, pre, limit):
    g = np.minimum(linear(h, W[pre + "gate"]), limit)
    u = np.clip(linear(h, W[pre + "up"]), -limit, limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), W[pre + "down"])


def route(z, top, count=1, keep=1):
    """Logits [T, E] -> the experts' weights [T, E], zero where not chosen."""
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    T, E = s.shape
    best = s.reshape(T, count, E // count).max(axis=-1)
    out = np.zeros_like(s)
    for t in range(T):
        open_groups = np.argsort(-best[t], kind="stable")[:keep]
        can = [e_ for e_ in range(E) if e_ // (E // count) in open_groups]
        for e_ in sorted(can, key=lambda i: -s[t, i])[:top]:
            out[t, e_] = s[t, e_]
    return out


def route_margin(z, top, count=1, keep=1):
    """How far (in logits) the nearest of all choices of groups and of experts is from turning out otherwise."""
    T, E = z.shape
    best = z.reshape(T, count, E // count).max(axis=-1)
    near = np.inf
    for t in range(T):
        order = np.argsort(-best[t], kind="stable")
        if keep < count:
            near = min(near, best[t, order[keep - 1]] - best[t, order[keep]])
        can = np.sort([z[t, e] for e in range(E) if e // (E // count) in order[:keep]])[::-1]
        if top < len(can):
            near = min(near, can[top - 1] - can[top])
    return near


def experts(f, W, h, pre, margins=None):
    r = f["router"]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    z = linear(h, W[pre + "router"])
    if margins is not None:
        margins.append(route_margin(z, r["top"], gr["count"], gr["keep"]))
    weights = route(z, r["top"], gr["count"], gr["keep"])
    y = np.zeros_like(np.asarray(h, F64))
    for e in range(r["experts"]):
        y += weights[:, e:e + 1] * clamped_expert(W, h, f"{pre}e{e}.", f["expert"]["limit"])
    if f.get("shared"):
        y += clamped_expert(W, h, pre + "shared.", f["shared"]["limit"])
    return y


def feed_forward(f, W, h, pre, margins=None):
    return dense(W, h, pre) if f["kind"] == "dense" else experts(f, W, h, pre, margins)


def forward(cfg, W, tokens, residuals=None, margins=None, noise=None):
    """Logits [T, vocab]; residuals: a list that receives the stream after every layer; margins: one that receives every
    router's route_margin; noise: called on every norm's output (to ask how far rounding of a given width reaches)."""
    eps = cfg["norm"]["eps"]
    noise = noise or (lambda a: a)
    x = np.asarray(W["embed"], F64)[np.asarray(tokens)]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        h = noise(stored_around_zero_norm(x, W[pre + "norm1"], eps))
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y = attention(m, W, h, pre + "mix.", v_first if mixes else None)
            if mixes and v_first is None:
                v_first = attention_values(m, W, h, pre + "mix.")
        elif layer["type"] == "latent_attention":
            y = latent_attention(m, eps, W, h, pre + "mix.")
        else:
            y = lightning(m, eps, W, h, pre + "mix.")
        if layer.get("mlp") is not None:
            y = y + feed_forward(layer["mlp"], W, h, pre + "mlp.", margins)
        x = x + y
        if residuals is not None:
            residuals.append(x.copy())
    return linear(noise(stored_around_zero_norm(x, W["final.norm"], eps)), W["embed"])
