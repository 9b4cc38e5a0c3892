"""A plain, slow float64 restatement of the Gebadra design, one function per mechanism, token by token.

It shares no code with the library: keys and values sit in Python lists, a pooled block is averaged from the list every
time a token looks at it, the linear recurrences keep one matrix per head, the hyper-connection streams are a list of
vectors.

Notation: W is applied as W @ x; `w` maps tensor names to float64 arrays; a mixer's tensors are '<layer>.mix.<name>'.
The keyword arguments named `fault_*` plant a mistake so that a test can show that the mistake would be seen.
"""
import math

import numpy as np


# ------------------------------------------------------------------------------------------------ small functions
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis (weight None: no weight)"""
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def layer_norm(x, weight, bias, eps):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * weight + bias"""
    c = x - np.mean(x)
    return c / math.sqrt(float(np.mean(c * c)) + eps) * weight + bias


# ------------------------------------------------------------------------------------------------ hyper-connections
def streams_read(streams, w_in):
    return sum(float(a) * x for a, x in zip(w_in, streams))


def streams_write(streams, mix, w_out, y, fault_transposed=False):
    """new stream t = sum over s of mix[s, t] * old stream s + w_out[t] * y"""
    m = mix.T if fault_transposed else mix
    n = len(streams)
    return [sum(float(m[s, t]) * streams[s] for s in range(n)) + float(w_out[t]) * y for t in range(n)]


# ------------------------------------------------------------------------------------------------ rotary positions
def rotate_neighbours(vec, pos, rot, pairing="neighbours", fault_unscaled=False):
    """rotary positions on the first rot.dims elements: element 2i pairs with 2i + 1 (pairing 'half' pairs i with
    i + dims/2 and exists so that a test can show that the pairing matters); frequencies base^(-2i/dims) / factor"""
    out = vec.copy()
    if not rot or not rot.get("dims"):
        return out
    dims = rot["dims"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    if fault_unscaled:
        factor = 1.0
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if pairing == "neighbours" else (i, i + dims // 2)
        ang = pos * rot["base"] ** (-2.0 * i / dims) / factor
        c, s = math.cos(ang), math.sin(ang)
        out[a] = vec[a] * c - vec[b] * s
        out[b] = vec[b] * c + vec[a] * s
    return out


# ------------------------------------------------------------------------------------------------ attention
def visible(pos, size, pool):
    """-> (block numbers, token positions) that position pos sees"""
    tokens = [j for j in range(pos + 1) if pos - j < size]
    blocks, b = [], 0
    while b * pool + pool - 1 <= pos - size:
        blocks.append(b)
        b += 1
    return blocks, tokens


def talking_attention(w, p, mx, h, pos, cache, eps, pairing="neighbours", fault_no_talk=False, fault_per_head_norm=False,
                      fault_unscaled=False, fault_no_pool=False, fault_pool_sees_early=0):
    """one token; cache: list of (keys [G, dim] normed and rotated, values [G, vdim]) of all earlier tokens"""
    H, G, d, vd = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    rot, size, pool = mx.get("rot"), mx["mask"]["size"], mx["mask"]["pool"]

    def normed(x, weight, heads):
        if fault_per_head_norm:
            return (rms_norm(x.reshape(heads, d), None, eps) * weight.reshape(heads, d))
        return rms_norm(x, weight, eps).reshape(heads, d)
    q = normed(w[p + "q"] @ h, w[p + "q.norm"], H)
    k = normed(w[p + "k"] @ h, w[p + "k.norm"], G)
    v = (w[p + "v"] @ h).reshape(G, vd)
    q = np.stack([rotate_neighbours(x, pos, rot, pairing, fault_unscaled) for x in q])
    k = np.stack([rotate_neighbours(x, pos, rot, pairing, fault_unscaled) for x in k])
    cache.append((k, v))
    blocks, tokens = visible(pos, size, pool)
    if fault_pool_sees_early:
        blocks, _ = visible(pos + fault_pool_sees_early, size, pool)
    if fault_no_pool:
        blocks = []
    keys, vals = [], []
    for b in blocks:
        members = [cache[j] for j in range(b * pool, (b + 1) * pool)]
        keys.append(sum(m[0] for m in members) / pool)
        vals.append(sum(m[1] for m in members) / pool)
    keys += [cache[j][0] for j in tokens]
    vals += [cache[j][1] for j in tokens]
    K, V = np.stack(keys), np.stack(vals)  # [n, G, dim], [n, G, vdim]
    weight = np.empty((H, len(keys)))
    for a in range(H):
        s = K[:, a // (H // G)] @ q[a] * mx["scale"]
        e = np.exp(s - s.max())
        weight[a] = e / e.sum()
    if not fault_no_talk:
        weight = w[p + "talk"] @ weight
    out = np.stack([weight[a] @ V[:, a // (H // G)] for a in range(H)])
    return w[p + "o"] @ out.reshape(-1)


# ------------------------------------------------------------------------------------------------ linear recurrences
def decayed_outer_step(state, q, k, v, decay):
    """state [heads, dim, vdim] in place: S = decay S + k v^T per head; -> o [heads, vdim] = S^T q"""
    out = np.empty((state.shape[0], state.shape[2]))
    for a in range(state.shape[0]):
        state[a] = decay[a] * state[a] + np.outer(k[a], v[a])
        out[a] = state[a].T @ q[a]
    return out


def lightning_step(w, p, mx, h, state, eps):
    H, d, vd = mx["heads"], mx["dim"], mx["vdim"]
    q = silu(w[p + "q"] @ h).reshape(H, d)
    k = silu(w[p + "k"] @ h).reshape(H, d)
    v = silu(w[p + "v"] @ h).reshape(H, vd)
    o = decayed_outer_step(state, q, k, v, mx["decay"]).reshape(-1)
    return w[p + "o"] @ (rms_norm(o, w[p + "norm"], eps) * sigmoid(w[p + "g"] @ h))


def retention_step(w, p, mx, h, state, eps):
    H, d, vd = mx["heads"], mx["dim"], mx["vdim"]
    q = (w[p + "q"] @ h).reshape(H, d)
    k = (w[p + "k"] @ h).reshape(H, d) / math.sqrt(d)
    v = (w[p + "v"] @ h).reshape(H, vd)
    o = rms_norm(decayed_outer_step(state, q, k, v, mx["decay"]), None, eps).reshape(-1)
    return w[p + "o"] @ (o * silu(w[p + "g"] @ h))


def parallel_step(w, p, mx, h, pos, carried, eps, **kw):
    """attention and retention of the same input; each output RMS-normed, half of their sum; carried: (cache, state)"""
    left = talking_attention(w, p + "left.", mx["left"], h, pos, carried[0], eps, **kw)
    right = retention_step(w, p + "right.", mx["right"], h, carried[1], eps)
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


def gated_feed_forward(w, p, h):
    return w[p + "down"] @ (silu(w[p + "gate"] @ h) * (w[p + "up"] @ h))


# ------------------------------------------------------------------------------------------------ the model
def weight_layer(cfg, i):
    """the layer whose tensors layer i uses"""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


class Stepper:
    """feeds tokens one by one; every layer keeps what its mixer carries, also a layer that uses another layer's weights"""

    def __init__(self, cfg, w, fault_transposed=False, fault_shared_state=False, **kw):
        self.cfg, self.w, self.pos, self.kw, self.fault_transposed = cfg, w, 0, kw, fault_transposed
        self.carried = []
        for i, ly in enumerate(cfg["layers"]):
            mx = ly["mixer"]
            if fault_shared_state and ly.get("weights_of") is not None:
                self.carried.append(self.carried[ly["weights_of"]])
            elif ly["type"] == "lightning":
                self.carried.append(np.zeros((mx["heads"], mx["dim"], mx["vdim"])))
            else:
                r = mx["right"]
                self.carried.append(([], np.zeros((r["heads"], r["dim"], r["vdim"]))))

    def step(self, token):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        streams = [w["embed"][token].copy() for _ in range(cfg["streams"])]
        after = []
        for i, ly in enumerate(cfg["layers"]):
            p = f"l{weight_layer(cfg, i)}."
            for q in (1, 2):
                if q == 2 and not ly.get("mlp"):
                    continue
                u = streams_read(streams, w[p + f"hc{q}.in"])
                h = layer_norm(u, w[p + f"norm{q}"], w[p + f"norm{q}.b"], eps)
                if q == 2:
                    y = gated_feed_forward(w, p + "mlp.", h)
                elif ly["type"] == "lightning":
                    y = lightning_step(w, p + "mix.", ly["mixer"], h, self.carried[i], eps)
                else:
                    y = parallel_step(w, p + "mix.", ly["mixer"], h, self.pos, self.carried[i], eps, **self.kw)
                streams = streams_write(streams, w[p + f"hc{q}.mix"], w[p + f"hc{q}.out"], y, self.fault_transposed)
            after.append(sum(streams))
        self.pos += 1
        return w["head"] @ layer_norm(sum(streams), w["final.norm"], w["final.norm.b"], eps), np.stack(after)

    def run(self, tokens):
        """-> logits [n, vocab], sum of the streams after every layer [layers, n, width]"""
        out = [self.step(t) for t in tokens]
        return np.stack([o[0] for o in out]), np.stack([o[1] for o in out], axis=1)


def forward(cfg, w, tokens, **kw):
    return Stepper(cfg, w, **kw).run(tokens)
