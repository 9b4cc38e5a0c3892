"""A plain, slow float64 restatement of the Gubanex design, one function per mechanism, token by token.

It shares no code with the library: keys and values sit in Python lists that are searched position by position, the gated
linear recurrence keeps one matrix per head, an expert is called with its scaled input, the loop is an explicit list of runs.

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


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def zero_centred_norm(x, weight, eps, fault_plain_weight=False):
    """an RMS norm with a zero-centred weight: the factor is 1 + weight"""
    return unit_rms(x, eps) * (weight if fault_plain_weight else 1.0 + weight)


def softcap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# ------------------------------------------------------------------------------------------------ rotary positions
def frequencies(rot, fault_unscaled=False, fault_no_blend=False):
    """f_i = base^(-2i/dims), with scaling by wavelength: short ones stay, long ones are divided by the factor, a blend between"""
    out = []
    sc = None if fault_unscaled else rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                if fault_no_blend:
                    s = 1.0
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(vec, pos, rot, pairing="half", **kw):
    """rotary positions on the first rot.dims elements: element i pairs with i + dims/2 (pairing 'neighbours' pairs 2i with
    2i + 1 and exists so that a test can show that the pairing matters)"""
    out = vec.copy()
    if not rot or not rot.get("dims"):
        return out
    half = rot["dims"] // 2
    for i, f in enumerate(frequencies(rot, **kw)):
        a, b = (i, i + half) if pairing == "half" else (2 * i, 2 * i + 1)
        c, s = math.cos(pos * f), math.sin(pos * f)
        out[a] = vec[a] * c - vec[b] * s
        out[b] = vec[b] * c + vec[a] * s
    return out


# ------------------------------------------------------------------------------------------------ mixers
def visible(pos, size, shift=0):
    """positions that pos sees: the ones of its own chunk up to itself (shift moves the chunks' borders: a planted mistake)"""
    return [j for j in range(pos + 1) if not size or (j + shift) // size == (pos + shift) // size]


def chunked_attention(w, p, mx, h, pos, cache, eps, fault_no_qk_norm=False, fault_chunk_shift=0, fault_window=False, pairing="half",
                      fault_unscaled=False, fault_no_blend=False, fault_heads_interleaved=False):
    """one token; cache: list of (keys [G, dim] rotated and normed, values [G, vdim]) of all earlier tokens"""
    H, G, d, vd = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    rot, size = mx.get("rot"), (mx.get("mask") or {}).get("size", 0)
    turn = dict(pairing=pairing, fault_unscaled=fault_unscaled, fault_no_blend=fault_no_blend)
    q = np.stack([rotate(x, pos, rot, **turn) for x in (w[p + "q"] @ h).reshape(H, d)])
    k = np.stack([rotate(x, pos, rot, **turn) for x in (w[p + "k"] @ h).reshape(G, d)])
    if not fault_no_qk_norm:
        q, k = unit_rms(q, eps), unit_rms(k, eps)
    cache.append((k, (w[p + "v"] @ h).reshape(G, vd)))
    seen = [j for j in range(pos + 1) if pos - j < size] if fault_window else visible(pos, size, fault_chunk_shift)
    out = np.empty((H, vd))
    for a in range(H):
        g = a % G if fault_heads_interleaved else a // (H // G)
        s = np.array([cache[j][0][g] @ q[a] for j in seen]) * mx["scale"]
        e = np.exp(s - s.max())
        out[a] = (e / e.sum()) @ np.stack([cache[j][1][g] for j in seen])
    return w[p + "o"] @ out.reshape(-1)


def channel_decay(w, p, mx, h, fault_no_tau=False):
    """decay of every key channel [heads, dim]: a low-rank map with a bias, squashed, to the power 1 / tau"""
    z = w[p + "a2"] @ (w[p + "a1"] @ h) + w[p + "a2.b"]
    return (sigmoid(z) ** (1.0 if fault_no_tau else 1.0 / mx["tau"])).reshape(mx["heads"], mx["dim"])


def gated_linear_step(w, p, mx, h, state, eps, fault_no_tau=False, fault_decay_after=False, fault_no_q_scale=False, fault_head_decay=False):
    """one token; state [heads, dim, vdim] in place: row d of a head's matrix decays with channel d"""
    H, d, vd = mx["heads"], mx["dim"], mx["vdim"]
    q = (w[p + "q"] @ h).reshape(H, d) * (1.0 if fault_no_q_scale else d ** -0.5)
    k = (w[p + "k"] @ h).reshape(H, d)
    v = (w[p + "v"] @ h).reshape(H, vd)
    alpha = channel_decay(w, p, mx, h, fault_no_tau)
    if fault_head_decay:
        alpha = np.repeat(alpha.mean(axis=1, keepdims=True), d, axis=1)
    out = np.empty((H, vd))
    for a in range(H):
        if fault_decay_after:
            state[a] = alpha[a][:, None] * (state[a] + np.outer(k[a], v[a]))
        else:
            state[a] = alpha[a][:, None] * state[a] + np.outer(k[a], v[a])
        out[a] = state[a].T @ q[a]
    o = (unit_rms(out, eps) * w[p + "norm"]).reshape(-1)
    return w[p + "o"] @ (o * silu(w[p + "g"] @ h))


# ------------------------------------------------------------------------------------------------ feed-forward
def route(z, top):
    """-> (chosen experts, their weights): the largest sigmoid scores, not renormalised, the lowest index among equals"""
    s = sigmoid(z)
    order = sorted(range(len(s)), key=lambda e: (-s[e], e))[:top]
    return order, [float(s[e]) for e in order]


def expert(w, p, x):
    return w[p + "down"] @ (silu(w[p + "gate"] @ x) * (w[p + "up"] @ x))


def expert_mixture(w, p, mlp, h, fault_output_weight=False, fault_renormalised=False):
    chosen, weights = route(w[p + "router"] @ h, mlp["router"]["top"])
    if fault_renormalised:
        weights = [x / sum(weights) for x in weights]
    if fault_output_weight:
        return sum(g * expert(w, p + f"e{e}.", h) for e, g in zip(chosen, weights))
    return sum(expert(w, p + f"e{e}.", g * h) for e, g in zip(chosen, weights))


# ------------------------------------------------------------------------------------------------ the model
def layer_runs(cfg):
    """-> list of (layer, pass number if the layer opens a pass of the loop, else None)"""
    n, lp = len(cfg["layers"]), cfg.get("loop") or {}
    a, b, times = lp.get("start", 0), lp.get("stop", 0), lp.get("times", 1)
    out = [(i, None) for i in range(a)]
    for t in range(times if b > a else 0):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(max(a, b), n)]


class Stepper:
    """feeds tokens one by one; every run of a layer keeps what its mixer carries"""

    def __init__(self, cfg, w, fault_shared_passes=False, fault_no_reentry=False, fault_plain_weight=False, mixer=None, linear=None, mlp=None):
        self.cfg, self.w, self.pos, self.runs = cfg, w, 0, layer_runs(cfg)
        self.no_reentry, self.plain = fault_no_reentry, fault_plain_weight
        self.mixer_kw, self.linear_kw, self.mlp_kw = mixer or {}, linear or {}, mlp or {}
        self.carried, first = [], {}
        for i, _ in self.runs:
            ly = cfg["layers"][i]
            mx = ly["mixer"]
            c = [] if ly["type"] == "attention" else np.zeros((mx["heads"], mx["dim"], mx["vdim"]))
            if fault_shared_passes:
                c = first.setdefault(i, c)
            self.carried.append(c)

    def step(self, token):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        entry = w["embed"][token] * cfg["embedding"]["scale"]
        x, after = entry.copy(), []
        for (i, opens), carried in zip(self.runs, self.carried):
            if opens and not self.no_reentry:
                x = x + entry
            ly, p = cfg["layers"][i], f"l{i}."
            h = zero_centred_norm(x, w[p + "norm1"], eps, self.plain)
            if ly["type"] == "attention":
                x = x + chunked_attention(w, p + "mix.", ly["mixer"], h, self.pos, carried, eps, **self.mixer_kw)
            else:
                x = x + gated_linear_step(w, p + "mix.", ly["mixer"], h, carried, eps, **self.linear_kw)
            if ly.get("mlp"):
                h = zero_centred_norm(x, w[p + "norm2"], eps, self.plain)
                x = x + expert_mixture(w, p + "mlp.", ly["mlp"], h, **self.mlp_kw)
            after.append(x.copy())
        self.pos += 1
        z = w["head"] @ zero_centred_norm(x, w["final.norm"], eps, self.plain) * cfg.get("logit_scale", 1.0)
        return softcap(z, cfg.get("logit_softcap", 0.0)), np.stack(after)

    def run(self, tokens):
        """-> logits [n, vocab], the residual stream after every layer run [runs, n, width]"""
        out = [self.step(t) for t in tokens]
        return np.stack([o[0] for o in out]), np.stack([o[1] for o in out], axis=1)


def forward(cfg, w, tokens, **kw):
    return Stepper(cfg, w, **kw).run(tokens)
