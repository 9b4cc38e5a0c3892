"""Helpers of the Gebadra tests: small configurations and bf16-exact random weights written as a model folder
(config.json + model.safetensors)."""
import numpy as np

from nogatar_util import bf16_round, rel_err, values, write_model  # noqa: F401  (format helpers, not model code)


def decays(n, lo=0.6, hi=0.995):
    return [float(x) for x in np.linspace(lo, hi, n)]


def lightning(heads=3, dim=6, vdim=5, decay=None, mlp=None, weights_of=None):
    ly = {"type": "lightning", "mixer": {"decay": decay or decays(heads), "dim": dim, "heads": heads, "vdim": vdim}, "mlp": mlp}
    if weights_of is not None:
        ly["weights_of"] = weights_of
    return ly


def parallel(heads=4, kv_heads=2, dim=6, vdim=5, size=7, pool=3, scale=0.6, rot_dims=4, base=100.0, factor=2.0, rheads=2, rdim=4, rvdim=6,
             decay=None, mlp=None, weights_of=None):
    left = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"pool": pool, "size": size}, "scale": scale, "vdim": vdim}
    if rot_dims:
        left["rot"] = {"base": base, "dims": rot_dims}
        if factor:
            left["rot"]["scaling"] = {"factor": factor}
    right = {"decay": decay or decays(rheads), "dim": rdim, "heads": rheads, "vdim": rvdim}
    ly = {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}
    if weights_of is not None:
        ly["weights_of"] = weights_of
    return ly


def dense(ff=14):
    return {"ff": ff, "kind": "dense"}


def make_config(layers, width=20, vocab=37, eps=1e-5, streams=2):
    return {"architecture": "Gebadra", "layers": layers, "norm": {"eps": eps}, "streams": streams, "vocab": vocab, "width": width}


def tensor_shapes(cfg):
    W, S = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], W)}
    for i, ly in enumerate(cfg["layers"]):
        if ly.get("weights_of") is not None:
            continue
        p, mx = f"l{i}.", ly["mixer"]
        for q in (1, 2):
            if q == 2 and not ly.get("mlp"):
                continue
            out.update({p + f"norm{q}": (W,), p + f"norm{q}.b": (W,), p + f"hc{q}.in": (S,), p + f"hc{q}.out": (S,), p + f"hc{q}.mix": (S, S)})
        lin, lp = (mx, p + "mix.") if ly["type"] == "lightning" else (mx["right"], p + "mix.right.")
        nk, nv = lin["heads"] * lin["dim"], lin["heads"] * lin["vdim"]
        out.update({lp + "q": (nk, W), lp + "k": (nk, W), lp + "v": (nv, W), lp + "g": (nv, W), lp + "o": (W, nv)})
        if ly["type"] == "lightning":
            out[p + "mix.norm"] = (nv,)
        else:
            lf, a = mx["left"], p + "mix.left."
            H, G, d, vd = lf["heads"], lf["kv_heads"], lf["dim"], lf["vdim"]
            out.update({a + "q": (H * d, W), a + "k": (G * d, W), a + "v": (G * vd, W), a + "q.norm": (H * d,), a + "k.norm": (G * d,),
                        a + "talk": (H, H), a + "o": (W, H * vd), a + "out": (W,), p + "mix.right.out": (W,)})
        if ly.get("mlp"):
            ff = ly["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    out.update({"final.norm": (W,), "final.norm.b": (W,), "head": (cfg["vocab"], W)})
    return out


def random_weights(cfg, seed=0, gain=1.0):
    """name -> (bf16 bits, float64 values)"""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        parts = name.split(".")
        if name == "embed":
            a = rng.standard_normal(shape)
        elif parts[-1] == "talk":
            a = np.eye(shape[0]) + 0.5 * rng.standard_normal(shape) / np.sqrt(shape[0])
        elif len(parts) > 2 and parts[1].startswith("hc"):
            a = np.eye(shape[0]) + 0.3 * rng.standard_normal(shape) if parts[2] == "mix" else 0.7 + 0.4 * rng.standard_normal(shape)
        elif len(shape) == 2:
            a = rng.standard_normal(shape) * gain / np.sqrt(shape[1])
        elif parts[-1] == "b":
            a = 0.3 * rng.standard_normal(shape)
        else:
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        out[name] = bf16_round(np.asarray(a, np.float32))
    return out


def set_values(weights, name, vals):
    weights[name] = bf16_round(np.asarray(vals, np.float32))
