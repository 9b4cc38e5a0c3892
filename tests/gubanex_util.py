"""Helpers of the Gubanex tests: small configurations and bf16-exact random weights written as a model folder
(config.json + model.safetensors)."""
import numpy as np

from nogatar_util import bf16_round, rel_err, values, write_model  # noqa: F401  (format helpers, not model code)


def waves(factor=3.0, low=1.0, high=4.0, original=32):
    return {"factor": factor, "high": high, "low": low, "original": original}


def attention(heads=4, kv_heads=2, dim=6, vdim=5, size=7, scale=0.9, rot_dims=4, base=50.0, scaling=None, mlp=None):
    mx = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if size:
        mx["mask"] = {"size": size}
    if rot_dims:
        mx["rot"] = {"base": base, "dims": rot_dims, "scaling": scaling if scaling is not None else waves()}
        if not mx["rot"]["scaling"]:
            del mx["rot"]["scaling"]
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def gla(heads=3, dim=6, vdim=5, tau=4.0, mlp=None):
    return {"type": "gla", "mixer": {"dim": dim, "heads": heads, "tau": tau, "vdim": vdim}, "mlp": mlp}


def moe(experts=5, top=2, ff=7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def make_config(layers, width=20, vocab=37, eps=1e-5, loop=None, embed_scale=2.0, logit_scale=0.5, softcap=8.0):
    cfg = {"architecture": "Gubanex", "embedding": {"scale": embed_scale}, "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps},
           "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if softcap:
        cfg["logit_softcap"] = softcap
    return cfg


def tensor_shapes(cfg, rank=3):
    """the rank of a layer's decays stands in no configuration: layer i gets rank + i"""
    W, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, ly in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{i}.", ly["mixer"], ly.get("mlp")
        H, d, vd = mx["heads"], mx["dim"], mx["vdim"]
        G = mx.get("kv_heads", H)
        out.update({p + "norm1": (W,), p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.v": (G * vd, W), p + "mix.o": (W, H * vd)})
        if ly["type"] == "gla":
            r = rank + i
            out.update({p + "mix.g": (H * vd, W), p + "mix.norm": (vd,), p + "mix.a1": (r, W), p + "mix.a2": (H * d, r), p + "mix.a2.b": (H * d,)})
        if mlp:
            out.update({p + "norm2": (W,), p + "mlp.router": (mlp["router"]["experts"], W)})
            for e in range(mlp["router"]["experts"]):
                q, ff = p + f"mlp.e{e}.", mlp["expert"]["ff"]
                out.update({q + "gate": (ff, W), q + "up": (ff, W), q + "down": (W, ff)})
    out.update({"final.norm": (W,), "head": (cfg["vocab"], W)})
    return out


def random_weights(cfg, seed=0, gain=1.0, rank=3):
    """name -> (bf16 bits, float64 values)"""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        last = name.split(".")[-1]
        if name == "embed":
            a = rng.standard_normal(shape)
        elif len(shape) == 2:
            a = rng.standard_normal(shape) * gain / np.sqrt(shape[1])
            if last in ("gate", "up"):
                a *= 2.0  # the router's weight, below 1, scales an expert's input
        elif last == "b":
            a = 2.0 + 1.5 * rng.standard_normal(shape)
        elif name.endswith("mix.norm"):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        else:
            a = 0.2 * rng.standard_normal(shape)  # zero-centred
        out[name] = bf16_round(np.asarray(a, np.float32))
    return out


def set_values(weights, name, vals):
    weights[name] = bf16_round(np.asarray(vals, np.float32))
