"""Small Rimidra configurations and weights for the tests.  The configurations differ in every size, in the
order of their layers and in which optional features they have: attention with windows shorter and longer
than a page and with none, with and without a query temperature, one kv head and as many as heads, values of
another size than keys; retention with full, partial and no rotation, values that are no multiple of four,
a decay of exactly 1; dense feed-forwards, mixtures that choose one, some and all of their experts, with and
without a shared expert, a layer without feed-forward; layers that use the weights of an earlier and of a
later layer; widths that are no multiple of 8."""
import copy
import json
import os

import torch


def _att(heads, kv, dim, vdim, scale, window=None, temp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m}


def _ret(dim, vdim, decay, rot=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "retention", "mixer": m}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    f = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def _layer(mixer, mlp, weights_of=None):
    e = dict(copy.deepcopy(mixer), mlp=copy.deepcopy(mlp))
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


_A0, _A1 = _ret(16, 24, (0.9, 0.97, 0.995), (8, 10000.0)), _att(4, 2, 32, 16, 0.3, window=20, temp=(0.7, 16))
RIM_A = {"architecture": "Rimidra", "vocab": 203, "width": 64, "norm": {"eps": 1e-5}, "layers": [
    _layer(_A0, _moe(5, 2, 40, 24)), _layer(_A1, _dense(48)), _layer(_att(3, 1, 24, 40, 0.35), None),
    _layer(_A0, _moe(5, 2, 40, 24), weights_of=0), _layer(_A1, _dense(48), weights_of=1)]}
# heads of 64 (bfloat16 runs the tensor-core kernels); a window that is no multiple of a page or a tile; a layer
# that uses the weights of a later one
_B1 = _att(4, 2, 64, 64, 0.2, window=100, temp=(0.4, 50))
RIM_B = {"architecture": "Rimidra", "vocab": 320, "width": 128, "norm": {"eps": 1e-6}, "layers": [
    _layer(_B1, _moe(4, 1, 72, 40), weights_of=2), _layer(_ret(32, 64, (0.95, 0.99), (32, 1000000.0)), _dense(96)),
    _layer(_B1, _moe(4, 1, 72, 40)), _layer(_ret(64, 32, (0.8, 0.98, 0.999), (64, 50000.0)), _moe(6, 3, 64))]}
# sizes that are no multiple of 8; a window shorter than a page; every expert chosen; a head that never forgets
RIM_C = {"architecture": "Rimidra", "vocab": 150, "width": 100, "norm": {"eps": 3e-6}, "layers": [
    _layer(_att(6, 2, 12, 20, 0.5, window=5, temp=(1.1, 7)), _moe(3, 3, 28, 36)),
    _layer(_ret(20, 11, (0.85, 1.0, 0.99), (6, 500.0)), None),
    _layer(_att(5, 5, 20, 12, 0.4, window=33), _dense(36)),
    _layer(_ret(9, 7, (0.93,)), _moe(7, 2, 20))]}
# the widest kernels: keys of 128, values of 64 and 160; windows of exactly four pages
_D0 = _att(6, 2, 128, 64, 0.13, window=128, temp=(0.25, 64))
RIM_D = {"architecture": "Rimidra", "vocab": 384, "width": 192, "norm": {"eps": 1e-6}, "layers": [
    _layer(_D0, _moe(6, 2, 96, 64)), _layer(_ret(128, 160, (0.97, 0.998), (96, 10000.0)), _moe(9, 2, 80, 48)),
    _layer(_att(4, 4, 64, 128, 0.2, window=70), _dense(112)), _layer(_D0, _moe(6, 2, 96, 64), weights_of=0),
    _layer(_ret(200, 36, (0.99,)), _dense(64))]}

# name -> (config, page size)
TINY = {"rim_a": (RIM_A, 16), "rim_b": (RIM_B, 8), "rim_c": (RIM_C, 8), "rim_d": (RIM_D, 32)}


def get(name):
    cfg, page = TINY[name]
    return copy.deepcopy(cfg), page


def tensor_shapes(cfg):
    """Names and shapes of a checkpoint of ``cfg``, from the design's naming rules."""
    D, s = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, lc in enumerate(cfg["layers"]):
        if lc.get("weights_of") is not None:
            continue
        p, m, f = f"l{i}.", lc["mixer"], lc["mlp"]
        s[p + "norm1"] = (D,)
        if lc["type"] == "attention":
            H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            s.update({p + "mix.q": (H * d, D), p + "mix.k": (G * d, D), p + "mix.v": (G * v, D), p + "mix.sink": (H,),
                      p + "mix.o": (D, H * v)})
        else:
            H, d, v = m["heads"], m["dim"], m["vdim"]
            s.update({p + "mix.q": (H * d, D), p + "mix.k": (H * d, D), p + "mix.v": (H * v, D), p + "mix.g": (H * v, D),
                      p + "mix.o": (D, H * v)})
        if f is None:
            continue
        if f["kind"] == "dense":
            parts = {"": f["ff"]}
        else:
            parts = {f"e{e}.": f["expert"]["ff"] for e in range(f["router"]["experts"])}
            s[p + "mlp.router"] = (f["router"]["experts"], D)
            if f.get("shared"):
                parts["shared."] = f["shared"]["ff"]
                s[p + "mlp.shared.sg"] = (1, D)
        for q, ff in parts.items():
            s.update({p + f"mlp.{q}gate": (ff, D), p + f"mlp.{q}up": (ff, D), p + f"mlp.{q}down": (D, ff)})
    s["final.norm"] = (D,)
    s["head"] = (cfg["vocab"], D)
    return s


def random_weights(cfg, seed):
    """Float32 tensors whose values are exact in bfloat16, so that the same checkpoint serves both modes.
    Matrices N(0, 1/fan_in) with a gain, routers wide enough that choices are seldom close, norm weights around
    0, sinks of the size of a large score."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith("sink"):
            t = 1.0 + torch.randn(shape, generator=g)
        elif len(shape) == 1:
            t = 0.2 * torch.randn(shape, generator=g)
        else:
            gain = 1.0 if name == "embed" else 2.0 if name.endswith(("router", "sg")) else 1.4
            t = torch.randn(shape, generator=g) * gain / (shape[1] ** 0.5 if name != "embed" else 1.0)
        w[name] = t.to(torch.bfloat16).to(torch.float32)
    return w


def as_numpy(weights):
    return {k: v.double().numpy() for k, v in weights.items()}


def model_folder(tmp, name, cfg, weights, dtype="bfloat16"):
    from gollmgo_b200.weights import save_file
    d = os.path.join(str(tmp), name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    td = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
    save_file(((k, v.to(td)) for k, v in weights.items()), os.path.join(d, "model.safetensors"), metadata={"format": "pt"})
    return d
