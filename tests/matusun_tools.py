"""Small Matusun configurations and weights for the tests.  The configurations differ in every size, in the order of
their layers, in the number of residual streams (one to five) and in which optional features they have: attention with
windows shorter and longer than a page and with none, full, partial and no rotation, one kv head and as many as heads,
values of another size than keys; selective scans with one to five taps, from 5 to 64 states, ranks and widths that are
no multiple of 8; mixtures that choose one, some and all of their experts, with and without identity experts, a shared
expert and a factor; layers without a feed-forward; loops over some layers, over all of them and none."""
import copy
import json
import math
import os

import torch


def att(heads, kv, dim, vdim, scale, window=None, rot=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m}


def scan(inner, state, rank, conv):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}}


def moe(experts, top, ff, identity=0, scale=None, shared=None):
    f = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if identity:
        f["router"]["identity"] = identity
    if scale is not None:
        f["router"]["scale"] = scale
    if shared:
        f["shared"] = {"ff": shared}
    return f


def _layer(mixer, mlp):
    return dict(copy.deepcopy(mixer), mlp=copy.deepcopy(mlp))


def _model(vocab, width, streams, eps, layers, loop=None):
    c = {"architecture": "Matusun", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


MAT_A = _model(203, 64, 2, 1e-5, [
    _layer(scan(96, 8, 5, 4), moe(5, 2, 40, 2, 1.5, 24)), _layer(att(4, 2, 32, 16, 0.3, 20, (20, 10000.0)), moe(4, 1, 48, shared=56)),
    _layer(scan(40, 16, 4, 2), None), _layer(att(3, 1, 24, 40, 0.35), moe(6, 3, 24, 1))], (1, 3, 2))
# heads of 64 with values of 64 (bfloat16 runs the tensor-core kernels); a window that is no multiple of a page or a tile
MAT_B = _model(320, 128, 4, 1e-6, [
    _layer(att(4, 2, 64, 64, 0.2, 100, (64, 50000.0)), moe(6, 2, 72, 2, 2.0, 40)), _layer(scan(128, 16, 8, 4), moe(4, 2, 64, scale=0.7)),
    _layer(scan(192, 32, 16, 4), moe(5, 2, 40, 3, shared=64))])
# sizes that are no multiple of 8; a window shorter than a page; more choices than experts with tensors
MAT_C = _model(150, 100, 3, 3e-6, [
    _layer(att(6, 2, 12, 20, 0.5, 5, (6, 500.0)), moe(2, 4, 28, 3, 1.3, 36)), _layer(scan(50, 5, 3, 5), moe(3, 3, 20)),
    _layer(att(5, 5, 20, 12, 0.4, 33, (20, 100.0)), None), _layer(scan(33, 12, 1, 3), moe(7, 2, 20, 1, 2.5))], (0, 2, 3))
# keys of 128 with values of 64; one stream; a convolution of one tap; all layers twice; windows of exactly four pages
MAT_D = _model(384, 192, 1, 1e-6, [
    _layer(att(6, 2, 128, 64, 0.13, 128, (96, 10000.0)), moe(6, 2, 96, 1, 1.2, 64)), _layer(scan(64, 64, 24, 1), moe(9, 3, 80, 2)),
    _layer(scan(72, 40, 12, 3), moe(4, 1, 48, shared=32))], (0, 3, 2))
# five streams, keys and values of 128 without a window, a layer that is repeated alone
MAT_E = _model(256, 136, 5, 1e-5, [
    _layer(att(2, 1, 128, 128, 0.1, None, (128, 10000.0)), moe(5, 2, 64, 1, 1.7, 40)), _layer(scan(160, 16, 8, 4), moe(4, 2, 56, 1)),
    _layer(att(4, 4, 64, 128, 0.2, 70, (32, 1000.0)), moe(3, 2, 40))], (1, 2, 3))

# name -> (config, page size)
TINY = {"mat_a": (MAT_A, 16), "mat_b": (MAT_B, 8), "mat_c": (MAT_C, 8), "mat_d": (MAT_D, 32), "mat_e": (MAT_E, 16)}


def get(name):
    cfg, page = TINY[name]
    return copy.deepcopy(cfg), page


def tensor_shapes(cfg):
    """Names and shapes of a checkpoint of ``cfg``, from the design's naming rules."""
    D, S, s = cfg["width"], cfg["streams"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, lc in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", lc["mixer"], lc["mlp"]
        for q in (1, 2) if f is not None else (1,):
            s.update({p + f"norm{q}": (D,), p + f"hc{q}.in": (S,), p + f"hc{q}.out": (S,), p + f"hc{q}.mix": (S, S)})
        if lc["type"] == "attention":
            H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            s.update({p + "mix.q": (H * d, D), p + "mix.k": (G * d, D), p + "mix.v": (G * v, D), p + "mix.q.norm": (H * d,),
                      p + "mix.k.norm": (G * d,), p + "mix.o": (D, H * v)})
        else:
            I, N, R, t = m["inner"], m["state"], m["dt_rank"], m["conv"]
            s.update({p + "mix.in": (2 * I, D), p + "mix.conv": (I, t), p + "mix.conv.b": (I,), p + "mix.x": (R + 2 * N, I),
                      p + "mix.dt": (I, R), p + "mix.dt.b": (I,), p + "mix.A_log": (I, N), p + "mix.D": (I,), p + "mix.o": (D, I)})
        if f is None:
            continue
        n = f["router"]["experts"]
        s.update({p + "mlp.router": (n + f["router"].get("identity", 0), D), p + "mlp.correction": (n + f["router"].get("identity", 0),)})
        parts = {f"e{e}.": f["expert"]["ff"] for e in range(n)}
        if f.get("shared"):
            parts["shared."] = f["shared"]["ff"]
        for q, ff in parts.items():
            s.update({p + f"mlp.{q}up": (ff, D), p + f"mlp.{q}down": (D, ff)})
    s["final.norm"] = (D,)
    return s


def random_tensor(name, shape, g):
    """Values of a size that lets every term be felt: decays from fast to slow, step sizes around e^-2.5, streams that are
    mixed but neither die out nor explode, corrections of the size of the differences between scores."""
    r = lambda *s: torch.randn(*s, generator=g)
    last = name.rsplit(".", 1)[-1]
    if name.endswith(".mix") and len(shape) == 2 and shape[0] == shape[1] and ".hc" in name:
        return torch.eye(shape[0]) + 0.2 * r(*shape) / shape[0] ** 0.5
    if ".hc" in name:
        return (1.0 / shape[0] if last == "in" else 0.5) * (1.0 + 0.4 * r(*shape))
    if last == "A_log":
        return 1.2 * r(*shape)
    if name.endswith("dt.b"):
        return -2.5 + 0.7 * r(*shape)
    if name.endswith("conv.b"):
        return 0.3 * r(*shape)
    if last == "D":
        return 1.0 + 0.4 * r(*shape)
    if last == "correction":
        return 0.1 * r(*shape)
    if last == "conv":
        return r(*shape) / shape[1] ** 0.5
    if last in ("norm", "norm1", "norm2"):
        return 1.0 + 0.2 * r(*shape)
    if name == "embed":
        return r(*shape)
    gain = {"router": 2.0, "up": 1.0, "down": 1.0, "x": 0.6, "dt": 1.0}.get(last, 1.4)
    return r(*shape) * gain / math.sqrt(shape[1])


def random_weights(cfg, seed):
    """Float32 tensors whose values are exact in bfloat16, so that the same checkpoint serves both modes."""
    g = torch.Generator().manual_seed(seed)
    return {name: random_tensor(name, shape, g).to(torch.bfloat16).to(torch.float32) for name, shape in tensor_shapes(cfg).items()}


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
