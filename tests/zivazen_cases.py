"""Small Zivazen configurations and random weights for the tests: sizes that are no powers of two, key and value sizes that
differ, grouped heads and one per head, one head, chunks and windows shorter than a page, longer than several and none,
rotation of part of a head, of none of it, with and without stretched wavelengths, layers that mix values and others that
do not, convolutions of one tap and more, states that fill no 16-byte pieces, grouped B and C, one norm part and several,
experts in groups and in none, groups of one expert, mixtures with and without a shared expert, layers without a
feed-forward, dense and mixed feed-forwards behind either mixer, output scales of one and others."""
from __future__ import annotations

import math

import torch


def attention(heads=4, kv_heads=2, dim=24, vdim=16, size=40, rot=12, scale=0.2, v_mix=True, scaling=(3.0, 1.0, 5.0, 90),
              base=5000.0, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if size:
        mixer["mask"] = {"size": size}
    if rot is not None:
        mixer["rot"] = {"base": base, "dims": rot}
        if scaling:
            mixer["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def parallel(heads=4, kv_heads=2, dim=16, vdim=16, size=30, rot=8, scale=0.25, ssm=(4, 12, 10, 2, 3, 2), left_scale=0.7,
             right_scale=1.2, base=800.0, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        left["mask"] = {"size": size}
    if rot is not None:
        left["rot"] = {"base": base, "dims": rot}
    right = dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), ssm))
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale,
                                          "right_scale": right_scale}, "mlp": mlp}


def dense(ff=44):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=3, ff=20, groups=(4, 2), scale=1.7, shared=36):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers, vocab=211, width=96, eps=1e-5) -> dict:
    return {"architecture": "Zivazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def _mixed():
    return config([attention(v_mix=False, mlp=dense()), parallel(mlp=moe()), attention(mlp=moe(shared=0)),
                   attention(heads=2, size=17, rot=None, mlp=dense(30)),
                   parallel(heads=3, kv_heads=1, dim=10, vdim=14, size=9, rot=4, ssm=(6, 7, 9, 3, 1, 1), left_scale=1.0,
                            mlp=None),
                   attention(heads=6, size=0, rot=24, scaling=None, mlp=None)])


def _tiled():
    return config([parallel(heads=4, kv_heads=1, dim=64, vdim=64, size=100, rot=64, scale=0.12,
                            ssm=(6, 32, 32, 2, 4, 3), mlp=dense(64)),
                   attention(heads=4, kv_heads=1, dim=64, vdim=64, size=300, rot=32, scale=0.12, mlp=moe(16, 2, 32, (4, 1))),
                   parallel(heads=3, kv_heads=3, dim=32, vdim=32, size=600, rot=16, scale=0.2, ssm=(2, 64, 64, 1, 2, 1),
                            left_scale=0.4, right_scale=0.9, mlp=moe(32, 5, 24, None, 0.8, 0)),
                   attention(heads=8, kv_heads=1, dim=48, vdim=64, size=64, rot=48, scale=0.15, mlp=dense(40))],
                  width=128, vocab=157)


def _narrow():
    return config([attention(heads=1, kv_heads=1, dim=10, vdim=6, size=5, rot=10, scale=0.3, scaling=(8.0, 1.0, 4.0, 40),
                             base=300.0, mlp=moe(6, 1, 9, (6, 4), 1.0, 11)),
                   parallel(heads=5, kv_heads=5, dim=4, vdim=7, size=130, rot=0, scale=0.5, ssm=(3, 5, 6, 1, 5, 3),
                            mlp=moe(5, 2, 12, None, 2.0, 8)),
                   attention(heads=3, kv_heads=1, dim=8, vdim=6, size=129, rot=2, scale=0.4, scaling=None, mlp=dense(21))],
                  width=64, vocab=97, eps=2e-2)


CASES = {
    # both mixers with either feed-forward and none, some layers that mix values among others that do not
    "mixed": _mixed,
    # sizes that tile for the tensor cores, a window over more than nine pages, chunks that end within pages and at them
    "tiled": _tiled,
    # one head, chunks of five, sizes that fill no 16-byte pieces, groups of one expert
    "narrow": _narrow,
}


def random_weights(config_dict: dict, seed: int = 0) -> dict:
    """bfloat16 tensors by checkpoint name, scaled so that activations stay of order one through the layers."""
    g = torch.Generator().manual_seed(seed)
    width = config_dict["width"]
    t: dict[str, torch.Tensor] = {}

    def matrix(name, rows, cols, gain=1.0):
        t[name] = (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(torch.bfloat16)

    def vector(name, size, mean=1.0, spread=0.2):
        t[name] = (mean + spread * torch.randn(size, generator=g)).to(torch.bfloat16)

    matrix("embed", config_dict["vocab"], width, gain=2.0)
    matrix("head", config_dict["vocab"], width)
    vector("embed.norm", width)
    vector("final.norm", width)
    for i, layer in enumerate(config_dict["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        vector(p + "norm1", width)
        if layer["type"] == "attention":
            attention_weights(matrix, vector, p + "mix.", width, m)
            if m["v_mix"]:
                t[p + "mix.vmix"] = torch.tensor(0.3 + 0.1 * i).to(torch.bfloat16)
        else:
            left = m["left"]
            for name, rows in (("q", left["heads"] * left["dim"]), ("k", left["kv_heads"] * left["dim"]),
                               ("v", left["kv_heads"] * left["vdim"])):
                matrix(p + f"mix.left.{name}", rows, width, 1.5)
            matrix(p + "mix.left.o", width, left["heads"] * left["vdim"])
            state_space_weights(matrix, vector, p + "mix.right.", width, m["right"])
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            for name, rows in (("gate", mlp["ff"]), ("up", mlp["ff"])):
                matrix(p + f"mlp.{name}", rows, width, 1.5)
                vector(p + f"mlp.{name}.b", rows, 0.0, 0.5)
            matrix(p + "mlp.down", width, mlp["ff"])
            vector(p + "mlp.down.b", width, 0.0, 0.2)
            continue
        matrix(p + "mlp.router", mlp["router"]["experts"], width, 1.5)
        vector(p + "mlp.correction", mlp["router"]["experts"], -1.0, 0.6)
        for e in range(mlp["router"]["experts"]):
            matrix(p + f"mlp.e{e}.up", mlp["expert"]["ff"], width, 1.0)
            matrix(p + f"mlp.e{e}.down", width, mlp["expert"]["ff"], 0.7)
        if mlp.get("shared"):
            matrix(p + "mlp.shared.up", mlp["shared"]["ff"], width, 1.0)
            matrix(p + "mlp.shared.down", width, mlp["shared"]["ff"], 0.5)
    return t


def attention_weights(matrix, vector, p, width, m, gain=1.5):
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    for name, rows in (("q", heads * dim), ("k", groups * dim), ("v", groups * vdim)):
        matrix(p + name, rows, width, gain)
        vector(p + name + ".b", rows, 0.0, 0.5)
    vector(p + "q.norm", dim, 1.3, 0.3)
    vector(p + "k.norm", dim, 1.3, 0.3)
    matrix(p + "o", width, heads * vdim)
    vector(p + "o.b", width, 0.0, 0.2)


def state_space_weights(matrix, vector, p, width, m, a_log=(-1.0, 1.2), dt_bias=(-1.5, 1.0)):
    inner = m["heads"] * m["vdim"]
    channels = inner + 2 * m["groups"] * m["state"]
    matrix(p + "in", inner + channels + m["heads"], width, 1.5)
    vector(p + "conv", channels * m["conv"], 0.1, 0.6)
    vector(p + "conv.b", channels, 0.0, 0.3)
    vector(p + "dt_bias", m["heads"], *dt_bias)
    vector(p + "A_log", m["heads"], *a_log)
    vector(p + "D", m["heads"], 0.8, 0.4)
    vector(p + "norm", inner, 1.1, 0.3)
    matrix(p + "o", width, inner)


def shaped(config_dict: dict, tensors: dict) -> dict:
    """The taps, drawn flat, as [channels, taps]."""
    for i, layer in enumerate(config_dict["layers"]):
        name = f"l{i}.mix.right.conv"
        if name in tensors:
            tensors[name] = tensors[name].reshape(-1, layer["mixer"]["right"]["conv"])
    return tensors


def make_weights(config_dict: dict, seed: int = 0) -> dict:
    return shaped(config_dict, random_weights(config_dict, seed))


def make_engine(config_dict: dict, tensors: dict, dtype: str, max_tokens: int = 2048, **kwargs):
    from etalii.dllm_b200.config.registry import config_from_dict
    from etalii.dllm_b200.engine.engine import Engine

    kwargs.setdefault("max_length", 1024)
    return Engine(config_from_dict(config_dict), tensors, dtype=dtype, device="cuda:0", max_tokens=max_tokens, **kwargs)


def tokens_for(config_dict: dict, lengths, seed: int = 5):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, config_dict["vocab"], (n,), generator=g).tolist() for n in lengths]


def as_numpy(tensors: dict) -> dict:
    return {name: value.to(torch.float64).numpy() for name, value in tensors.items()}
