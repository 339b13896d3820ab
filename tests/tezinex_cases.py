"""Small Tezinex configurations and random weights for the tests: sizes that are no powers of two, key and value sizes that
differ, fewer key/value heads than query heads and as many, one head and several, windows shorter than a page and longer
than eight, first positions kept within a page, across a page border, and none, no window at all, layers that borrow keys
with a wider and with a narrower window than the owner's, convolutions of one tap and more, low-rank projections of
unequal and odd inner sizes, layers without a feed-forward (the first among them or not), caps and none."""
from __future__ import annotations

import math

import torch


def attention(heads=4, kv_heads=2, dim=24, vdim=16, size=40, keep_first=3, scale=0.2, softcap=9.0, ff=48, kv_from=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        mixer["mask"] = {"size": size, "keep_first": keep_first}
    if softcap:
        mixer["softcap"] = softcap
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=3, ff=40):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}
    return {"type": "channel_delta", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, vocab=211, width=96, eps=1e-5, residual_mult=0.6, logit_softcap=11.0) -> dict:
    out = {"architecture": "Tezinex", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "residual_mult": residual_mult, "layers": layers}
    if logit_softcap:
        out["logit_softcap"] = logit_softcap
    return out


def _mixed():
    return config([attention(), delta(ff=0), attention(size=90, keep_first=70, kv_from=0, softcap=0, ff=0), delta(),
                   attention(heads=6, kv_heads=6, dim=8, vdim=12, size=0, ff=0),
                   attention(heads=2, size=9, keep_first=0, kv_from=0)])


def _tiled():
    return config([delta(heads=6, kv_heads=3, dim=32, vdim=16, conv=4, ff=0),
                   attention(heads=4, kv_heads=1, dim=64, vdim=64, size=600, keep_first=70, scale=0.12, softcap=20.0, ff=64),
                   attention(heads=4, kv_heads=1, dim=64, vdim=64, size=100, keep_first=64, scale=0.12, softcap=5.0, ff=0,
                             kv_from=1),
                   delta(heads=2, kv_heads=2, dim=64, vdim=48, conv=2, ff=64),
                   attention(heads=3, kv_heads=3, dim=40, vdim=72, size=64, keep_first=0, scale=0.15, ff=32)],
                  width=128, vocab=157, residual_mult=0.35, logit_softcap=0)


def _narrow():
    return config([attention(heads=1, kv_heads=1, dim=10, vdim=6, size=5, keep_first=1, scale=0.3, softcap=4.0, ff=20),
                   delta(heads=3, kv_heads=1, dim=6, vdim=10, conv=1, ff=0),
                   attention(heads=5, kv_heads=5, dim=4, vdim=7, size=130, keep_first=2, scale=0.5, softcap=0, ff=0)],
                  width=64, vocab=97, eps=2e-2, residual_mult=1.0, logit_softcap=6.0)


CASES = {
    # both mixers, grouped heads and one per head, borrowed keys under a wider and a narrower window, no window
    "mixed": _mixed,
    # sizes that tile for the tensor cores, a window over more than nine pages, kept positions across a page border
    "tiled": _tiled,
    # one head, a window of five, sizes that fill no 16-byte pieces, one tap, a multiplier of one
    "narrow": _narrow,
}


def ranks(index: int, mixer: dict) -> tuple[int, int]:
    """Inner sizes of a layer's two low-rank projections: whatever the checkpoint has."""
    return 5 + 3 * index, 11 + index


def random_weights(config_dict: dict, seed: int = 0) -> dict:
    """bfloat16 tensors by checkpoint name, scaled so that activations stay of order one through the layers."""
    g = torch.Generator().manual_seed(seed)
    width = config_dict["width"]
    t: dict[str, torch.Tensor] = {}

    def matrix(name, rows, cols, gain=1.0):
        t[name] = (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(torch.bfloat16)

    def vector(name, size, mean=1.0, spread=0.2):
        t[name] = (mean + spread * torch.randn(size, generator=g)).to(torch.bfloat16)

    matrix("embed", config_dict["vocab"], width, gain=math.sqrt(width))
    vector("final.norm", width, 0.0, 0.3)
    for i, layer in enumerate(config_dict["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for name in ("norm1", "norm1b", *(("norm2", "norm2b") if layer["mlp"] else ())):
            vector(p + name, width, 0.0, 0.3)
        vector(p + "dwa", i + 2, 0.0, 0.4)
        t[p + "dwa"][-1] += 1.0
        if layer["type"] == "channel_delta":
            a_rank, g_rank = ranks(i, m)
            for name, rows in (("q", groups * dim), ("k", groups * dim), ("v", heads * vdim)):
                matrix(p + f"mix.{name}", rows, width, 1.5)
                t[p + f"mix.{name}.conv"] = (torch.randn(rows, m["conv"], generator=g) * 0.6).to(torch.bfloat16)
            matrix(p + "mix.b", heads, width, 1.5)
            vector(p + "mix.A_log", heads, -1.0, 1.2)
            vector(p + "mix.norm", vdim, 1.1, 0.3)
            matrix(p + "mix.a1", a_rank, width, 1.5)
            matrix(p + "mix.a2", heads * dim, a_rank, 1.5)
            vector(p + "mix.dt_bias", heads * dim, -1.5, 1.5)
            matrix(p + "mix.g1", g_rank, width, 1.5)
            matrix(p + "mix.g2", heads * vdim, g_rank, 1.5)
        else:
            named = [("q", heads * dim)]
            if m.get("kv_from") is None:
                named += [("k", groups * dim), ("v", groups * vdim)]
            for name, rows in named:
                matrix(p + f"mix.{name}", rows, width, 2.0)
                vector(p + f"mix.{name}.b", rows, 0.0, 0.5)
            vector(p + "mix.sink", heads, 1.0, 1.0)
        matrix(p + "mix.o", width, heads * vdim)
        if layer["mlp"]:
            matrix(p + "mlp.gate", layer["mlp"]["ff"], width, 1.5)
            matrix(p + "mlp.up", layer["mlp"]["ff"], width, 1.5)
            matrix(p + "mlp.down", width, layer["mlp"]["ff"])
    return t


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
