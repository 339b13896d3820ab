"""Tezinex on the GPU against the plain implementation (tests/plain_tezinex.py): every mechanism alone through its part or
kernel, then whole models through the engine's step function, decode graph and generation loop, cut and batched in
every way a server would."""
import numpy as np
import pytest
import torch

import plain_tezinex as P
import tezinex_cases as C
from helpers import TOL, host, rel_error
from test_revupel_gpu import PartHarness, _bf16, _feed, _inputs, _mixer_call, _runtime, _vector

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [("float32", torch.float32), ("bfloat16", torch.bfloat16)]
PART_TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}
SHARP_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.14}
"""For the tests whose weights make one score stand out: such sharp maps amplify the rounding of bfloat16 rows, and
what the tests decide (a key seen or not) moves the output by more than 0.2."""
SCHEDULE = [[(0, 70), (1, 2), (2, 17)], [(0, 1), (1, 1), (2, 1)], [(0, 1), (1, 1), (2, 1)], [(0, 2), (2, 65)],
            [(0, 1), (2, 1)], [(2, 1)]]


def _np(weights, renames=()):
    out = {}
    for name, value in weights.items():
        for old, new in renames:
            name = name.replace(old, new)
        out[name] = value.to(torch.float64).numpy()
    return out


# ---- positions, norms, caps and the stream ------------------------------------------------------------------------------


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("width", [8, 96, 520])
def test_embedding_with_a_sinusoid(name, dtype, width):
    """First positions, page borders and positions far out: every angle right to float32 whatever the position."""
    from etalii.dllm_b200.parts import PartSpec, build_part

    rt = _runtime(dtype)
    g = torch.Generator().manual_seed(width)
    part = build_part("embedding", PartSpec("token_embedding", {
        "vocab_size": 50, "hidden_size": width, "position": PartSpec("sinusoidal", {"hidden_size": width})}))
    table = _bf16(g, 50, width, 3.0)
    part.bind({"weight": table}, rt)
    positions = [0, 1, 2, 63, 64, 65, 999, 4096, 20011, 32767]
    tokens = [7, 7, 0, 49, 3, 7, 21, 21, 5, 11]
    ints = lambda values: torch.tensor(values, dtype=torch.int32, device=DEV)  # noqa: E731
    got = host(part.forward(ints(tokens), len(tokens), rt, positions=ints(positions)))
    want = table.double().numpy()[tokens] + P.sinusoid(positions, width)
    assert np.abs(got - want).max() < 2e-6


def test_capped_rows():
    from etalii.dllm_b200.kernels import ops

    x = torch.randn(5, 333, generator=torch.Generator().manual_seed(0)) * 20
    rows = x.to(DEV).contiguous()
    ops.softcap_rows(rows, 7.5)
    assert np.abs(host(rows) - P.cap(x.double().numpy(), 7.5)).max() < 2e-6


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 40, 200])
@pytest.mark.parametrize("width", [8, 96, 520, 2048, 8192])
@pytest.mark.parametrize("form", ["sum only", "next norm", "first layer", "first layer at once", "later", "last"])
def test_stream_update(name, dtype, rows, width, form):
    """Behind a sublayer: the output's norm and the residual sum, the weighted sum over earlier results (none, the first
    layer's in one kernel and in two, many), what is kept for later sums, and the norm in front of the next reader."""
    from etalii.dllm_b200.kernels import ops

    g = torch.Generator().manual_seed(rows + width)
    layers = 9
    index = {"later": 5, "last": 8}.get(form, 0)
    x, y = torch.randn(rows, width, generator=g), 3 * torch.randn(rows, width, generator=g)
    results = torch.randn(layers, rows, width, generator=g)
    w, next_w = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    c = torch.randn(index + 2, generator=g)
    mixes = form not in ("sum only", "next norm")
    dev = lambda t: t.to(DEV).contiguous()  # noqa: E731
    xd, rd = dev(x), dev(results)
    normed = torch.empty(rows, width, dtype=dtype, device=DEV) if form != "sum only" else None
    at_once = form == "first layer at once"
    ops.stream_update(xd, dev(y), dev(w), 1e-3, first_result=rd[0] if at_once or form == "next norm" else None,
                      results=rd if mixes else None, index=index, coefficients=dev(c) if mixes else None,
                      first_from_stream=at_once, next_weight=dev(next_w) if normed is not None else None,
                      next_eps=1e-2, normed=normed)
    n64 = lambda t: t.double().numpy()  # noqa: E731
    v = n64(x) + P.rms(n64(y), 1e-3) * n64(w)
    earlier = [n64(r) for r in results[:index + 1]]
    if at_once:
        earlier[0] = n64(x)
    want = P.depth_average(n64(c), [*earlier, v]) if mixes else v
    assert rel_error(host(xd), want) < 2e-6
    if at_once or form == "next norm":
        assert torch.equal(rd[0].cpu(), x)  # the stream as it was, bit by bit
    if mixes and index + 1 < layers:
        assert rel_error(host(rd[index + 1]), v) < 2e-6
        assert torch.equal(rd[index + 2].cpu(), results[index + 2])
    if form in ("later", "last"):
        assert torch.equal(rd[:index + 1].cpu(), results[:index + 1])
    if normed is not None:
        assert rel_error(host(normed), P.rms(want, 1e-2) * n64(next_w)) < (2e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("rows,width,ff", [(1, 72, 44), (20, 96, 50), (150, 64, 333), (70, 128, 40)])
def test_feed_forward_of_any_inner_size(name, dtype, rows, width, ff):
    from etalii.dllm_b200.kernels import ops
    from etalii.dllm_b200.parts import PartSpec, build_part

    rt = _runtime(dtype)
    g = torch.Generator().manual_seed(rows + ff)
    part = build_part("feed_forward", PartSpec("swiglu", {"hidden_size": width, "intermediate_size": ff, "pad": True}))
    weights = {"gate": _bf16(g, ff, width, 2.5), "up": _bf16(g, ff, width, 1.5), "down": _bf16(g, width, ff)}
    part.bind(weights, rt)
    h = torch.randn(rows, width, generator=g).to(dtype).float()
    out = torch.full((rows, width), 7.0, device=DEV)
    part.forward(h.to(DEV).to(dtype), out, None, rt, epilogue=ops.EPI_STORE_F32)
    assert rel_error(host(out), P.feed_forward(_np(weights), h.double().numpy())) <= PART_TOL[dtype]


# ---- the delta rule by channels -----------------------------------------------------------------------------------------


def _delta(width, m, eps=1e-5):
    from etalii.dllm_b200.parts import PartSpec, build_part

    return build_part("mixer", PartSpec("channel_delta_rule", {
        "hidden_size": width, "heads": m["heads"], "qk_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
        "conv": m["conv"], "eps": eps}))


def _delta_weights(g, width, m, a_rank=7, g_rank=12, a_log=(-1.0, 1.2), bias=(-1.5, 1.5)):
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    qk, values = m["kv_heads"] * dim, heads * vdim
    taps = lambda rows: (0.6 * torch.randn(rows, m["conv"], generator=g)).to(torch.bfloat16)  # noqa: E731
    return {"q": _bf16(g, qk, width, 1.5), "k": _bf16(g, qk, width, 1.5), "v": _bf16(g, values, width, 1.5),
            "q_conv": taps(qk), "k_conv": taps(qk), "v_conv": taps(values), "b": _bf16(g, heads, width, 1.5),
            "A_log": _vector(g, heads, *a_log), "dt_bias": _vector(g, heads * dim, *bias),
            "a1": _bf16(g, a_rank, width, 1.5), "a2": _bf16(g, heads * dim, a_rank, 1.5),
            "g1": _bf16(g, g_rank, width, 1.5), "g2": _bf16(g, values, g_rank, 1.5), "norm": _vector(g, vdim, 1.1, 0.3),
            "o": _bf16(g, width, values)}


def _plain_delta(w, m, h, eps=1e-5):
    names = _np(w, (("_conv", ".conv"),))
    return P.channel_delta(names, m, h.double().numpy(), None, eps)[0]


def _m(heads, kv_heads, dim, vdim, conv):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


DELTA_SHAPES = {
    "grouped": _m(4, 2, 12, 20, 3),
    "one_head": _m(1, 1, 6, 10, 1),
    "odd": _m(3, 3, 9, 7, 2),
    "tiles": _m(8, 2, 32, 32, 4),
    "wide": _m(3, 1, 72, 40, 4),
    "widest": _m(2, 2, 256, 24, 5),
    "real": _m(2, 2, 128, 128, 4),
    "many_heads": _m(48, 16, 16, 16, 3),
}


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("shape", sorted(DELTA_SHAPES))
def test_channel_delta_part_in_pieces(name, dtype, shape):
    """Three sequences fed as a server would: a long portion, portions of two tokens, single tokens beside neighbours, a
    sequence that ends early; against the plain mixer on each whole sequence."""
    rt = _runtime(dtype)
    m, width = DELTA_SHAPES[shape], 72
    part = _delta(width, m)
    g = torch.Generator().manual_seed(len(shape))
    weights = _delta_weights(g, width, m, a_rank=5 + m["heads"], g_rank=16 - m["heads"] % 9)
    part.bind(weights, rt)
    sequences = _inputs(dtype, width, 3)
    got = _feed(PartHarness(part.cache_need(), dtype, 3), _mixer_call(part, rt), sequences, SCHEDULE, width)
    for rows, h in zip(got, sequences):
        assert rel_error(rows, _plain_delta(weights, m, h)) <= PART_TOL[dtype]


@pytest.mark.parametrize("name,dtype", DTYPES)
def test_every_key_channel_shrinks_by_its_own_decay(name, dtype):
    """Decays from 0.02 to nearly 1 inside each head: the output differs from one decay per head (their mean), from no
    decay, and from none of the state surviving, by far more than the tolerance."""
    rt = _runtime(dtype)
    m, width = _m(3, 1, 24, 16, 2), 64
    part = _delta(width, m)
    g = torch.Generator().manual_seed(4)
    weights = _delta_weights(g, width, m, a_log=(0.0, 0.1), bias=(-2.0, 3.0))
    part.bind(weights, rt)
    h = _inputs(dtype, width, 8, [120])[0]
    schedule = [[(0, 60)]] + [[(0, 1)]] * 60
    got = _feed(PartHarness(part.cache_need(), dtype, 1), _mixer_call(part, rt), [h], schedule, width)[0]
    want = _plain_delta(weights, m, h)
    assert rel_error(got, want) <= PART_TOL[dtype]
    decays = P.channel_decay(_np(weights), m, h.double().numpy())
    assert decays.min() < 0.02 and decays.max() > 0.99  # the test's premises
    exact = P.channel_decay
    for other in (lambda *a: np.broadcast_to(decays.mean(axis=2, keepdims=True), decays.shape),
                  lambda *a: np.ones_like(decays), lambda *a: np.zeros_like(decays)):
        try:
            P.channel_decay = other
            assert rel_error(_plain_delta(weights, m, h), want) > 0.15
        finally:
            P.channel_decay = exact


@pytest.mark.parametrize("name,dtype", DTYPES)
def test_a_state_is_carried_far_and_not_into_the_slots_next_sequence(name, dtype):
    """Decays next to 1: what the first tokens wrote is still read after hundreds of tokens, through portions and single
    tokens; a new sequence in the same slot starts from zero (state and the convolution's history)."""
    rt = _runtime(dtype)
    m, width = _m(2, 2, 64, 16, 4), 64
    part = _delta(width, m)
    g = torch.Generator().manual_seed(5)
    weights = _delta_weights(g, width, m, a_log=(-7.0, 0.1), bias=(-3.0, 0.3))
    weights["b"] = torch.zeros_like(weights["b"])
    part.bind(weights, rt)
    harness = PartHarness(part.cache_need(), dtype, 1)
    first, second = _inputs(dtype, width, 9, [400, 30])
    got = _feed(harness, _mixer_call(part, rt), [first], [[(0, 250)], [(0, 2)], [(0, 98)]] + [[(0, 1)]] * 50, width)[0]
    want = _plain_delta(weights, m, first)
    assert rel_error(got, want) <= PART_TOL[dtype]
    late = _plain_delta(weights, m, first[60:])[-1]
    assert rel_error(late, want[-1]) > (0.05 if dtype == torch.bfloat16 else 0.01)  # the premise: it reaches that far
    harness.again(0)
    again = _feed(harness, _mixer_call(part, rt), [second], [[(0, 1)]] * 3 + [[(0, 27)]], width)[0]
    assert rel_error(again, _plain_delta(weights, m, second)) <= PART_TOL[dtype]


# ---- attention with capped scores, a sink and kept first positions --------------------------------------------------------


def _shape(heads, kv_heads, dim, vdim, size, keep_first, scale=0.2, softcap=9.0):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if size:
        m["mask"] = dict(size=size, keep_first=keep_first)
    if softcap:
        m["softcap"] = softcap
    return m


def _attention(width, m, **more):
    from etalii.dllm_b200.parts import PartSpec, build_part

    mask = m.get("mask")
    return build_part("mixer", PartSpec("sink_attention", dict({
        "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "dim": m["dim"],
        "vdim": m["vdim"], "scale": m["scale"], "softcap": m.get("softcap") or 0.0,
        "window": mask["size"] if mask else None, "keep_first": mask["keep_first"] if mask else 0, "biases": True,
        "sink": True}, **more)))


def _attention_weights(g, width, m, sink=(1.0, 1.0), gain=2.0):
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": _bf16(g, heads * dim, width, gain), "q_bias": _vector(g, heads * dim, 0.0, 0.5),
            "k": _bf16(g, groups * dim, width, gain), "k_bias": _vector(g, groups * dim, 0.0, 0.5),
            "v": _bf16(g, groups * vdim, width, 1.5), "v_bias": _vector(g, groups * vdim, 0.0, 0.5),
            "sink": _vector(g, heads, *sink), "o": _bf16(g, width, heads * vdim)}


_RENAMES = (("_bias", ".b"),)


def _plain_attention(w, m, h):
    return P.attention(_np(w, _RENAMES), m, h.double().numpy(), None)[0]


ATTENTION_SHAPES = {
    "grouped": _shape(4, 2, 24, 16, 40, 3),
    "one_head": _shape(1, 1, 10, 6, 5, 1, scale=0.3),
    "unequal": _shape(5, 1, 40, 72, 50, 20, scale=0.15),
    "wider_keys": _shape(6, 3, 112, 8, 30, 70, scale=0.1),
    "squares": _shape(4, 1, 64, 64, 33, 31, scale=0.12),
    "heads_of_128": _shape(2, 1, 128, 128, 64, 2, scale=0.08, softcap=2.0),
    "nothing_kept": _shape(6, 6, 8, 12, 70, 0),
    "no_window": _shape(3, 3, 48, 48, 0, 0, scale=0.15, softcap=30.0),
    "no_cap": _shape(3, 1, 20, 24, 500, 0, scale=0.2, softcap=0),
    "kept_beyond_the_window": _shape(2, 2, 64, 64, 16, 100, scale=0.12),
    "many_heads": _shape(40, 2, 16, 40, 33, 31),
    "beyond_tiles": _shape(2, 1, 136, 200, 60, 9, scale=0.1),
}


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("shape", sorted(ATTENTION_SHAPES))
def test_attention_part_in_pieces(name, dtype, shape):
    rt = _runtime(dtype)
    m, width = ATTENTION_SHAPES[shape], 72
    part = _attention(width, m)
    g = torch.Generator().manual_seed(len(shape))
    weights = _attention_weights(g, width, m)
    part.bind(weights, rt)
    sequences = _inputs(dtype, width, 3)
    got = _feed(PartHarness(part.cache_need(), dtype, 3), _mixer_call(part, rt), sequences, SCHEDULE, width)
    for rows, h in zip(got, sequences):
        assert rel_error(rows, _plain_attention(weights, m, h)) <= PART_TOL[dtype]


def _attend_by(monkeypatch, kernel, shape=-1):
    """Every step of the part runs through one kernel, whatever the part would choose (None: as it chooses)."""
    from etalii.dllm_b200.kernels import ops

    general, prefill, tcgen05, decode = (ops.sink_attention, ops.sink_attention_prefill, ops.sink_attention_tcgen05,
                                         ops.sink_attention_decode)

    def run(*args):
        batch = args[-1]
        if kernel == "general":
            general(*args, split=False)
        elif kernel == "split":
            general(*args, split=True)
        elif kernel == "decode" and batch.is_decode:
            decode(*args, shape=shape)
        elif kernel == "tcgen05" and not batch.is_decode:
            tcgen05(*args)
        else:
            (decode if batch.is_decode else prefill)(*args)

    for name in ("sink_attention_prefill", "sink_attention_tcgen05", "sink_attention_decode"):
        monkeypatch.setattr(ops, name, run)


KERNELS = [("general", -1), ("split", -1), ("prefill", -1), ("tcgen05", -1), *(("decode", s) for s in range(5))]


@pytest.mark.parametrize("kernel,launch", KERNELS)
@pytest.mark.parametrize("dim", [64, 128])
@pytest.mark.parametrize("size,keep_first,softcap", [(100, 20, 3.0), (300, 130, 40.0), (0, 0, 0), (64, 64, 1.0)])
def test_every_kernel_gives_the_same_attention(monkeypatch, kernel, launch, dim, size, keep_first, softcap):
    """The general kernel in both forms, the mma.sync tiles, the tcgen05 tiles and the cluster kernel in all its launch
    shapes: prompts over several pages, portions, single tokens; scores under the cap's bend and far beyond it."""
    dtype, width = torch.bfloat16, 64
    rt = _runtime(dtype)
    m = _shape(6, 2, dim, dim, size, keep_first, scale=0.8 / dim ** 0.5, softcap=softcap)
    part = _attention(width, m)
    g = torch.Generator().manual_seed(dim + size)
    weights = _attention_weights(g, width, m)
    part.bind(weights, rt)
    _attend_by(monkeypatch, kernel, launch)
    sequences = _inputs(dtype, width, 6, [460, 33, 150])
    schedule = [[(0, 300), (1, 1), (2, 129)], [(0, 1), (1, 1), (2, 1)], [(0, 140), (1, 30)]]
    schedule += [[(0, 1), (2, 1)]] * 19 + [[(1, 1), (2, 1)]]
    got = _feed(PartHarness(part.cache_need(), dtype, 3), _mixer_call(part, rt), sequences, schedule, width)
    for rows, h in zip(got, sequences):
        assert rel_error(rows, _plain_attention(weights, m, h)) <= PART_TOL[dtype]


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("dim", [24, 64])
@pytest.mark.parametrize("sink", [-30.0, 0.0, 4.0, 30.0])
def test_a_sink_takes_its_share_and_gives_nothing(name, dtype, dim, sink):
    """A sink far below every score changes nothing, one far above leaves next to nothing for the keys, and between the
    two it takes exactly its share: in a prompt, in portions and in tokens decoded alone, at the first token too, whose
    only key is itself. It is not capped: a sink above the cap wins over every key."""
    rt = _runtime(dtype)
    m, width = _shape(5, 5, dim, dim, 90, 3, scale=0.3, softcap=6.0), 72
    part = _attention(width, m)
    g = torch.Generator().manual_seed(7)
    weights = _attention_weights(g, width, m, sink=(sink, 0.5), gain=1.0)
    part.bind(weights, rt)
    h = _inputs(dtype, width, 4, [230])[0]
    schedule = [[(0, 1)], [(0, 129)], [(0, 3)]] + [[(0, 1)]] * 97
    got = _feed(PartHarness(part.cache_need(), dtype, 1), _mixer_call(part, rt), [h], schedule, width)[0]
    want = _plain_attention(weights, m, h)
    assert rel_error(got, want) <= PART_TOL[dtype]
    without = _plain_attention(dict(weights, sink=torch.full((5,), -80.0)), m, h)
    if sink <= -30:
        assert rel_error(want, without) < 1e-9
    else:
        assert rel_error(want, without) > 0.1  # the test's premise: the sink matters
    if sink >= 30:
        assert np.abs(got).max() < 1e-5 * np.abs(without).max()


def _pointing(g, width, m, far, rows, n):
    """Weights and inputs for which the queries of `rows` score key `far` far above all others: the first half of an
    input makes the query, the second half the key, through the same matrix."""
    heads, groups, dim, half = m["heads"], m["kv_heads"], m["dim"], width // 2
    weights = _attention_weights(g, width, m, sink=(0.0, 0.3))
    base = torch.randn(dim, half, generator=g) / half ** 0.5
    q, k = torch.zeros(heads, dim, width), torch.zeros(groups, dim, width)
    q[:, :, :half], k[:, :, half:] = base, base
    weights["q"], weights["k"] = q.view(-1, width).to(torch.bfloat16), k.view(-1, width).to(torch.bfloat16)
    for name in ("q_bias", "k_bias"):
        weights[name] = torch.zeros_like(weights[name])
    h = torch.randn(n, width, generator=g)
    u = 2.5 * torch.randn(half, generator=g)
    h[far, half:] = u
    for row in rows:
        h[row, :half] = u
    return weights, h


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 127, 128, 300])
def test_a_far_key_among_hundreds(name, dtype, dim, far):
    """One key far back, at the sequence's first places and at and around page borders, takes the weight of the last
    tokens, in the prompt and in a token decoded alone; without it the output differs by far more than the tolerance."""
    rt = _runtime(dtype)
    n, width = 420, 48
    m = _shape(3, 1, dim, dim, 0, 0, scale=4.0 / dim, softcap=40.0)
    g = torch.Generator().manual_seed(20 + far)
    weights, h = _pointing(g, width, m, far, (n - 1, n), n + 1)
    h = h.to(dtype).float()
    part = _attention(width, m)
    part.bind(weights, rt)
    got = _feed(PartHarness(part.cache_need(), dtype, 1), _mixer_call(part, rt), [h], [[(0, n)], [(0, 1)]], width)[0]
    want = _plain_attention(weights, m, h)
    without = h.clone()
    without[far, width // 2:] = torch.randn(width // 2, generator=g).to(dtype).float()
    other = _plain_attention(weights, m, without)
    for row in (n - 1, n):
        assert rel_error(want[row], other[row]) > 0.2  # the test's premise: that key matters
        assert rel_error(got[row], want[row]) <= SHARP_TOL[dtype]


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("size,keep_first,marked", [(120, 24, 23), (120, 24, 24), (64, 1, 0), (64, 64, 63), (64, 65, 64),
                                                    (200, 0, 150), (33, 130, 129), (5, 3, 2), (257, 129, 128)])
def test_one_marked_value_shows_exactly_where_it_is_seen(name, dtype, dim, size, keep_first, marked):
    """One position's value is made huge and every score zero: the rows that see the position (inside the window, or
    because it is one of the kept first positions) differ from the run without the mark, all others do not, in a prompt of
    300 tokens and in 150 tokens decoded alone behind it. The position is the last kept one, the first that is not kept,
    at a page's border, or deep in the sequence."""
    rt = _runtime(dtype)
    width = 48
    m = _shape(3, 3, dim, dim, size, keep_first)
    part = _attention(width, m)
    g = torch.Generator().manual_seed(size + marked)
    weights = _attention_weights(g, width, m, sink=(-2.0, 0.3))
    for name_ in ("q", "q_bias"):
        weights[name_] = torch.zeros_like(weights[name_])
    v = torch.zeros(3 * dim, width)
    v[:, 0] = 1.0  # every value coordinate reads the input's first place
    weights["v"] = v.to(torch.bfloat16)
    part.bind(weights, rt)
    n = 450
    h = torch.randn(n, width, generator=g)
    h[:, 0] = 0.0
    plain = h.to(dtype).float().clone()
    h[marked, 0] = 1000.0
    h = h.to(dtype).float()
    schedule = [[(0, 300)]] + [[(0, 1)]] * 150
    got = _feed(PartHarness(part.cache_need(), dtype, 1), _mixer_call(part, rt), [h], schedule, width)[0]
    want, without = _plain_attention(weights, m, h), _plain_attention(weights, m, plain)
    seen = [i for i in range(n) if i >= marked and (i - marked < size or marked < keep_first)]
    unseen = [i for i in range(n) if i not in seen]
    scale = np.abs(without).max()
    moved = np.abs(want - without).max(axis=1) / scale
    assert all(moved[i] > 0.5 for i in seen) and all(moved[i] == 0 for i in unseen)  # the test's premise
    assert seen and (marked < keep_first or unseen[-1] > marked)
    assert max(np.abs(got[i] - want[i]).max() / np.abs(want[i]).max() for i in seen) <= PART_TOL[dtype]
    if unseen:
        assert np.abs(got[unseen] - without[unseen]).max() <= PART_TOL[dtype] * scale


@pytest.mark.parametrize("name,dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim", [(24, 40), (64, 64)])
def test_a_borrower_reads_the_owners_keys_under_its_own_window(name, dtype, dim, vdim):
    """The owner writes keys and values; a second mixer with tensors for queries alone and a wider (then a narrower) window
    reads them in the same step, in prompts, portions and single tokens, and writes nothing."""
    width = 64
    rt = _runtime(dtype)
    owner = _shape(4, 2, dim, vdim, 30, 2, scale=0.2)
    g = torch.Generator().manual_seed(dim)
    weights = _attention_weights(g, width, owner)
    for size, keep_first in ((150, 70), (7, 0)):
        borrower = dict(_shape(4, 2, dim, vdim, size, keep_first, scale=0.3, softcap=4.0))
        own = {k: v for k, v in _attention_weights(g, width, borrower).items() if k in ("q", "q_bias", "sink", "o")}
        readers = ((30, 2), (size, keep_first))
        first, second = _attention(width, owner, readers=readers), _attention(width, borrower, shares_keys=True)
        first.bind(weights, rt)
        second.bind(own, rt)

        def call(h, out, batch, view):
            from etalii.dllm_b200.kernels import ops

            first.forward(h.to(dtype), out, batch, view, rt, True, epilogue=ops.EPI_STORE_F32)
            second.forward(h.to(dtype), out, batch, view, rt, False, epilogue=ops.EPI_STORE_F32)

        h = _inputs(dtype, width, 10, [260])[0]
        schedule = [[(0, 200)], [(0, 2)]] + [[(0, 1)]] * 58
        got = _feed(PartHarness(first.cache_need(), dtype, 1), call, [h], schedule, width)[0]
        n64 = h.double().numpy()
        _, kept = P.attention(_np(weights, _RENAMES), owner, n64, None)
        want, _ = P.attention(_np(own, _RENAMES), borrower, n64, None, borrowed=kept)
        assert rel_error(got, want) <= PART_TOL[dtype]


@pytest.mark.parametrize("name,dtype", DTYPES)
def test_many_sequences_decode_side_by_side_over_pages_used_before(name, dtype):
    """Forty sequences of unequal lengths take slots and pages that other sequences have just given back, then decode
    together for eighty steps while their windows pass over what they decoded."""
    rt = _runtime(dtype)
    m, width, count = _shape(4, 2, 16, 24, 50, 6), 64, 40
    part = _attention(width, m)
    g = torch.Generator().manual_seed(11)
    weights = _attention_weights(g, width, m)
    part.bind(weights, rt)
    harness = PartHarness(part.cache_need(), dtype, count, pages=200)
    lengths = [1 + (7 * i) % 90 for i in range(count)]
    waste = _inputs(dtype, width, 5, [100] * count)
    _feed(harness, _mixer_call(part, rt), waste, [[(i, 100) for i in range(count)]], width)
    for i in range(count):
        harness.again(i)
    sequences = _inputs(dtype, width, 6, [n + 80 for n in lengths])
    schedule = [[(i, n) for i, n in enumerate(lengths)]] + [[(i, 1) for i in range(count)]] * 80
    got = _feed(harness, _mixer_call(part, rt), sequences, schedule, width)
    for rows, h in zip(got, sequences):
        assert rel_error(rows, _plain_attention(weights, m, h)) <= PART_TOL[dtype]
    harness.cache.check()


# ---- whole models through the engine -------------------------------------------------------------------------------------


class Case:
    def __init__(self, case, seed=1):
        self.config = C.CASES[case]()
        self.tensors = C.random_weights(self.config, seed)
        self.weights = C.as_numpy(self.tensors)
        self._memo = {}

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self._memo:
            self._memo[key] = P.forward(self.config, self.weights, list(tokens))
        return self._memo[key]


_CASES = {}


def _case(name) -> Case:
    if name not in _CASES:
        _CASES[name] = Case(name)
    return _CASES[name]


def _run(engine, prompts, schedule):
    """Feeds `prompts` by `schedule` (steps of (prompt, count)); a prompt's slot is given back with its last token.
    Returns every position's logits per prompt."""
    at = [0] * len(prompts)
    slots = {}
    rows = [[] for _ in prompts]
    for step in schedule:
        for i, _ in step:
            if i not in slots:
                slots[i] = engine.open(1)[0]
        pieces = [prompts[i][at[i]:at[i] + n] for i, n in step]
        out = host(engine.step([slots[i] for i, _ in step], pieces, [list(range(len(p))) for p in pieces]))
        engine.check()
        offset = 0
        for (i, n) in step:
            rows[i].append(out[offset:offset + n])
            offset += n
            at[i] += n
            if at[i] == len(prompts[i]):
                engine.close([slots.pop(i)])
    assert not slots
    return [np.concatenate(r) for r in rows]


def _compare(case, got, prompts, dtype_name):
    """Every logit of every position within the tolerance in float32. bfloat16: nine of ten positions within twice the
    tolerance, the median within it and none beyond four times it (the sums over the layers' results take differences of
    streams, which keep the streams' rounding; what a lost key or a stale page does is decided in float32, where the same
    schedules run through the same cache and step function, and by the tests with weights made to point)."""
    errors = []
    for rows, tokens in zip(got, prompts):
        want = case.logits(tokens)
        assert rows.shape == want.shape
        errors += list(np.abs(rows - want).max(axis=1) / np.abs(want).max())
    errors = np.sort(np.asarray(errors))
    print(dtype_name, np.median(errors), errors[int(0.9 * (len(errors) - 1))], errors[-1])
    if dtype_name == "float32":
        assert errors[-1] <= TOL[dtype_name]
    else:
        assert errors[int(0.9 * (len(errors) - 1))] <= 2 * TOL[dtype_name] and errors[-1] <= 4 * TOL[dtype_name]
        assert np.median(errors) <= TOL[dtype_name]


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_whole_prompts_alone_and_as_one_batch(name, dtype_name):
    case = _case(name)
    engine = C.make_engine(case.config, case.tensors, dtype_name)
    prompts = C.tokens_for(case.config, [1, 2, 70, 231, 5])
    alone = _run(engine, prompts, [[(i, len(p))] for i, p in enumerate(prompts)])
    _compare(case, alone, prompts, dtype_name)
    together = _run(engine, prompts, [[(i, len(p)) for i, p in enumerate(prompts)]])
    _compare(case, together, prompts, dtype_name)
    if dtype_name == "float32":  # batch mates change nothing beyond rounding; in float32 that is very little
        assert all(rel_error(a, b) <= 1e-5 for a, b in zip(alone, together))
    engine.cache.check()


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_portions_and_single_tokens(name, dtype_name):
    """One prompt cut into portions of 64, 2, 65, 3 and 1, 1, ...: the pieces cross page borders and window edges and
    end in token-by-token decoding; then the first tokens one by one from an empty cache."""
    case = _case(name)
    engine = C.make_engine(case.config, case.tensors, dtype_name)
    prompt = C.tokens_for(case.config, [250], seed=6)[0]
    schedule = [[(0, 64)], [(0, 2)], [(0, 65)], [(0, 3)]] + [[(0, 1)]] * 116
    _compare(case, _run(engine, [prompt], schedule), [prompt], dtype_name)
    schedule = [[(0, 1)]] * 5 + [[(0, 245)]]
    _compare(case, _run(engine, [prompt], schedule), [prompt], dtype_name)
    engine.cache.check()
    assert engine.cache.pages_held() == 0


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_a_window_passes_over_many_pages(dtype_name):
    """A window of 600 with 70 kept first positions, a borrower's of 100 with 64: a prompt of 750 tokens in uneven portions
    and then single tokens, so that pages between the kept ones and the window go back to the pool on the way."""
    case = _case("tiled")
    engine = C.make_engine(case.config, case.tensors, dtype_name)
    prompt = C.tokens_for(case.config, [790], seed=16)[0]
    schedule = [[(0, 700)], [(0, 2)], [(0, 48)]] + [[(0, 1)]] * 40
    _compare(case, _run(engine, [prompt], schedule), [prompt], dtype_name)
    engine.cache.check()


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_unequal_batches_early_finishers_and_slots_used_again(name, dtype_name):
    """Requests of unequal length start together and decode together; the shorter ones end earlier and give their
    slots and pages back; later requests take those slots and pages (which still hold the old rows) and run beside the
    survivors."""
    case = _case(name)
    engine = C.make_engine(case.config, case.tensors, dtype_name, max_tokens=64 * 10, max_slots=4)
    prompts = C.tokens_for(case.config, [40, 9, 75, 30, 12], seed=8)
    schedule = [[(0, 30), (1, 6), (2, 66)]]
    schedule += [[(0, 1), (1, 1), (2, 1)]] * 3          # request 1 ends here
    schedule += [[(0, 1), (2, 1)]] * 6                  # request 2 ends here
    schedule += [[(3, 25), (4, 10)]]                    # two new requests take the freed slots
    schedule += [[(0, 1), (3, 1), (4, 1)]]              # ... and decode beside the survivor
    schedule += [[(3, 1), (4, 1)], [(3, 3)]]
    got = _run(engine, prompts, schedule)
    _compare(case, got, prompts, dtype_name)
    engine.cache.check()
    assert engine.cache.pages_held() == 0


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_long_decoding_through_the_decode_graph(dtype_name):
    """A hundred and fifty single-token steps of three sequences as the generation loop runs them (one captured graph
    replayed), across page borders and with every window passing over decoded tokens; then the last step's logits
    against the plain implementation on the whole history."""
    case = _case("mixed")
    engine = C.make_engine(case.config, case.tensors, dtype_name, decode_logits=True)
    assert engine.cuda_graphs
    prompts = C.tokens_for(case.config, [7, 20, 66], seed=9)
    slots = engine.open(3)
    first = host(engine.step(slots, prompts)).argmax(axis=1).tolist()
    chosen = engine.decode(slots, first, 150)
    histories = [p + [f] + [step[i] for step in chosen] for i, (p, f) in enumerate(zip(prompts, first))]
    graph_logits = host(engine.last_decode_graph.logits)  # of the last step: history without its last token
    for i, history in enumerate(histories):
        want = case.logits(history[:-1])[-1]
        assert rel_error(graph_logits[i], want) <= TOL[dtype_name] * (3.0 if dtype_name == "bfloat16" else 1.0)
        if dtype_name == "float32":
            assert int(np.argmax(want)) == history[-1]
    engine.close(slots)
    engine.cache.check()


def test_greedy_generation_through_the_generation_loop():
    """`Engine.generate` (batches planned by the scheduler, prompt step, decode graphs, early finishers) gives the
    tokens the plain implementation chooses greedily through its own carried state, in float32."""
    from etalii.dllm_b200 import SamplingOptions

    case = _case("mixed")
    engine = C.make_engine(case.config, case.tensors, "float32")
    prompts = C.tokens_for(case.config, [3, 18, 70], seed=10)
    results = engine.generate(prompts, 12, SamplingOptions(), ignore_eos=True)
    for prompt, result in zip(prompts, results):
        assert list(result.tokens) == P.greedy(case.config, case.weights, prompt, 12)
    again = engine.generate(prompts[:2], 5, SamplingOptions(), ignore_eos=True)  # the slots are used again
    assert [list(r.tokens) for r in again] == [list(r.tokens)[:5] for r in results[:2]]


def test_sampled_generation_runs_in_bfloat16():
    from etalii.dllm_b200 import SamplingOptions

    case = _case("tiled")
    engine = C.make_engine(case.config, case.tensors, "bfloat16")
    prompts = C.tokens_for(case.config, [5, 33], seed=11)
    a = engine.generate(prompts, 20, SamplingOptions(temperature=0.8, top_k=20, seed=3), ignore_eos=True)
    b = engine.generate(prompts, 20, SamplingOptions(temperature=0.8, top_k=20, seed=3), ignore_eos=True)
    assert [list(r.tokens) for r in a] == [list(r.tokens) for r in b] and all(len(r.tokens) == 20 for r in a)


def test_trace_replay_and_command_line_on_a_tezinex_folder(tmp_path):
    """bin/trace_run and `dllm-b200 generate` as subprocesses on a model folder the library wrote."""
    import json
    import os
    import subprocess
    import sys

    from etalii.dllm_b200.weights.random_init import write_model

    case = _case("narrow")
    folder = write_model(str(tmp_path / "model"), case.config, case.tensors)
    tokens = C.tokens_for(case.config, [20], seed=12)[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[18:20], "want": [1]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype",
                           "float32", "--out", str(out), "--max-tokens", "128"],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                          timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.split("\n") if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = case.logits(tokens)
    first = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    last = np.fromfile(out / "2.f32", dtype="<f4").reshape(1, -1)
    assert not (out / "1.f32").exists()
    assert rel_error(first, want[[0, 16]]) <= TOL["float32"] and rel_error(last, want[[19]]) <= TOL["float32"]

    tool = [sys.executable, os.path.join(root, "bin", "dllm-b200")]
    done = subprocess.run(tool + ["--model", folder, "info"], capture_output=True, text=True, timeout=600)
    assert done.returncode == 0 and json.loads(done.stdout)["architecture"] == "Tezinex"
    prompt = tokens[:9]
    done = subprocess.run(tool + ["--model", folder, "--dtype", "float32", "--cache-tokens", "256", "generate",
                                  "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "6", "--ignore-eos"],
                          capture_output=True, text=True, timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [int(t) for t in done.stdout.split()] == P.greedy(case.config, case.weights, prompt, 6)
