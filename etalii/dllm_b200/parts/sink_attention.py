"""Grouped-query softmax attention with everything around the scores optional: biases, norms of queries and keys, rotary
positions, values mixed with another layer's, capped scores, a sink, and a window that also keeps a sequence's first
positions, or chunks.

Per token, from the mixer's input h: q = W_q h [heads x dim], k = W_k h [kv_heads x dim], v = W_v h [kv_heads x vdim]
(with `biases`, each plus its bias, and the output plus one with `output_bias`). With `qk_eps` every head of q and of k is
RMS-normed over dim with a weight shared by the heads; then a `position` part turns its first dimensions. Query head a uses
key/value head a / (heads / kv_heads). Position i sees j <= i with i - j < window (None: all) or, with `chunk`, those of
its own chunk of that many positions (counted from the sequence's start), and the sequence's first `keep_first` positions
at any distance. A visible key's score is q . k * scale, then softcap * tanh(score / softcap) (0: as it is). The softmax's
denominator also holds exp(sink_a) with `sink` True (a learned number per head that has no key and no value, is neither
scaled nor capped and counts once), 1 with `sink` "unit", nothing with False. W_o runs over the concatenated heads.

`value_mix`: None; "keep" (the layer's values of the step, as projected, stay in a float32 work buffer); or "mix": v <-
(1 - share) v + share kept, share a learned number and kept what the step's "keep" layer left. The cache holds the mixed v.

A mixer built with `shares_keys=True` has no key and value tensors: it reads the cache entry another layer wrote (the
schedule names it) with queries, window and everything else of its own. `readers` lists (window, keep_first) of all the
mixers that read an entry, its owner included: the cache keeps a position while any of them can still see it.

One product makes everything a token needs of h: [q | k | v]. Its biases are added behind it, or with `ones_column` inside
it, as one more column of the matrix (the input rows then carry a 1: `ops.norm_operands`). Biases, norms, angles, scores,
cap, softmax and sums are float32; the cache holds keys and values in the activation type."""
from __future__ import annotations

import torch

from ..cache.paged import CacheNeed
from ..kernels import ops
from .attention import TCGEN05_ATTENTION_FROM
from .feed_forward import with_bias_column
from .norm import row_rule
from .registry import build_part, register_part
from .spec import ParamSpec


class SinkAttention:
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float,
                 softcap: float = 0.0, window: int | None = None, keep_first: int = 0, biases: bool = False,
                 sink: bool | str = True, shares_keys: bool = False, readers=(), chunk: int | None = None, position=None,
                 qk_eps: float | None = None, output_bias: bool = False, ones_column: bool = False,
                 value_mix: str | None = None) -> None:
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} kv heads")
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.dim, self.vdim, self.scale, self.softcap = int(dim), int(vdim), float(scale), float(softcap or 0.0)
        self.window = int(window) if window else 0
        self.keep_first = int(keep_first) if self.window or chunk else 0
        self.biases, self.sink, self.shares_keys = bool(biases), sink, bool(shares_keys)
        if sink not in (True, False, "unit") or value_mix not in (None, "keep", "mix"):
            raise ValueError(f"sink {sink!r}: True, False or unit; value_mix {value_mix!r}: None, keep or mix")
        self.chunk = int(chunk) if chunk else 0
        if self.chunk and (shares_keys or readers):
            raise ValueError("borrowed keys with chunks are not built")
        self.position = build_part("position", position) if position is not None else None
        self.qk_eps = float(qk_eps) if qk_eps is not None else None
        self.has_output_bias, self.wants_ones, self.value_mix = bool(output_bias), bool(ones_column), value_mix
        self.share = None
        readers = tuple(readers) or ((self.window or None, self.keep_first),)
        bounded = all(window for window, _ in readers)
        self.cache_window = max(int(window) for window, _ in readers) if bounded else None
        self.cache_keep = max(int(keep) for _, keep in readers) if bounded else 0
        self.padded = -(-self.num_heads * self.vdim // 8) * 8
        """The output product's rows: heads x vdim filled up with zeros to 16-byte pieces."""
        self.output_scale = 1.0
        self.w_in = self.w_o = self.bias_rows = self.sinks = self.norm_weights = self.output_bias = None

    @staticmethod
    def parameters(hidden_size, num_heads, num_kv_heads, dim, vdim, biases=False, sink=True, shares_keys=False,
                   qk_eps=None, output_bias=False, value_mix=None, **_) -> dict[str, ParamSpec]:
        heads, groups, dim, vdim = int(num_heads), int(num_kv_heads), int(dim), int(vdim)
        sizes = {"q": heads * dim}
        if not shares_keys:
            sizes.update(k=groups * dim, v=groups * vdim)
        out = {name: ParamSpec((rows, hidden_size)) for name, rows in sizes.items()}
        if biases:
            out.update({name + "_bias": ParamSpec((rows,)) for name, rows in sizes.items()})
        if sink is True:
            out["sink"] = ParamSpec((heads,))
        if qk_eps is not None:
            out["q_norm"] = ParamSpec((dim,), "ones")
            if not shares_keys:
                out["k_norm"] = ParamSpec((dim,), "ones")
        if output_bias:
            out["o_bias"] = ParamSpec((hidden_size,))
        if value_mix is not None:
            out["share"] = ParamSpec(())
        out["o"] = ParamSpec((hidden_size, heads * vdim))
        return out

    def supports(self, rt) -> str | None:
        if self.dim > 256 or self.vdim > 256:
            return f"dim {self.dim}, vdim {self.vdim}: the attention kernels take at most 256 each"
        return row_rule(rt, hidden_size=self.hidden_size)

    def cache_need(self) -> CacheNeed:
        return CacheNeed("kv", kv_heads=self.num_kv_heads, head_dim=self.dim,
                         value_dim=0 if self.vdim == self.dim else self.vdim, window=self.cache_window,
                         keep_first=self.cache_keep, chunk=self.chunk or None)

    def bind(self, tensors, rt) -> None:
        names = ("q",) if self.shares_keys else ("q", "k", "v")
        w_in = torch.cat([tensors[name].to(rt.dtype) for name in names], dim=0)
        if self.wants_ones:
            w_in = with_bias_column(w_in, torch.cat([tensors[name + "_bias"] for name in names]) if self.biases else None)
        self.w_in = w_in.contiguous().to(rt.device)
        values = self.num_heads * self.vdim
        o = torch.zeros(self.hidden_size, self.padded, dtype=rt.dtype)
        o[:, :values] = tensors["o"].to(rt.dtype)
        self.w_o = o.to(rt.device)
        if self.biases and not self.wants_ones:
            rows = [tensors[name + "_bias"].to(torch.float32).contiguous().to(rt.device) for name in names]
            self.bias_rows = (*rows, None, None)[:3]
        if self.sink is True:
            self.sinks = rt.to_device(tensors["sink"], torch.float32)
        elif self.sink:  # (a sink whose score is zero)
            self.sinks = torch.zeros(self.num_heads, dtype=torch.float32, device=rt.device)
        if self.qk_eps is not None:
            self.norm_weights = tuple(rt.to_device(tensors[name], torch.float32) if name in tensors else None
                                      for name in ("q_norm", "k_norm"))
        if self.has_output_bias:
            self.output_bias = rt.to_device(tensors["o_bias"], torch.float32)
        if self.value_mix == "mix":
            self.share = float(tensors["share"].to(torch.float32).reshape(()).item())
        if self.position is not None:
            self.position.bind({}, rt)

    def give_output_matrix(self, rt, scale: float) -> torch.Tensor | None:
        """As `Attention.give_output_matrix` (None also for an output that has a bias or ends between 16-byte pieces)."""
        if self.has_output_bias or self.padded != self.num_heads * self.vdim:
            return None
        w, self.w_o, self.output_scale = self.w_o, None, float(scale)
        return w

    def take_output_bias(self) -> torch.Tensor | None:
        """The output bias (None: there is none); the part no longer adds it itself."""
        bias, self.output_bias = self.output_bias, None
        return bias

    def forward(self, h: torch.Tensor, residual: torch.Tensor, batch, cache, rt, write_cache: bool = True,
                epilogue: int = ops.EPI_RESIDUAL, operand=None) -> None:
        """h: the mixer's input [tokens, hidden] in the activation type. Adds the output to `residual` (float32), or
        with `epilogue=ops.EPI_STORE_F32` writes it there, or with `operand` = (rows, column) leaves what the output
        matrix multiplies there (`give_output_matrix`)."""
        n = batch.n_tokens
        heads, groups, dim, vdim = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        rows = rt.ws.buffer("mixer_rows", (n, self.w_in.shape[0]), torch.float32)
        ops.gemm(rows, h, self.w_in, ops.EPI_STORE_F32)
        q = rt.ws.buffer("sink_q", (n, heads * dim), rt.dtype)
        k_at = heads * dim
        first = None
        if self.value_mix is not None:
            first = rt.ws.buffer("kept_values", (n, groups * vdim), torch.float32)
        table = self.position.table() if self.position is not None else None
        ops.qkv_prepare(rows, 0, k_at, k_at + groups * dim, q, cache, heads, batch,
                        write_cache and not self.shares_keys, biases=self.bias_rows, norm_weights=self.norm_weights,
                        eps=self.qk_eps or 0.0, table=table,
                        rotary_dim=self.position.rotary_dim if self.position is not None else 0, first=first,
                        share=self.share)
        attended, at = operand or (rt.ws.buffer("attended", (n, self.padded), rt.dtype), None)
        attend = ops.sink_attention
        if ops.sink_attention_tiles(rt.dtype, dim, vdim, cache.page_size):
            reach = batch.max_context
            if self.window or self.chunk:  # (keys a tile of queries walks)
                reach = min(reach, min(self.window or self.chunk, self.chunk or self.window) + self.keep_first + 64)
            if batch.is_decode:
                attend = ops.sink_attention_decode
            elif ops.sink_attention_tcgen05_supported(cache) and reach > TCGEN05_ATTENTION_FROM[dim]:
                attend = ops.sink_attention_tcgen05
            else:
                attend = ops.sink_attention_prefill
        more = {"chunk": self.chunk} if self.chunk else {}
        if operand is not None:
            more.update(out_scale=self.output_scale, out_at=at)
        attend(attended, q, cache, heads, self.scale, self.softcap, self.sinks, self.window, self.keep_first, batch, **more)
        if operand is not None:
            return
        ops.gemm(residual, attended, self.w_o, epilogue)
        if self.output_bias is not None:
            ops.add_row(residual, self.output_bias)

    def kernel_libraries(self, rt) -> set[str]:
        names = {"elementwise", "qkv_prepare"}
        if rt.dtype != torch.bfloat16:
            return names | {"gemm_simt", "sink_attention"}
        names |= {"gemv", "gemv_cluster", "gemm_tcgen05"}
        if not ops.sink_attention_tiles(rt.dtype, self.dim, self.vdim):
            return names | {"sink_attention"}
        if self.dim == self.vdim and self.dim in TCGEN05_ATTENTION_FROM:
            names.add("sink_attention_tcgen05")
        return names | {"sink_attention_prefill", "sink_attention_decode"}


register_part("mixer", "sink_attention", SinkAttention)
