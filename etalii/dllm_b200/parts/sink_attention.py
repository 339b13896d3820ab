"""Grouped-query softmax attention with capped scores, a sink, and a sliding window that also keeps a sequence's first
positions.

Per token, from the mixer's input h: q = W_q h [heads x dim], k = W_k h [kv_heads x dim], v = W_v h [kv_heads x vdim]
(with `biases`, each plus its bias). Query head a uses key/value head a / (heads / kv_heads); there is no rotation.
Position i sees j <= i with i - j < window (None: all), and the sequence's first `keep_first` positions at any distance.
A visible key's score is q . k * scale, then softcap * tanh(score / softcap) (0: as it is); the softmax's denominator
also holds exp(sink_a), a learned number per head (`sink`) that has no key and no value, is neither scaled nor capped and
counts once. W_o runs over the concatenated heads.

A mixer built with `shares_keys=True` has no key and value tensors: it reads the cache entry another layer wrote (the
schedule names it) with queries, window and everything else of its own. `readers` lists (window, keep_first) of all the
mixers that read an entry, its owner included: the cache keeps a position while any of them can still see it.

One product makes everything a token needs of h: [q | k | v]. Biases, scores, cap, softmax and sums are float32; the cache
holds keys and values in the activation type."""
from __future__ import annotations

import torch

from ..cache.paged import CacheNeed
from ..kernels import ops
from .attention import TCGEN05_ATTENTION_FROM
from .norm import row_rule
from .registry import register_part
from .spec import ParamSpec


class SinkAttention:
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float,
                 softcap: float = 0.0, window: int | None = None, keep_first: int = 0, biases: bool = False,
                 sink: bool = True, shares_keys: bool = False, readers=()) -> None:
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} kv heads")
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.dim, self.vdim, self.scale, self.softcap = int(dim), int(vdim), float(scale), float(softcap or 0.0)
        self.window = int(window) if window else 0
        self.keep_first = int(keep_first) if self.window else 0
        self.biases, self.sink, self.shares_keys = bool(biases), bool(sink), bool(shares_keys)
        readers = tuple(readers) or ((self.window or None, self.keep_first),)
        bounded = all(window for window, _ in readers)
        self.cache_window = max(int(window) for window, _ in readers) if bounded else None
        self.cache_keep = max(int(keep) for _, keep in readers) if bounded else 0
        self.padded = -(-self.num_heads * self.vdim // 8) * 8
        """The output product's rows: heads x vdim filled up with zeros to 16-byte pieces."""
        self.w_in = self.w_o = self.bias_rows = self.sinks = None

    @staticmethod
    def parameters(hidden_size, num_heads, num_kv_heads, dim, vdim, biases=False, sink=True, shares_keys=False,
                   **_) -> dict[str, ParamSpec]:
        heads, groups, dim, vdim = int(num_heads), int(num_kv_heads), int(dim), int(vdim)
        sizes = {"q": heads * dim}
        if not shares_keys:
            sizes.update(k=groups * dim, v=groups * vdim)
        out = {name: ParamSpec((rows, hidden_size)) for name, rows in sizes.items()}
        if biases:
            out.update({name + "_bias": ParamSpec((rows,)) for name, rows in sizes.items()})
        if sink:
            out["sink"] = ParamSpec((heads,))
        out["o"] = ParamSpec((hidden_size, heads * vdim))
        return out

    def supports(self, rt) -> str | None:
        if self.dim > 256 or self.vdim > 256:
            return f"dim {self.dim}, vdim {self.vdim}: the attention kernels take at most 256 each"
        return row_rule(rt, hidden_size=self.hidden_size)

    def cache_need(self) -> CacheNeed:
        return CacheNeed("kv", kv_heads=self.num_kv_heads, head_dim=self.dim,
                         value_dim=0 if self.vdim == self.dim else self.vdim, window=self.cache_window,
                         keep_first=self.cache_keep)

    def bind(self, tensors, rt) -> None:
        names = ("q",) if self.shares_keys else ("q", "k", "v")
        self.w_in = torch.cat([tensors[name].to(rt.dtype) for name in names], dim=0).contiguous().to(rt.device)
        values = self.num_heads * self.vdim
        o = torch.zeros(self.hidden_size, self.padded, dtype=rt.dtype)
        o[:, :values] = tensors["o"].to(rt.dtype)
        self.w_o = o.to(rt.device)
        if self.biases:
            rows = [tensors[name + "_bias"].to(torch.float32).contiguous().to(rt.device) for name in names]
            self.bias_rows = (*rows, None, None)[:3]
        self.sinks = rt.to_device(tensors["sink"], torch.float32) if self.sink else None

    def forward(self, h: torch.Tensor, residual: torch.Tensor, batch, cache, rt, write_cache: bool = True,
                epilogue: int = ops.EPI_RESIDUAL) -> None:
        """h: the mixer's input [tokens, hidden] in the activation type. Adds the output to `residual` (float32), or
        with `epilogue=ops.EPI_STORE_F32` writes it there."""
        n = batch.n_tokens
        heads, groups, dim, vdim = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        rows = rt.ws.buffer("mixer_rows", (n, self.w_in.shape[0]), torch.float32)
        ops.gemm(rows, h, self.w_in, ops.EPI_STORE_F32)
        q = rt.ws.buffer("sink_q", (n, heads * dim), rt.dtype)
        k_at = heads * dim
        ops.sigmoid_prepare(rows, 0, k_at, k_at + groups * dim, q, cache, heads, self.bias_rows, None, 0.0, batch,
                            write_cache and not self.shares_keys)
        attended = rt.ws.buffer("attended", (n, self.padded), rt.dtype)
        attend = ops.sink_attention
        if ops.sink_attention_tiles(rt.dtype, dim, vdim, cache.page_size):
            reach = batch.max_context
            if self.window:
                reach = min(reach, self.window + self.keep_first + 64)  # (keys a tile of queries walks)
            if batch.is_decode:
                attend = ops.sink_attention_decode
            elif ops.sink_attention_tcgen05_supported(cache) and reach > TCGEN05_ATTENTION_FROM[dim]:
                attend = ops.sink_attention_tcgen05
            else:
                attend = ops.sink_attention_prefill
        attend(attended, q, cache, heads, self.scale, self.softcap, self.sinks, self.window, self.keep_first, batch)
        ops.gemm(residual, attended, self.w_o, epilogue)

    def kernel_libraries(self, rt) -> set[str]:
        names = {"elementwise", "sigmoid_attention"}
        if rt.dtype != torch.bfloat16:
            return names | {"gemm_simt", "sink_attention"}
        names |= {"gemv", "gemv_cluster", "gemm_tcgen05"}
        if not ops.sink_attention_tiles(rt.dtype, self.dim, self.vdim):
            return names | {"sink_attention"}
        if self.dim == self.vdim and self.dim in TCGEN05_ATTENTION_FROM:
            names.add("sink_attention_tcgen05")
        return names | {"sink_attention_prefill", "sink_attention_decode"}


register_part("mixer", "sink_attention", SinkAttention)
