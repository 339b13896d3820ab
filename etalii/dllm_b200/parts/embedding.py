"""Token embedding (row gather into the float32 residual stream) and the output head (final hidden rows times the
head matrix, float32 logits). A tied head names the embedding's tensor and shares its device copy
(reference: src/etalii_dllm/transformer.py:659-663, 427-443)."""
from __future__ import annotations

import torch

from ..kernels import ops
from .norm import project, row_rule
from .registry import build_part, register_part
from .spec import ParamSpec


class TokenEmbedding:
    wants_positions = True

    def __init__(self, vocab_size: int, hidden_size: int, scale: float = 1.0, position=None,
                 norm_eps: float | None = None) -> None:
        """`scale`: every embedding row is multiplied by it on the way into the stream (in float32). `position`: a
        position part whose vector is then added (sinusoidal). `norm_eps`: the rows are then RMS-normed with a weight of
        their own (a tensor `norm`), in the same kernel."""
        self.vocab_size, self.hidden_size, self.scale = int(vocab_size), int(hidden_size), float(scale)
        self.position = build_part("position", position) if position is not None else None
        self.norm_eps = float(norm_eps) if norm_eps is not None else None
        if self.norm_eps is not None and self.position is not None:
            raise ValueError("normed embedding rows with a position vector are not built")
        self.weight = self.norm_weight = None

    @staticmethod
    def parameters(vocab_size, hidden_size, norm_eps=None, **_) -> dict[str, ParamSpec]:
        out = {"weight": ParamSpec((vocab_size, hidden_size))}
        if norm_eps is not None:
            out["norm"] = ParamSpec((hidden_size,), "ones")
        return out

    def bind(self, tensors, rt) -> None:
        self.weight = rt.to_device(tensors["weight"], rt.dtype)
        if self.norm_eps is not None:
            self.norm_weight = rt.to_device(tensors["norm"], torch.float32)
        if self.position is not None:
            self.position.bind({}, rt)

    def forward(self, tokens: torch.Tensor, n_tokens: int, rt, positions: torch.Tensor | None = None) -> torch.Tensor:
        # a token outside the table sets the kernels' shared status word, which the engine looks at after each
        # step it waits for (kernels/ops.py::raise_if_failed)
        x = rt.ws.buffer("residual", (n_tokens, self.hidden_size), torch.float32)
        if self.position is not None:
            ops.embed_sinusoid(x, self.weight, tokens, positions, self.position.frequencies(), scale=self.scale)
        elif self.norm_eps is not None:
            ops.embed_normed(x, self.weight, tokens, self.norm_weight, self.norm_eps, scale=self.scale)
        else:
            ops.embed(x, self.weight, tokens, scale=self.scale)
        return x


class LinearHead:
    accepts_pending_norm = True

    def __init__(self, vocab_size: int, hidden_size: int, softcap: float = 0.0) -> None:
        """`softcap`: the logits become softcap * tanh(logits / softcap) (0: as they are). The cap keeps their order,
        so the greedy choice inside the product is made before it."""
        self.vocab_size, self.hidden_size, self.softcap = int(vocab_size), int(hidden_size), float(softcap or 0.0)
        self.weight = None

    @staticmethod
    def parameters(vocab_size, hidden_size, **_) -> dict[str, ParamSpec]:
        return {"weight": ParamSpec((vocab_size, hidden_size))}

    def bind(self, tensors, rt) -> None:
        self.weight = rt.to_device(tensors["weight"], rt.dtype)

    def supports(self, rt) -> str | None:
        return row_rule(rt, hidden_size=self.hidden_size)

    def choose_greedy(self, hidden, rt, out: torch.Tensor) -> bool:
        """The greedy choice without logits: out[r] = argmax of row r's logits (lowest index on ties), made inside
        the head product. Returns False, having done nothing, where that kernel does not take the step."""
        from .norm import NormedInput, fuses_norm

        rows = hidden.shape[0]
        if not ops.head_argmax_supported(rows, self.weight):
            return False
        scratch = rt.ws.buffer("head_candidates", (ops.head_argmax_scratch(rows, self.vocab_size),), torch.float32)
        if isinstance(hidden, NormedInput):
            if fuses_norm(self.weight):
                ops.head_argmax(out, hidden.x, self.weight, scratch, norm_weight=hidden.weight, eps=hidden.eps)
                return True
            hidden = hidden.tensor()
        ops.head_argmax(out, hidden, self.weight, scratch)
        return True

    def forward(self, hidden, rt) -> torch.Tensor:
        """hidden: final-normed rows, or the norm still pending (`NormedInput`)."""
        logits = rt.ws.buffer("logits", (hidden.shape[0], self.vocab_size), torch.float32)
        project(logits, hidden, self.weight, ops.EPI_STORE_F32)
        if self.softcap > 0.0:
            ops.softcap_rows(logits, self.softcap)
        return logits


register_part("embedding", "token_embedding", TokenEmbedding)
register_part("head", "linear", LinearHead)
