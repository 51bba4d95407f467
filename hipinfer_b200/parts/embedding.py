"""Token embedding (a row gather without scaling, src/kernels.cuh:1877-1881) into the 32-bit
residual stream, and the output head (logits = xn W^T, W the embedding table when tied,
src/api.cu:1367, 1795-1812) producing 32-bit logits."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import ParamSpec
from .norm import RMSNorm
from .registry import Part, build_part, register_part, to_compute


class TokenEmbedding(Part):
    """params: name, vocab_size, hidden_size."""

    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        self.name, self.vocab, self.hidden = params["name"], int(params["vocab_size"]), int(params["hidden_size"])
        self.table = None

    def param_specs(self):
        return [ParamSpec(self.name, (self.vocab, self.hidden))]

    def load(self, tensors):
        self.table = to_compute(tensors[self.name], self.ctx)

    def forward(self, tokens):
        x = torch.empty(tokens.numel(), self.hidden, dtype=torch.float32, device=tokens.device)
        return ops.embedding(self.table, tokens, x)


class ScaledPositionEmbedding(Part):
    """x = table[token] * scale + position_table[position]: a scaled token embedding and a learned vector per absolute
    position (not scaled). params: name, vocab_size, hidden_size, scale (default 1), position_name (absent: no position
    vectors), max_position. The decoder hands it the step's positions (`takes_positions`)."""

    takes_positions = True

    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        self.name, self.vocab, self.hidden = params["name"], int(params["vocab_size"]), int(params["hidden_size"])
        self.scale = float(params.get("scale", 1.0))
        self.position_name = params.get("position_name")
        self.max_position = int(params.get("max_position", 0))
        self.table = self.position_table = None

    def param_specs(self):
        specs = [ParamSpec(self.name, (self.vocab, self.hidden))]
        if self.position_name:
            specs.append(ParamSpec(self.position_name, (self.max_position, self.hidden)))
        return specs

    def load(self, tensors):
        self.table = to_compute(tensors[self.name], self.ctx)
        if self.position_name:
            self.position_table = to_compute(tensors[self.position_name], self.ctx).to(self.table.dtype)

    def forward(self, tokens, positions):
        x = torch.empty(tokens.numel(), self.hidden, dtype=torch.float32, device=tokens.device)
        return ops.embedding_scaled(self.table, tokens, x, self.scale, self.position_table, positions)


class NormedTokenEmbedding(Part):
    """x = norm(table[token]): a token embedding whose rows go through a norm of the model's kind before they enter the
    32-bit residual stream (the norm's result stays 32-bit). params: name, vocab_size, hidden_size, norm (the PartSpec
    of a norm over hidden_size)."""

    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        self.name, self.vocab, self.hidden = params["name"], int(params["vocab_size"]), int(params["hidden_size"])
        self.norm = build_part("norm", params["norm"], ctx, prefix)
        self.table = None

    def param_specs(self):
        return [ParamSpec(self.name, (self.vocab, self.hidden))] + self.norm.param_specs()

    def load(self, tensors):
        self.table = to_compute(tensors[self.name], self.ctx)
        self.norm.load(tensors)

    def forward(self, tokens):
        raw = torch.empty(tokens.numel(), self.hidden, dtype=torch.float32, device=tokens.device)
        ops.embedding(self.table, tokens, raw)
        return self.norm.forward(raw, out=torch.empty_like(raw))


class BigramTokenEmbedding(Part):
    """x = norm(table[token] * scale + bigram[row]): a scaled token embedding, a second table addressed by the token and the one
    before it, and a norm whose result stays 32-bit. The row is (previous * mul_prev + token * mul_cur) mod buckets, and row
    `buckets` (the last) for a sequence's first token. The previous token is state of the request: a step's first row of a
    request finds it in the request's slot. All of it is one kernel (csrc/residual_rows.cu).

    params: name, vocab_size, hidden_size, scale (default 1), bigram (buckets, mul_prev, mul_cur) or None, bigram_name (default
    "bigram"), norm (the PartSpec of an RMS norm over hidden_size) or None."""

    takes_batch = True

    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        self.name, self.vocab, self.hidden = params["name"], int(params["vocab_size"]), int(params["hidden_size"])
        self.scale = float(params.get("scale", 1.0))
        self.bigram = tuple(int(v) for v in params["bigram"]) if params.get("bigram") else None
        if self.bigram and (self.bigram[0] < 1 or min(self.bigram[1:]) < 0):
            raise ValueError(f"bigram embedding: {self.bigram[0]} buckets, multipliers {self.bigram[1:]}")
        self.bigram_name = params.get("bigram_name", "bigram")
        self.norm = build_part("norm", params["norm"], ctx, prefix) if params.get("norm") else None
        if self.norm is not None and not isinstance(self.norm, RMSNorm):
            raise ValueError("bigram embedding: the norm must be an RMS norm")
        self.table = self.bigram_table = self.norm_weight = None

    def param_specs(self):
        specs = [ParamSpec(self.name, (self.vocab, self.hidden))]
        if self.bigram:
            specs.append(ParamSpec(self.bigram_name, (self.bigram[0] + 1, self.hidden)))
        return specs + (self.norm.param_specs() if self.norm else [])

    def state_need(self):
        return {"previous": ((), torch.int32)} if self.bigram else {}

    def load(self, tensors):
        self.table = to_compute(tensors[self.name], self.ctx)
        if self.bigram:
            self.bigram_table = to_compute(tensors[self.bigram_name], self.ctx).to(self.table.dtype)
        if self.norm:
            self.norm.load(tensors)
            self.norm_weight = self.norm.weight.to(torch.float32).contiguous()

    def forward(self, batch, state, copy=None):
        x = torch.empty(batch.tokens.numel(), self.hidden, dtype=torch.float32, device=batch.tokens.device)
        bigram = (self.bigram_table, *self.bigram, state["previous"]) if self.bigram else None
        return ops.embedding_rows(self.table, batch, x, self.scale, bigram, self.norm_weight, self.norm.eps if self.norm else 0.0, copy)


class StreamsTokenEmbedding(Part):
    """A token embedding into `streams` residual streams: every token's row of the 32-bit stream tensor holds `streams`
    copies of its embedding, [T, streams * hidden_size]. params: name, vocab_size, hidden_size, streams."""

    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        self.name, self.vocab, self.hidden = params["name"], int(params["vocab_size"]), int(params["hidden_size"])
        self.streams = int(params["streams"])
        self.table = None

    def param_specs(self):
        return [ParamSpec(self.name, (self.vocab, self.hidden))]

    def load(self, tensors):
        self.table = to_compute(tensors[self.name], self.ctx)

    def forward(self, tokens):
        x = torch.empty(tokens.numel(), self.hidden, dtype=torch.float32, device=tokens.device)
        ops.embedding(self.table, tokens, x)
        if self.streams == 1:
            return x
        return ops.streams_expand(x, torch.empty(tokens.numel(), self.streams * self.hidden, dtype=torch.float32,
                                                 device=tokens.device), self.streams)


class LMHead(Part):
    """params: name (its own tensor) or tied_to (the embedding's tensor name), vocab_size, hidden_size, scale (multiplies
    the 32-bit logits; default 1)."""

    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        self.tied = params.get("tied_to")
        self.name = self.tied or params["name"]
        self.vocab, self.hidden = int(params["vocab_size"]), int(params["hidden_size"])
        self.scale = float(params.get("scale", 1.0))
        self.weight = None

    def param_specs(self):
        return [] if self.tied else [ParamSpec(self.name, (self.vocab, self.hidden))]

    def load(self, tensors):
        self.weight = ops.Weight(to_compute(tensors[self.name], self.ctx))

    def weight_bytes(self):
        return self.weight.nbytes

    def forward(self, xn):
        logits = torch.empty(xn.shape[0], self.vocab, dtype=torch.float32, device=xn.device)
        if xn.shape[0]:
            ops.linear(xn, self.weight, logits)
            if self.scale != 1.0:
                ops.scale_bias_rows(logits, self.scale)
        return logits


register_part("embedding", "token", TokenEmbedding)
register_part("embedding", "token_position", ScaledPositionEmbedding)
register_part("embedding", "token_normed", NormedTokenEmbedding)
register_part("embedding", "token_bigram", BigramTokenEmbedding)
register_part("embedding", "token_streams", StreamsTokenEmbedding)
register_part("head", "linear", LMHead)
