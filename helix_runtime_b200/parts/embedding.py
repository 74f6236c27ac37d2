"""Token embedding and the output head.

Embedding: ``hidden[t] = table[id[t]] * scale`` widened into the float32 residual stream
(src/model/cpu_llama.cpp:21-27, 49); with the parameter ``norm`` (a norm's part spec) the
looked-up rows pass that norm, float32 in and out.  With the parameter ``pairs`` (``buckets``,
``mul_prev``, ``mul_cur``) a row of a second table (tensor ``pairs`` ``[buckets + 1, hidden]``) is
added, number ``(previous id * mul_prev + id * mul_cur) mod buckets``, the last one for a sequence's
first token; the id in front of a request's portion is per-request state.  Head: ``logits = x @ head.T`` in float32
(src/model/cpu_llama.cpp:107); when the checkpoint has no head tensor and ties its
embeddings the table stands in (tools/convert_hf_llama.py:497-510).  With the parameter
``softcap`` the logits run into a level, ``softcap * tanh(logits / softcap)``, in the product's
epilogue.
"""
from __future__ import annotations

from typing import List, Mapping, Optional

import torch

from ..cache.manager import StateNeed
from ..config.spec import PartSpec
from ..ops import library as ops
from ..weights.loader import TensorRequest
from .base import Part, StepContext, build_part, register_part
from .linear import Weight, project


class TokenEmbedding(Part):
    def __init__(self, spec: PartSpec, hidden_size: int) -> None:
        super().__init__(spec, hidden_size)
        self.vocab_size = int(spec["vocab_size"])
        # the looked-up row times this constant, in float32 (1: the row as it is)
        self.scale = float(spec.get("scale", 1.0))
        self.name = spec.tensors["weight"]
        self.table: Optional[torch.Tensor] = None
        norm = spec.get("norm")
        self.norm = None if norm is None else build_part("norm", norm, hidden_size)
        pairs = spec.get("pairs")
        self.pairs = None if pairs is None else {key: int(pairs[key]) for key in
                                                 ("buckets", "mul_prev", "mul_cur")}
        if self.pairs is not None and self.pairs["buckets"] < 1:
            raise ValueError("the table of pairs has at least one bucket")
        self.pairs_name = spec.tensors.get("pairs")
        self.pair_table: Optional[torch.Tensor] = None

    def state_need(self) -> Optional[StateNeed]:
        """One number per request, when a token's row depends on the token before it."""
        return None if self.pairs is None else StateNeed((1,), torch.int32)

    def tensor_requests(self) -> List[TensorRequest]:
        requests = [TensorRequest(self.name, (self.vocab_size, self.hidden_size), role="embedding")]
        if self.pairs is not None:
            requests.append(TensorRequest(self.pairs_name, (self.pairs["buckets"] + 1, self.hidden_size),
                                          role="embedding"))
        if self.norm is not None:
            requests += self.norm.tensor_requests()
        return requests

    def bind(self, tensors: Mapping[str, torch.Tensor], dtype, device) -> None:
        self.table = tensors[self.name].to(device=device, dtype=dtype).contiguous()
        if self.pairs is not None:
            self.pair_table = tensors[self.pairs_name].to(device=device, dtype=dtype).contiguous()
        if self.norm is not None:
            self.norm.bind(tensors, dtype, device)

    def _look_up(self, ctx: StepContext, out: torch.Tensor, state: Optional[torch.Tensor]) -> None:
        n = ctx.n_tokens
        if self.pairs is None:
            ops.embed(self.table, ctx.token_ids[:n], out[:n], ctx.status, self.scale)
        else:
            ops.embed_pairs(self.table, self.pair_table, ctx.token_ids, ctx.positions,
                            ctx.token_request, ctx.request_slot, ctx.request_start, state, out, n,
                            status=ctx.status, scale=self.scale, **self.pairs)

    def forward(self, ctx: StepContext, residual: torch.Tensor,
                state: Optional[torch.Tensor] = None) -> None:
        """``residual[:n]`` = the tokens' rows.  ``state`` ``[slots, 1]``: the previous tokens, when the
        embedding keeps them (``state_need``); a call moves them on, so it is made once a step."""
        if self.norm is None:
            self._look_up(ctx, residual, state)
            return
        looked_up = ctx.workspace.get(f"embedding.rows/{self.hidden_size}",
                                      (ctx.capacity, self.hidden_size), torch.float32)
        self._look_up(ctx, looked_up, state)
        self.norm.forward(ctx, looked_up, residual)     # a float32 output: the norm stores float32


class LmHead(Part):
    def __init__(self, spec: PartSpec, hidden_size: int) -> None:
        super().__init__(spec, hidden_size)
        self.vocab_size = int(spec["vocab_size"])
        self.name = spec.tensors["weight"]
        self.fallback = spec.tensors.get("tied_to") if spec.get("tied", False) else None
        self.softcap = float(spec.get("softcap") or 0.0)       # 0: the logits as they are
        self.weight: Optional[Weight] = None

    def tensor_requests(self) -> List[TensorRequest]:
        return [TensorRequest(self.name, (self.vocab_size, self.hidden_size),
                              fallback=self.fallback)]

    def bind(self, tensors: Mapping[str, torch.Tensor], dtype, device) -> None:
        self.weight = Weight(tensors[self.name].to(device=device, dtype=dtype).contiguous())

    def weight_bytes(self) -> int:
        return self.weight.nbytes()

    def forward(self, ctx: StepContext, x: torch.Tensor, logits: torch.Tensor, rows: int) -> None:
        project(x, self.weight, logits, rows, ops.EPI_STORE_F32, ctx.status, softcap=self.softcap)


register_part("embedding", "token_table", TokenEmbedding)
register_part("lm_head", "linear", LmHead)
