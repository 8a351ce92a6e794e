"""Choice of kernel form by the shape of a step, shared by the models that serve flat token batches (`legavik`, `totatar`)."""
from __future__ import annotations

import torch

from . import ops
from .state import BatchMeta

TILES_MIN_TOKENS = 64           # a step with fewer tokens, or fewer than 16 per sequence, is decode-shaped
PROMPT_TILES_MIN_CTAS = 64      # (64-token blocks x heads) from which a prompt portion takes the tile form of its attention


def attend_window(qf: torch.Tensor, cache_k: torch.Tensor, cache_v: torch.Tensor, out: torch.Tensor, meta: BatchMeta, window: int,
                  scale: float, *, tiles: bool, min_tokens: int = TILES_MIN_TOKENS, min_ctas: int = PROMPT_TILES_MIN_CTAS, **kw) -> None:
    """Softmax attention of the step's queries qf [T, H, D] over a layer's cache rows (window, kept tokens, sink, gates: see
    `ops.seq_window_attention`). tiles: whether the tensor-core forms may be taken -- 64 tokens per CTA with the keys through shared memory
    once one sequence's portion is long enough, 16 tokens per CTA for other prompt-shaped batches, the heads of a group as rows for
    decoding; sizes they do not cover, and float32, take the plain form."""
    T, H, D = qf.shape
    G, DV = cache_v.shape[2], cache_v.shape[3]
    if tiles:
        prompt_shaped = T >= min_tokens and T >= 16 * len(meta.segments)
        if prompt_shaped and len(meta.segments) == 1 and ((T + 63) // 64) * H >= min_ctas and \
                ops.seq_prompt_attention_mma_supported(out.dtype, D, 0, DV):
            ops.seq_prompt_attention_mma(qf, cache_k, None, cache_v, out, meta.segments[0][1], meta.segments[0][2], window, scale, **kw)
            return
        if ops.seq_window_attention_mma_supported(out.dtype, D, 0, DV, H, G, prompt_shaped):
            ops.seq_window_attention_mma(qf, cache_k, None, cache_v, out, meta.table, window, scale, prompt_shaped, **kw)
            return
    ops.seq_window_attention(qf, None, cache_k, cache_v, out, meta.table, window, scale, **kw)


def run_experts(h: torch.Tensor, gate_up: torch.Tensor, down: torch.Tensor, idx: torch.Tensor, pair: torch.Tensor, experts: int, ff: int,
                *, tiles: bool, limit: float = 0.0, act: str = "silu") -> None:
    """Every chosen expert of every token into pair [T, top, W]: grouped tensor-core tiles once an expert sees several rows on average,
    the row-per-CTA form for a handful of tokens."""
    if tiles and idx.numel() >= 4 * experts and ops.moe_expert_grouped_supported(h, ff):
        ops.moe_expert_grouped(h, gate_up, down, idx, pair, experts, ff, limit, act=act)
    else:
        ops.moe_expert_tokens(h, gate_up, down, idx, pair, experts, ff, limit, act=act)
