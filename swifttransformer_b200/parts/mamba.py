"""The selective scan mixer (Mamba): a diagonal recurrence driven by the token itself.

With C inner channels and a state of N numbers per channel, zero when a request starts:

    [u | z]  = W_in h                              C columns each
    x        = silu(conv(u) + b)                   a short causal convolution over time, one filter per channel
    [r|B|G]  = W_x x                               ``dt_rank`` | N | N columns
    d        = softplus(W_dt r + b_dt)             the step sizes, one per channel
    S[c, n] <- exp(-d_c exp(A_log[c, n])) S[c, n] + d_c x_c B_n;    y_c = sum_n S[c, n] G_n + D_c x_c
    out      = W_o (y * silu(z))

Per request the mixer keeps the last taps - 1 rows of u and the state S, both float32, in state slots.  -exp(A_log) is
formed once, in double precision, when the weights are bound; W_x's product is written in float32, and the step sizes,
the recurrence, its read-out and the output gate are float arithmetic in the kernels.  Steps of single tokens: product
of W_dt, recurrence and gate are one kernel.  Portions longer than a chunk are scanned in chunks side by side
(``TokenChunkPlan``).
"""
from __future__ import annotations

import dataclasses
from typing import Any, Dict, List, Optional, Tuple

import numpy as np
import torch

from .. import ops
from ..weights.spec import MATRIX, VECTOR, ParamSpec
from .base import MIXERS, Delta, Mixer, RowTaker, StateSpec, StepPlan, stack_rows


@dataclasses.dataclass
class TokenChunks:
    chunks: Optional[torch.Tensor]      # int32 [n_chunks, 2] = (request, offset); None: no portion is longer than a chunk
    first: Optional[torch.Tensor]       # int32 [requests + 1]
    n_chunks: int
    chunk: int


class TokenChunkPlan(StepPlan):
    """The step's tokens in chunks of ``chunk`` tokens that do not cross requests, the chunks of a request side by side
    and in order, for recurrences that are scanned chunk by chunk.  A step whose portions all fit one chunk gets none."""

    PAD_OFFSET = 1 << 24               # past any request's tokens: such a chunk's block leaves at once

    def __init__(self, chunk: int):
        self.chunk = int(chunk)
        self.name = f"token_chunks_{self.chunk}"

    def _cap(self, n_cap: int, b_cap: int) -> int:
        return (n_cap + self.chunk - 1) // self.chunk + b_cap

    def words(self, n_cap: int, b_cap: int) -> int:
        return 2 * self._cap(n_cap, b_cap) + b_cap + 1

    def shape_key(self, lens, start, n_cap: int, b_cap: int) -> Tuple:
        return (self._cap(n_cap, b_cap) if len(lens) and int(lens.max()) > self.chunk else 0,)

    def fill(self, lens, q_start, start, out, n_cap: int, b_cap: int) -> Tuple:
        if not len(lens):
            # a step that is all padding: no chunk of any request
            cap = self._cap(n_cap, b_cap)
            out[0:2 * cap:2] = 0
            out[1:2 * cap:2] = self.PAD_OFFSET
            out[2 * cap:] = 0
            return (0,)
        if int(lens.max()) <= self.chunk:
            return (0,)
        cap = self._cap(n_cap, b_cap)
        counts = (lens + self.chunk - 1) // self.chunk
        first = np.zeros(len(lens) + 1, dtype=np.int32)
        np.cumsum(counts, out=first[1:])
        n = int(first[-1])
        req = np.repeat(np.arange(len(lens), dtype=np.int32), counts)
        out[0:2 * n:2] = req
        out[1:2 * n:2] = (np.arange(n, dtype=np.int32) - first[req]) * self.chunk
        out[2 * n:2 * cap:2] = 0
        out[2 * n + 1:2 * cap:2] = self.PAD_OFFSET
        out[2 * cap:2 * cap + len(first)] = first
        out[2 * cap + len(first):] = n
        return (n,)

    def view(self, dev: torch.Tensor, key: Tuple, n_cap: int, b_cap: int) -> TokenChunks:
        if key[0] == 0:
            return TokenChunks(None, None, 0, self.chunk)
        cap = self._cap(n_cap, b_cap)
        return TokenChunks(dev[:2 * key[0]], dev[2 * cap:2 * cap + b_cap + 1], key[0], self.chunk)


@MIXERS.register("mamba")
class Mamba(RowTaker, Mixer):
    """names: matrices {"in", "x", "dt", "o"} ([out, in]), "conv" [inner, taps], "conv_bias" [inner], "dt_bias" [inner],
    "A_log" [inner, state], "D" [inner]."""

    def __init__(self, hidden: int, inner: int, state: int, dt_rank: int, conv_taps: int, names: Dict[str, str],
                 float_out: bool = False, chunk: int = ops.MAMBA_CHUNK):
        if conv_taps < 1:
            raise ValueError("a convolution needs at least one tap")
        self.hidden, self.inner, self.n, self.rank, self.taps = hidden, inner, state, dt_rank, int(conv_taps)
        self.names, self.float_out = dict(names), bool(float_out)
        self._plan = TokenChunkPlan(chunk)
        self.extra_n = 0
        self.w_in = self.w_x = self.w_dt = self.w_o = self.conv_w = self.conv_b = self.A = self.D = self.dt_bias = None

    def param_specs(self) -> List[ParamSpec]:
        n, C = self.names, self.inner
        return [ParamSpec(n["in"], (2 * C, self.hidden), MATRIX), ParamSpec(n["conv"], (C, self.taps), VECTOR),
                ParamSpec(n["conv_bias"], (C,), VECTOR), ParamSpec(n["x"], (self.rank + 2 * self.n, C), MATRIX),
                ParamSpec(n["dt"], (C, self.rank), MATRIX), ParamSpec(n["dt_bias"], (C,), VECTOR),
                ParamSpec(n["A_log"], (C, self.n), VECTOR), ParamSpec(n["D"], (C,), VECTOR),
                ParamSpec(n["o"], (self.hidden, C), MATRIX)]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.names
        mats = [tensors.pop(n["in"])]
        if self.extra_rows is not None:
            mats.append(self.extra_rows)
            self.extra_n, self.extra_rows = self.extra_rows.shape[0], None
        self.w_in, off = stack_rows(mats)
        self.extra_off = off[-1]
        # the low-rank inputs are filled up to a multiple of eight with zero rows (and W_dt with zero columns)
        w_x, w_dt = tensors.pop(n["x"]), tensors.pop(n["dt"])
        self.w_x, (_, self.b_off) = stack_rows([w_x[:self.rank], w_x[self.rank:]])
        self.g_off = self.b_off + self.n
        self.w_dt = w_dt.new_zeros((self.inner, self.b_off))
        self.w_dt[:, :self.rank] = w_dt
        self.w_o = tensors.pop(n["o"])
        self.conv_w, self.conv_b = tensors[n["conv"]].contiguous(), tensors[n["conv_bias"]]
        self.A = -torch.exp(tensors.pop(n["A_log"]).to(torch.float64)).to(torch.float32).contiguous()
        self.D, self.dt_bias = tensors[n["D"]], tensors[n["dt_bias"]]

    def cache_spec(self):
        # the convolution's last inputs, and the recurrent state
        return (StateSpec((self.taps - 1, self.inner), torch.float32), StateSpec((self.inner, self.n), torch.float32))

    def step_plan(self) -> StepPlan:
        return self._plan

    def forward(self, h: torch.Tensor, ctx: Any, cache: Any) -> Delta:
        tails, states = cache
        C, single = self.inner, bool(getattr(ctx, "single_tokens", False))
        proj = ops.linear(h, self.w_in)
        moves = single and tails.writable
        x = ops.conv_act(proj, C, self.conv_w, self.conv_b, "silu", tails.state, ctx.positions, ctx.seq_of_token,
                         ctx.q_start, ctx.slots, move_state=moves)
        if self.taps > 1 and tails.writable and not moves:
            ops.conv_state_update(proj, C, tails.state, ctx.positions, ctx.q_start, ctx.slots, ctx.n_seqs)
        xd = ops.linear(x, self.w_x, out_dtype=torch.float32)
        y = torch.empty_like(x)
        if single:
            ops.mamba_single(x, xd, self.b_off, self.g_off, self.w_dt, proj, C, self.A, self.D, self.dt_bias, states.state, y,
                             ctx.positions, ctx.seq_of_token, ctx.slots, write_state=states.writable)
        else:
            dt = ops.linear(ops.slice_rows(xd, 0, self.b_off, h.dtype), self.w_dt, out_dtype=torch.float32)
            plan = ctx.plan(self._plan.name)
            scratch = None
            if plan.n_chunks:
                scratch = ctx.scratch_f32(ops.mamba_scan_scratch(plan.n_chunks, C, self.n))
            ops.mamba_scan(x, dt, xd, self.b_off, self.g_off, proj, C, self.A, self.D, self.dt_bias, states.state, y,
                           ctx.positions, ctx.q_start, ctx.slots, ctx.n_seqs, write_state=states.writable,
                           chunks=plan.chunks, chunk_first=plan.first, n_chunks=plan.n_chunks, chunk=plan.chunk,
                           scratch=scratch)
        extra = proj[:, self.extra_off:self.extra_off + self.extra_n] if self.extra_n else None
        return Delta(ops.linear(y, self.w_o, out_dtype=torch.float32 if self.float_out else None), extra=extra)

    def param_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_x, self.w_dt, self.w_o, self.A))
