"""A selective scan mixer (a state-space layer of the Mamba-1 kind).  One product makes [x | z] (``inner`` channels
each); x passes a short causal convolution per channel (with bias) and SiLU; a second product of x makes [low | B | C]
(``dt_rank`` and twice ``state`` values, the same B and C for all channels), a third one of low the step sizes:

    dt = softplus(W_dt low + b);   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = S[c] . C + D_c x_c

with A = -exp(A_log); y is multiplied by silu(z) and projected back.

State per request, in its state slot: S in float32 [inner, state] and the last taps - 1 inputs of the convolution
[taps - 1, inner].  Nothing is paged.  Between the products there are two kernels (csrc/selective_scan.cu): the
convolution, and the recurrence from the products' rows to the gated rows, in float32; in steps of few single tokens the
latter makes the step sizes' product itself.

params: hidden_size, inner, state, dt_rank, conv (taps), out_buffer, names (optional dict: in, conv, conv_bias, x, dt,
dt_bias, A_log, D, o).
"""
from __future__ import annotations

import math
import os

import torch

from ..cache import FixedStateNeed
from ..csrc import ops
from ..weights import WeightSpec
from .linear import linear
from .registry import register_mixer

_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "x": "x", "dt": "dt", "dt_bias": "dt.b", "A_log": "A_log",
          "D": "D", "o": "o"}
# Steps of at most this many single tokens make the step sizes inside the recurrence (every token reads W_dt again).
FUSE_DT_TOKENS = int(os.environ.get("GOLLMGO_B200_SCAN_FUSE_DT", "8"))


def _up8(n):
    return -(-n // 8) * 8


class SelectiveScanMixer:
    def __init__(self, spec, ctx):
        self.ctx = ctx
        self.hidden = int(spec["hidden_size"])
        self.inner = int(spec["inner"])
        self.n = int(spec["state"])
        self.rank = int(spec["dt_rank"])
        self.taps = int(spec["conv"])
        self.names = dict(_NAMES, **(spec.get("names") or {}))
        self.out_buffer = spec.get("out_buffer") or "mixer_out"
        if self.n > ops.SCAN_MAX_STATE:
            raise ValueError(f"{self.n} states a channel are beyond what the scan takes ({ops.SCAN_MAX_STATE})")
        if not (1 <= self.taps <= 64):
            raise ValueError(f"{self.taps} taps are outside 1..64")
        self.low_width = self.rank + 2 * self.n
        self.low_padded = _up8(self.low_width)                # rows of zeros: the product's rows start on 16-byte borders
        ws, T = ctx.workspace, ctx.max_tokens
        ws.reserve("scan_proj", T * 2 * self.inner, ctx.act_dtype)
        ws.reserve("scan_x", T * self.inner, ctx.act_dtype)
        ws.reserve("scan_low", T * self.low_padded, ctx.act_dtype)
        ws.reserve("scan_dt", T * self.inner, ctx.act_dtype)
        ws.reserve("scan_out", T * self.inner, ctx.act_dtype)
        ws.reserve(self.out_buffer, T * self.hidden, ctx.act_dtype)
        self.w_in = self.w_x = self.w_dt = self.w_o = None
        self.conv_w = self.conv_b = self.dt_b = self.a2 = self.d_skip = None

    def cache_need(self):
        need = [FixedStateNeed((self.inner, self.n), "float32")]
        if self.taps > 1:
            need.append(FixedStateNeed((self.taps - 1, self.inner), "float32"))
        return tuple(need)

    def weights(self):
        n, I = self.names, self.inner
        return {n["in"]: WeightSpec((2 * I, self.hidden)),
                n["conv"]: WeightSpec((I, self.taps), init="taps"),
                n["conv_bias"]: WeightSpec((I,), init="normal"),
                n["x"]: WeightSpec((self.low_width, I)),
                n["dt"]: WeightSpec((I, self.rank)),
                n["dt_bias"]: WeightSpec((I,), init="normal"),
                n["A_log"]: WeightSpec((I, self.n)),
                n["D"]: WeightSpec((I,), init="normal"),
                n["o"]: WeightSpec((self.hidden, I))}

    def load(self, get):
        n = self.names
        self.w_in = get(n["in"]).contiguous()
        w = get(n["x"])
        if self.low_padded != self.low_width:
            w = torch.cat([w, torch.zeros(self.low_padded - self.low_width, self.inner, dtype=w.dtype, device=w.device)])
        self.w_x = w.contiguous()
        self.w_dt = get(n["dt"]).contiguous()
        self.w_o = get(n["o"]).contiguous()
        self.conv_w = get(n["conv"]).float().contiguous()
        self.conv_b = get(n["conv_bias"]).float().contiguous()
        self.dt_b = get(n["dt_bias"]).float().contiguous()
        # exp(dt A) = 2^(dt A log2 e), the factor made in float64 and rounded once
        self.a2 = (-torch.exp(get(n["A_log"]).double()) * math.log2(math.e)).float().contiguous()
        self.d_skip = get(n["D"]).float().contiguous()

    def forward(self, x, batch, cache, writes_cache=True, then=None):
        T, I, ws = x.shape[0], self.inner, self.ctx.workspace
        state, conv_state = cache[0], cache[1] if self.taps > 1 else None
        B = batch.num_seqs
        proj = linear(x, self.w_in, ws.get("scan_proj", T, 2 * I))
        xc = ws.get("scan_x", T, I)
        ops.scan_conv(proj, self.conv_w, self.conv_b, conv_state, batch.cu_q_lens, batch.context_lens, batch.state_slots, B, xc)
        low = linear(xc, self.w_x, ws.get("scan_low", T, self.low_padded))
        single = T == B
        fuse = single and T <= FUSE_DT_TOKENS and self.w_dt.dtype == xc.dtype
        v = None if fuse else linear(low[:, :self.rank], self.w_dt, ws.get("scan_dt", T, I))
        out = ws.get("scan_out", T, I)
        ops.selective_scan(xc, proj, low, self.rank, v, self.w_dt if fuse else None, self.dt_b, self.a2, self.d_skip, state,
                           conv_state, self.taps, batch.cu_q_lens, batch.context_lens, batch.state_slots, B, single, out)
        return linear(out, self.w_o, ws.get(self.out_buffer, T, self.hidden), then)


register_mixer("mamba1", SelectiveScanMixer)
