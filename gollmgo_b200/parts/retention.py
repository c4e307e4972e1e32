"""Retention: a recurrent mixer whose state per head is a matrix S [d, dv] with one fixed decay g_h,

    S <- g_h S + k v^T,        o = S^T q,

with q = Wq x and k = Wk x rotated by the token's position (``position``: a rotation or none), k times
head_dim^-1/2 after it, and v = Wv x; no softmax and no denominator.  Each head's o is divided by its root
mean square (no weight), the heads together are multiplied by silu(Wg x) and projected.

State per request, in its state slot: S in float32 [heads, dv, d].  Nothing is paged.  Everything between
the projections and the gated rows is float32 (csrc/retention.cu).

params: hidden_size, num_heads, head_dim, v_head_dim, decay (one number in (0, 1] per head), position
(PartSpec), eps, out_buffer, names (optional dict: q, k, v, gate, o).
"""
from __future__ import annotations

import torch

from ..cache import FixedStateNeed
from ..csrc import ops
from ..weights import WeightSpec
from .linear import linear
from .registry import build_position, register_mixer

_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o"}


class Retention:
    def __init__(self, spec, ctx):
        self.ctx = ctx
        self.hidden = int(spec["hidden_size"])
        self.nh = int(spec["num_heads"])
        self.d = int(spec["head_dim"])
        self.dv = int(spec["v_head_dim"])
        self.eps = float(spec["eps"])
        self.decay = tuple(float(g) for g in spec["decay"])
        self.names = dict(_NAMES, **(spec.get("names") or {}))
        self.out_buffer = spec.get("out_buffer") or "mixer_out"
        self.position = build_position(spec["position"], ctx)
        if len(self.decay) != self.nh:
            raise ValueError(f"{len(self.decay)} decays for {self.nh} heads")
        if not all(0.0 < g <= 1.0 for g in self.decay):
            raise ValueError("a decay lies in (0, 1]")
        if self.d > 256:
            raise ValueError(f"key size {self.d} is beyond what the recurrence kernel takes (256)")
        if hasattr(self.position, "apply") or float(getattr(self.position, "magnitude", 1.0)) != 1.0:
            raise TypeError("retention takes a plain rotation or none")
        pad8 = lambda n: -(-n // 8) * 8
        self.row_width = self.nh * (2 * self.d + self.dv)
        self.gate_col = pad8(self.row_width)
        self.proj_width = pad8(self.gate_col + self.nh * self.dv)
        ws, T = ctx.workspace, ctx.max_tokens
        ws.reserve("ret_proj", T * self.proj_width, ctx.act_dtype)
        ws.reserve("ret_rows", T * self.row_width, torch.float32)
        ws.reserve("ret_o", T * self.nh * self.dv, torch.float32)
        ws.reserve("ret_y", T * self.nh * self.dv, ctx.act_dtype)
        ws.reserve(self.out_buffer, T * self.hidden, ctx.act_dtype)
        self.ones = torch.ones(T, self.nh, dtype=torch.float32, device=ctx.device)
        self.decay_rows = torch.tensor(self.decay, dtype=torch.float32, device=ctx.device).expand(T, self.nh).contiguous()
        self.w_proj = self.w_o = None

    def cache_need(self):
        return FixedStateNeed((self.nh, self.dv, self.d), "float32")

    def weights(self):
        n, H, qk, vv = self.names, self.hidden, self.nh * self.d, self.nh * self.dv
        return {n["q"]: WeightSpec((qk, H)), n["k"]: WeightSpec((qk, H)), n["v"]: WeightSpec((vv, H)),
                n["gate"]: WeightSpec((vv, H)), n["o"]: WeightSpec((H, vv))}

    def load(self, get):
        n = self.names
        parts = [get(n[x]) for x in ("q", "k", "v")]
        gate = get(n["gate"])
        dt = torch.float32 if any(p.dtype == torch.float32 for p in parts + [gate]) else parts[0].dtype
        w = torch.zeros(self.proj_width, self.hidden, dtype=dt, device=gate.device)
        w[:self.row_width] = torch.cat([p.to(dt) for p in parts], dim=0)
        w[self.gate_col:self.gate_col + self.nh * self.dv] = gate.to(dt)
        self.w_proj = w.contiguous()
        self.w_o = get(n["o"]).contiguous()

    def forward(self, x, batch, cache, writes_cache=True, then=None):
        T, ws, H = x.shape[0], self.ctx.workspace, self.nh
        state = cache
        proj = linear(x, self.w_proj, ws.get("ret_proj", T, self.proj_width))
        rows = ws.get("ret_rows", T, self.row_width)
        ops.retention_rows(proj, batch.positions, self.position.rope_table(), self.position.interleaved, H, self.d, self.dv,
                           self.d ** -0.5, rows)
        o = ws.get("ret_o", T, H * self.dv)
        ops.delta_recur(rows, self.ones[:T], self.decay_rows[:T], state, batch.cu_q_lens, batch.context_lens,
                        batch.state_slots, batch.num_seqs, H, H, self.d, self.dv, o, plain=True)
        y = ws.get("ret_y", T, H * self.dv)
        ops.delta_out(o, proj[:, self.gate_col:self.gate_col + H * self.dv], None, self.eps, H, self.dv, y)
        return linear(y, self.w_o, ws.get(self.out_buffer, T, self.hidden), then)


register_mixer("retention", Retention)
