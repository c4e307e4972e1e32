"""Retention: a recurrent mixer whose state per head is a matrix S [d, dv] with one fixed decay g_h,

    S <- g_h S + k v^T,        o = S^T q,

with q = Wq x and k = Wk x rotated by the token's position (``position``: a rotation or none), k times
head_dim^-1/2 after it, and v = Wv x; no softmax and no denominator.  Each head's o is divided by its root
mean square (no weight), the heads together are multiplied by silu(Wg x) and projected.

State per request, in its state slot: S in float32 [heads, dv, d].  Nothing is paged.  Everything between
the projections and the gated rows is float32 (csrc/retention.cu): single decoded tokens in one kernel, prompt
portions in chunks whose states follow one another and whose rows are then all made at once.  Heads of more
than 512 values go token by token through the engine's plain linear recurrence (csrc/delta_rule.cu) instead.

params: hidden_size, num_heads, head_dim, v_head_dim, decay (one number in (0, 1] per head), position
(PartSpec), eps, out_buffer, names (optional dict: q, k, v, gate, o).
"""
from __future__ import annotations

import math

import torch

from ..cache import FixedStateNeed
from ..csrc import ops
from ..weights import WeightSpec
from .context import QueryTiles
from .linear import linear
from .registry import build_position, register_mixer

CHUNKS = QueryTiles(ops.RETENTION_CHUNK)          # the chunks of prompt portions

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
        ws.reserve("ret_y", T * self.nh * self.dv, ctx.act_dtype)
        ws.reserve(self.out_buffer, T * self.hidden, ctx.act_dtype)
        self.decays = torch.tensor(self.decay, dtype=torch.float32, device=ctx.device)
        self.log2_decays = torch.tensor([math.log2(g) for g in self.decay], dtype=torch.float32, device=ctx.device)
        self.chunked = self.dv <= ops.RETENTION_MAX_V
        if self.chunked:
            ws.reserve("ret_states", ops.retention_scratch_floats(T, ctx.max_seqs, self.nh, self.d, self.dv), torch.float32)
        else:
            ws.reserve("ret_o", T * self.nh * self.dv, torch.float32)
            ws.reserve("ret_beta", T * self.nh, torch.float32)
            ws.reserve("ret_decay", T * self.nh, torch.float32)
        self.w_proj = self.w_o = None

    def cache_need(self):
        return FixedStateNeed((self.nh, self.dv, self.d), "float32")

    def query_tiles(self):
        return [CHUNKS] if self.chunked else []

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
        T, ws, H, d, dv = x.shape[0], self.ctx.workspace, self.nh, self.d, self.dv
        state, kscale = cache, self.d ** -0.5
        table, pairs = self.position.rope_table(), self.position.interleaved
        proj = linear(x, self.w_proj, ws.get("ret_proj", T, self.proj_width))
        gate = proj[:, self.gate_col:self.gate_col + H * dv]
        y = ws.get("ret_y", T, H * dv)
        if batch.num_portions or not self.chunked:
            rows = ws.get("ret_rows", T, self.row_width)
            ops.retention_rows(proj, batch.positions, table, pairs, H, d, dv, kscale, rows)
        if not self.chunked:
            o, beta, decay = ws.get("ret_o", T, H * dv), ws.get("ret_beta", T, H), ws.get("ret_decay", T, H)
            beta.fill_(1.0)
            decay.copy_(self.decays.expand(T, H))
            ops.delta_recur(rows, beta, decay, state, batch.cu_q_lens, batch.context_lens, batch.state_slots, batch.num_seqs,
                            H, H, d, dv, o, plain=True)
            ops.delta_out(o, gate, None, self.eps, H, dv, y)
        else:
            if batch.num_portions:
                if CHUNKS not in batch.tiles:
                    raise RuntimeError("the step's batch was built without the index list this mixer declares in "
                                       "query_tiles(): give it to the BatchBuilder (query_tiles=...)")
                tiles = batch.tiles[CHUNKS]
                scratch = ws.get("ret_states", 1, ops.retention_scratch_floats(T, batch.num_seqs, H, d, dv))
                ops.retention_chunks(rows, self.log2_decays, state, scratch, tiles.seq, tiles.q0, tiles.count, batch.cu_q_lens,
                                     batch.context_lens, batch.state_slots, batch.num_seqs, gate, self.eps, H, d, dv, y)
            if batch.num_decode:
                ops.retention_decode(proj, self.gate_col, batch.positions, table, pairs, self.decays, state, batch.dec_seqs,
                                     batch.num_decode, batch.cu_q_lens, batch.context_lens, batch.state_slots, H, d, dv, kscale,
                                     self.eps, y)
        return linear(y, self.w_o, ws.get(self.out_buffer, T, self.hidden), then)


register_mixer("retention", Retention)
