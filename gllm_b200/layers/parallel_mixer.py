"""Mixers assembled from cores. A core (`RotaryChunkCore`, `GatedDeltaCore`, `DecayLinearCore`, ...) declares the rows
of the input projection it reads (`in_names`, `in_rows`), the width of what it hands to the output projection
(`n_out`), what it keeps in the cache (`cache_entry`) and a `core(inp, proj, cache, run_id, out, out_scale)` step.

`CoreMixer` wraps cores that read the same input: ONE input GEMM over the concatenated projection rows (with the
projections' biases in its epilogue, for cores that have them), each core
writes scale_i * result_i into its column slice of one buffer, ONE output GEMM over the concatenated output
projections — sum_i scale_i * o_i(core_i(h)). With a single core it is the plain mixer.

A gated feed-forward can be one more branch of the same sum (`ff`): silu(gate h) * (up h) fills its own columns of the
joint buffer, so a block whose mixer and feed-forward run side by side has one output GEMM,
mixer(h) + ff(h) = [core(h) | act(h)] [W_o | W_down]^T, summed in the accumulator. Its gate and up rows follow the cores'
rows in the input weight. Small batches (decode) run ONE input GEMM over all rows and a small activation kernel; larger
ones run the cores' rows and the gate / up rows apart, the latter with the tcgen05 GEMM's SiLU-gate epilogue (rows
interleaved per 128; bf16 on CUDA with ff % 128 == 0).
"""
from __future__ import annotations

from typing import Sequence

import torch
from torch import nn

from gllm_b200.layers import functional as Fn


_JOINT_INPUT_MAX_TOKENS = 128      # up to here one launch less is worth more than the fused activation


class CoreMixer(nn.Module):
    def __init__(self, hidden: int, cores: Sequence[nn.Module], names: Sequence[str], scales: Sequence[float], dtype,
                 device, ff: int = 0):
        super().__init__()
        self.cores = nn.ModuleList(cores)
        self.names, self.scales = list(names), [float(s) for s in scales]
        self.n_in = sum(c.n_in for c in cores)
        self.n_out = sum(c.n_out for c in cores)
        # a parallel feed-forward: `ff` more columns of the joint buffer (its slice starts at a multiple of 8)
        self.ff, self.ff_at = int(ff), (self.n_out + 7) // 8 * 8
        self.n_joint = self.ff_at + self.ff if ff else self.n_out
        self.ff_block = 128 if torch.device(device).type == "cuda" and dtype == torch.bfloat16 and ff and \
            ff % 128 == 0 and hidden % 8 == 0 else 0
        # the tensor-core GEMM wants N % 8 == 0; pad rows stay zero
        self.n_in_pad = (self.n_in + 7) // 8 * 8
        n_in_pad = self.n_in_pad + 2 * self.ff
        self.in_w = nn.Parameter(torch.zeros(n_in_pad, hidden, dtype=dtype, device=device), requires_grad=False)
        self.o_w = nn.Parameter(torch.zeros(hidden, self.n_joint, dtype=dtype, device=device), requires_grad=False)
        # biases of the input projection ('<projection>.b'), for cores that declare them (`bias_names`); other rows stay 0
        self.in_b = nn.Parameter(torch.zeros(n_in_pad, dtype=dtype, device=device), requires_grad=False) \
            if any(getattr(c, "bias_names", ()) for c in cores) else None
        self.uses_pages = any(c.uses_pages for c in cores)
        self.uses_state = any(c.uses_state for c in cores)

    def cache_entry(self):
        if len(self.cores) == 1:
            return self.cores[0].cache_entry()
        kv = [c.cache_entry() for c in self.cores if c.uses_pages]
        rec = [c.cache_entry() for c in self.cores if c.uses_state]
        assert len(kv) <= 1 and len(rec) <= 1, "one paged and one recurrent core per mixer"
        return {"kind": "multi", "kv": kv[0] if kv else None, "rec": rec[0] if rec else None}

    def forward(self, inp, h: torch.Tensor, cache, run_id: int) -> torch.Tensor:
        joint = torch.empty(h.shape[0], self.n_joint, dtype=h.dtype, device=h.device)
        if self.ff and self.ff_at > self.n_out:
            joint[:, self.n_out:self.ff_at].zero_()            # meets zero weight columns, must be finite
        if self.ff_block and h.shape[0] > _JOINT_INPUT_MAX_TOKENS and self.in_b is None:
            proj = Fn.linear_any(h, self.in_w[:self.n_in_pad])
            Fn.linear_silu_mul(h, self.in_w[self.n_in_pad:], joint[:, self.ff_at:])
        else:
            proj = Fn.linear_any(h, self.in_w, self.in_b)
            if self.ff:
                Fn.silu_mul(proj[:, self.n_in_pad:], joint[:, self.ff_at:], self.ff_block)
        ci = co = 0
        for c, s in zip(self.cores, self.scales):
            c.core(inp, proj[:, ci:ci + c.n_in], cache, run_id, joint[:, co:co + c.n_out], s)
            ci, co = ci + c.n_in, co + c.n_out
        return Fn.linear_any(joint, self.o_w)

    def load(self, reader, pre: str, put, ff_pre: str = ""):
        """Checkpoint names: '<pre><core name>.<projection>' ('<pre><projection>' for a nameless single core);
        '<ff_pre>{gate,up,down}' of a parallel feed-forward."""
        rows, cols, at = [], [], 0
        for c, name in zip(self.cores, self.names):
            p = pre + (name + "." if name else "")
            for n, r in zip(c.in_names, c.in_rows):
                t = reader.get(p + n)
                assert t.shape[0] == r, (p + n, tuple(t.shape), r)
                rows.append(t)
                if n in getattr(c, "bias_names", ()):
                    b = reader.get(p + n + ".b")
                    assert tuple(b.shape) == (r,), (p + n + ".b", tuple(b.shape), r)
                    self.in_b.data[at:at + r].copy_(b)
                at += r
            cols.append(reader.get(p + "o"))
            c.load_extra(reader, p, put)
        w = torch.cat(rows, 0)
        self.in_w.data[: w.shape[0]].copy_(w)
        if not self.ff:
            put(self.o_w, torch.cat(cols, 1))
            return
        from gllm_b200.ops import ref
        gu = torch.cat([reader.get(ff_pre + "gate"), reader.get(ff_pre + "up")], 0)
        put(self.in_w.data[self.n_in_pad:], ref.interleave_gate_up(gu, self.ff_block) if self.ff_block else gu)
        put(self.o_w.data[:, :self.n_out], torch.cat(cols, 1))
        put(self.o_w.data[:, self.ff_at:], reader.get(ff_pre + "down"))
