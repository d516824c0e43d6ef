"""Python front-ends of csrc/seq/ssd_ops.cu (ctypes -> libgllm_b200.so): the Mamba-2 recurrence (one-token step, chunked
tensor-core form), the gate before a grouped norm, the gated per-layer token input, cos / sin rows of a step. No
fallback: a missing library on a GPU box raises."""
from __future__ import annotations

from ctypes import c_float, c_int, c_long, c_void_p
from typing import Optional

import torch

from gllm_b200.ops import lib as _lib
from gllm_b200.ops import sm100, sm100_seq
from gllm_b200.ops.lib import check, stream_ptr
from gllm_b200.ops.sm100_seq import _f32, _p

_declared = False
_CHUNK_MIN_TOKENS = 2      # portions at least this long (on average) run in the chunked form


def _L():
    global _declared
    L = _lib.load()
    if not _declared:
        P, I, G, F = c_void_p, c_int, c_long, c_float
        scan = [P, G, P, G, P, G, P, G, P, P, P, P, P, P, P, I, I, I, I, I, P]
        sigs = {
            "gllm_ssd_rotary_angles": [P, P, I, P, I, P],
            "gllm_ssd_gelu_gate_embed": [P, G, P, I, P, G, I, P, I, I, I, P],
            "gllm_ssd_gate_then_norm": [P, I, P, G, P, I, F, P, G, I, I, P],
            "gllm_ssd_step": scan + [I, P],
            "gllm_ssd_chunk": scan + [P],
        }
        for name, args in sigs.items():
            fn = getattr(L, name)
            fn.argtypes, fn.restype = args, c_int
        _declared = True
    return L


def rotary_angles(positions: torch.Tensor, freqs: torch.Tensor) -> torch.Tensor:
    assert positions.dim() == 1 and positions.dtype == torch.int32 and freqs.dtype == torch.float64
    t, n = positions.shape[0], freqs.shape[0]
    out = torch.empty(t, 2 * n, dtype=torch.float32, device=positions.device)
    check(_L().gllm_ssd_rotary_angles(_p(positions), _p(freqs), n, _p(out), t, stream_ptr()), "ssd_rotary_angles")
    sm100._count()
    return out


def gelu_gate_embed(g: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, col0: int) -> torch.Tensor:
    t, dim = g.shape
    assert g.stride(1) == 1 and table.stride(1) == 1 and table.dtype == g.dtype and ids.dtype == torch.int32
    assert 0 <= col0 and col0 + dim <= table.shape[1], (col0, dim, tuple(table.shape))
    out = torch.empty(t, dim, dtype=g.dtype, device=g.device)
    check(_L().gllm_ssd_gelu_gate_embed(_p(g), g.stride(0), _p(ids), table.shape[0], _p(table), table.stride(0), col0,
                                        _p(out), t, dim, _f32(g), stream_ptr()), "ssd_gelu_gate_embed")
    sm100._count()
    return out


def gate_then_norm(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, group: int, eps: float,
                   out: Optional[torch.Tensor] = None, out_dtype=None) -> torch.Tensor:
    t, n = o.shape
    assert o.dtype == torch.float32 and o.is_contiguous() and gate.stride(1) == 1 and gate.shape == (t, n)
    assert w.dtype == torch.float32 and w.is_contiguous() and w.shape == (n,) and n % group == 0
    if out is None:
        out = torch.empty(t, n, dtype=out_dtype or gate.dtype, device=o.device)
    assert out.stride(1) == 1 and out.dtype == gate.dtype and out.shape == (t, n)
    check(_L().gllm_ssd_gate_then_norm(_p(o), n, _p(gate), gate.stride(0), _p(w), int(group), float(eps), _p(out),
                                       out.stride(0), t, _f32(gate), stream_ptr()), "ssd_gate_then_norm")
    sm100._count()
    return out


def ssd_scan(x, b, c, dt, neg_a, dt_bias, d_skip, state, rec_slots, seq_lens, query_start_loc, heads, groups, nstate,
             v_dim, num_decode_seqs: int = 0, max_q_len: Optional[int] = None, force: Optional[str] = None):
    """The first `num_decode_seqs` sequences (one token each) on the step kernel, the rest in the chunked form (bf16) or on
    the token-serial matrix-state kernel (fp32 operands, unaligned sizes). `force`: "serial" | "step" | "chunk" for all
    sequences."""
    t, nseq = x.shape[0], seq_lens.shape[0]
    for y in (x, b, c, dt):
        assert y.stride(1) == 1 and y.dtype == x.dtype
    assert state is None or (state.dtype == torch.float32 and state.is_contiguous())
    for y in (neg_a, dt_bias, d_skip):
        assert y.dtype == torch.float32 and y.is_contiguous() and y.shape == (heads,)
    assert heads % groups == 0
    out = torch.empty(t, heads * v_dim, dtype=torch.float32, device=x.device)
    L, st = _L(), stream_ptr()

    def args(s0, n):
        return (_p(x), x.stride(0), _p(b), b.stride(0), _p(c), c.stride(0), _p(dt), dt.stride(0), _p(neg_a),
                _p(dt_bias), _p(d_skip), _p(state), _p(rec_slots[s0:]) if rec_slots is not None else None,
                _p(seq_lens[s0:]), _p(query_start_loc[s0:]), n, heads, groups, nstate, v_dim, _p(out))

    def serial(s0, n):
        sm100_seq.linear_state_scan(c, b, x, None, dt, neg_a, dt_bias, None, state,
                                    rec_slots[s0:s0 + n] if rec_slots is not None else None, seq_lens[s0:s0 + n],
                                    query_start_loc[s0:s0 + n + 1], heads, groups, nstate, v_dim, False, False, 1.0,
                                    False, step=True, d_skip=d_skip, out=out)

    def run(kind, s0, n):
        if n <= 0:
            return
        rc = 2
        if kind == "step":
            rc = L.gllm_ssd_step(*args(s0, n), _f32(x), st)
        elif kind == "chunk" and x.dtype == torch.bfloat16:
            rc = L.gllm_ssd_chunk(*args(s0, n), st)
        if rc == 2:                          # sizes outside that kernel's envelope
            assert force is None or kind == "serial", f"ssd_scan: {kind} does not take these sizes"
            return serial(s0, n)
        check(rc, "ssd_" + kind)
        sm100._count()

    if force is not None:
        run(force, 0, nseq)
        return out
    nd = min(int(num_decode_seqs), nseq)
    run("step", 0, nd)
    rest = nseq - nd
    run("chunk" if (max_q_len is None or max_q_len >= _CHUNK_MIN_TOKENS) else "serial", nd, rest)
    return out
