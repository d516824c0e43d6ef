"""Sliding-window grouped-query attention over the paged cache with an optional softmax sink.

Mechanism (parameters, so other designs can use it):
  * per-head RMS norm of queries and keys with one weight vector shared by all heads (`qk_norm`);
  * no positional rotation — scores depend on content only;
  * `window`: position i attends to j with 0 <= i - j < window (None = the whole past);
  * `use_sink`: one learned logit per query head joins the softmax denominator and carries no value;
  * `values="key"`: there is no value projection, the values are the keys as projected (before their norm). The
    K cache holds the normed keys and the V cache the raw keys, so the attention kernel itself is an ordinary
    paged K/V attention.
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn

from gllm_b200.layers import functional as Fn


class SinkWindowAttention(nn.Module):
    uses_pages = True
    state_shapes = None

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, scale: float, window: Optional[int],
                 eps: float, dtype, device, use_sink: bool = True, qk_norm: bool = True, values: str = "key"):
        super().__init__()
        assert values == "key", "only key-valued attention is implemented"
        assert heads % kv_heads == 0, (heads, kv_heads)
        self.hidden, self.heads, self.kv_heads, self.dim = hidden, heads, kv_heads, dim
        self.scale, self.window, self.eps = float(scale), window, eps

        def par(*shape, dt=dtype):
            return nn.Parameter(torch.zeros(*shape, dtype=dt, device=device), requires_grad=False)

        self.qk_w = par((heads + kv_heads) * dim, hidden)        # [q rows ; k rows]
        self.q_norm_w = par(dim) if qk_norm else None
        self.k_norm_w = par(dim) if qk_norm else None
        self.sink = par(heads, dt=torch.float32) if use_sink else None
        self.o_w = par(hidden, heads * dim)

    def cache_entry(self):
        return {"kind": "kv", "heads": self.kv_heads, "dim": self.dim}

    def forward(self, inp, h: torch.Tensor, cache, run_id: int) -> torch.Tensor:
        qk = Fn.linear_any(h, self.qk_w)
        hd = self.heads * self.dim
        if cache is None:      # memory probe without a cache
            return Fn.linear_any(qk[:, :hd].contiguous(), self.o_w)
        kc, vc = cache.k_cache[run_id], cache.v_cache[run_id]
        q = Fn.qk_norm_kv_write(qk, self.heads, self.kv_heads, self.dim, self.q_norm_w, self.k_norm_w, self.eps,
                                kc, vc, inp.slot_mapping)
        a = Fn.window_attention(q, kc, vc, inp, self.scale, self.heads, self.dim, self.window, self.sink)
        return Fn.linear_any(a, self.o_w)


class RotaryChunkCore(nn.Module):
    """Grouped-query softmax attention over the paged cache with
      * per-head RMS norm of q and k (weights shared by the heads), applied before the rotation (`qk_norm`);
      * rotary positions on the first `rot_dims` entries of each head, entry i paired with i + rot_dims / 2; with
        `rot_scaling` {factor, original, fast, slow} the pair frequencies are the YaRN blend of
        `ops.ref.pair_rotary_frequencies` and cos / sin carry its magnitude;
      * a mask made of the causal rule and, optionally, a sliding `window` and / or a `chunk`: position i sees j only
        if floor(i / chunk) == floor(j / chunk), chunks counted from the start of the sequence;
      * `softcap` > 0: every scaled score s becomes softcap * tanh(s / softcap);
      * `unit_sink`: the softmax denominator has one more term exp(0) = 1 that carries no value;
      * values of their own width `v_dim`;
      * `bias`: the q / k / v projections have biases (the mixer adds them in the joint projection);
      * `kv_from` (a layer index): the core has no key / value projections and no cache of its own; it reads the
        pages that layer wrote (rotated keys, values) with its own queries and mask;
      * `unit_qk`: q and k are divided by their root mean square per head, without a weight (a rotation keeps that
        norm, so the order of the two does not matter);
      * `turn_values`: the value of position j is rotated by j over its whole width (entry m with m + v_dim / 2,
        frequencies of `rot_base` over v_dim, unscaled) and cached so; the result at position i is turned back by i;
      * `dist_bias`: r1[h] ln(1 + r2[h] (i - j)) is taken off the scaled score (per-head numbers 'r1', 'r2');
      * `out_gate`: the heads' results are multiplied by sigmoid of one more projection of the input ('g');
      * `rot_scaling` with {factor, low, high, original}: the frequency bands of `ops.ref.banded_rotary_frequencies`;
        with a factor alone every frequency is divided by it;
      * `whole_norm`: the RMS norms of q and k run over the whole projection, before it is split into heads (weights
        'q.norm' [heads * dim], 'k.norm' [kv_heads * dim]);
      * `q_temp` (coef, every): the query at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1), after
        norm and rotation;
      * `dist_rows`, `dist_max`: a learned bias per head and distance bucket ('rel' [rows, heads], buckets of
        `ops.ref.distance_buckets`) is added to the scaled scores; kept expanded to one fp32 row per distance;
      * `v_mix`: every core with it but the first one to run in a step caches (1 - lam) v + lam v_first, v_first the
        first one's values of the same tokens (`inp.first_values`), lam a learned number ('vmix').
    With `unit_qk`, `turn_values`, bands or a linear scaling (or on request, `step_angles`) the cos / sin rows come from
    `inp.angles` (formed once per step by the model, see `angle_tables`) instead of from every layer's own kernel.
    A core in the sense of layers/parallel_mixer.py: it reads [q | k | v] rows of a joint projection."""
    uses_pages, uses_state = True, False

    def __init__(self, heads: int, kv_heads: int, dim: int, v_dim: int, scale: float, rot_dims: int, rot_base: float,
                 chunk: Optional[int], window: Optional[int], eps: float, dtype, device, qk_norm: bool = True,
                 rot_scaling: Optional[dict] = None, softcap: float = 0.0, unit_sink: bool = False,
                 bias: bool = False, kv_from: Optional[int] = None, unit_qk: bool = False, turn_values: bool = False,
                 dist_bias: bool = False, out_gate: bool = False, whole_norm: bool = False, q_temp=None,
                 dist_rows: int = 0, dist_max: float = 0.0, v_mix: bool = False, step_angles: bool = False):
        super().__init__()
        assert heads % kv_heads == 0, (heads, kv_heads)
        assert rot_dims % 2 == 0 and rot_dims <= dim, (rot_dims, dim)
        self.heads, self.kv_heads, self.dim, self.v_dim = heads, kv_heads, dim, v_dim
        self.scale, self.rot_dims, self.rot_base, self.chunk, self.window, self.eps = \
            float(scale), int(rot_dims), float(rot_base), chunk, window, eps
        self.softcap, self.kv_from = float(softcap or 0.0), kv_from
        if kv_from is None:
            self.in_names = ("q", "k", "v")
            self.in_rows = (heads * dim, kv_heads * dim, kv_heads * v_dim)
        else:
            self.in_names = ("q",)
            self.in_rows = (heads * dim,)
        self.unit_qk, self.turn_values, self.out_gate = bool(unit_qk), bool(turn_values), bool(out_gate)
        self.bias_names = self.in_names if bias else ()
        self.whole_norm = bool(whole_norm)
        self.q_temp = (float(q_temp[0]), int(q_temp[1])) if q_temp is not None else None
        assert not whole_norm or (qk_norm and kv_from is None)
        assert kv_from is None or (q_temp is None and not v_mix)
        assert not (unit_qk and qk_norm) and not ((unit_qk or turn_values) and kv_from is not None)
        assert not turn_values or v_dim % 2 == 0, v_dim
        if out_gate:
            self.in_names += ("g",)
            self.in_rows += (heads * v_dim,)
        if dist_bias:
            self.r1 = nn.Parameter(torch.zeros(heads, dtype=torch.float32, device=device), requires_grad=False)
            self.r2 = nn.Parameter(torch.zeros(heads, dtype=torch.float32, device=device), requires_grad=False)
        else:
            self.r1 = self.r2 = None
        self.n_in, self.n_out = sum(self.in_rows), heads * v_dim

        def par(n, dt=dtype):
            return nn.Parameter(torch.zeros(n, dtype=dt, device=device), requires_grad=False)

        self.q_norm_w = par(heads * dim if whole_norm else dim) if qk_norm else None
        self.k_norm_w = par(kv_heads * dim if whole_norm else dim) if qk_norm else None
        self.vmix = par(1, torch.float32) if v_mix else None
        self.mag = 1.0
        from gllm_b200.ops import ref
        if dist_rows:
            assert not dist_bias
            self.dist_rows, self.buckets = int(dist_rows), ref.distance_buckets(int(dist_rows), float(dist_max))
            self.dist_table = nn.Parameter(torch.zeros(len(self.buckets), heads, dtype=torch.float32, device=device),
                                           requires_grad=False)
        else:
            self.dist_table = None
        self.step_angles = bool(step_angles) or self.unit_qk or self.turn_values or \
            bool(rot_scaling and ("low" in rot_scaling or "original" not in rot_scaling))
        if self.step_angles:
            self.register_buffer("freqs", ref.banded_rotary_frequencies(rot_dims, rot_base, rot_scaling).to(device),
                                 persistent=False)
            self.register_buffer("v_freqs", ref.banded_rotary_frequencies(v_dim, rot_base).to(device)
                                 if turn_values else None, persistent=False)
        elif rot_scaling and rot_dims > 0:
            f, self.mag = ref.pair_rotary_frequencies(rot_dims, rot_base, rot_scaling, dtype=torch.float64)
            self.register_buffer("freqs", f.to(device), persistent=False)
        else:
            self.freqs = None
        if unit_sink:
            self.register_buffer("sink", torch.zeros(heads, dtype=torch.float32, device=device), persistent=False)
        else:
            self.sink = None

    def cache_entry(self):
        if self.kv_from is not None:
            return {"kind": "shared", "layer": int(self.kv_from)}
        return {"kind": "kv", "heads": self.kv_heads, "dim": self.dim, "vdim": self.v_dim}

    def angle_tables(self):
        """[(key, fp64 frequencies)] of the cos / sin rows this core reads from `inp.angles`; equal keys are equal
        tables, so layers that rotate alike share one."""
        if not self.step_angles:
            return []
        out = [(self._angle_key(f), f) for f in (self.freqs, self.v_freqs) if f is not None and f.numel()]
        return out

    @staticmethod
    def _angle_key(f):
        return tuple(f.tolist())

    def _angles(self, inp, name):
        f = getattr(self, name)
        if f is None or not f.numel():
            return None
        if name not in self.__dict__.setdefault("_keys", {}):
            self._keys[name] = self._angle_key(f)
        tabs = getattr(inp, "angles", None)
        if tabs is not None and self._keys[name] in tabs:
            return tabs[self._keys[name]]
        return Fn.rotary_angles(inp.positions, f)          # a core driven without its model

    def core(self, inp, proj, cache, run_id, out, out_scale=1.0):
        if cache is None:      # memory probe without a cache
            out.zero_()
            return out
        kc, vc = cache.k_cache[run_id], cache.v_cache[run_id]
        own = self.kv_from is None
        v_mix = None
        if self.vmix is not None:
            v = proj[:, (self.heads + self.kv_heads) * self.dim:][:, :self.kv_heads * self.v_dim]
            if getattr(inp, "first_values", None) is None:
                inp.first_values = v
            else:
                v_mix = (inp.first_values, self.vmix)
        if self.step_angles or self.r1 is not None or self.out_gate or self.whole_norm or self.q_temp is not None or \
                self.vmix is not None or self.dist_table is not None:
            ang = self._angles(inp, "freqs") if self.step_angles else None
            v_ang = self._angles(inp, "v_freqs") if self.step_angles else None
            q = Fn.qk_norm_rope_kv_write(proj, self.heads, self.kv_heads if own else 0, self.dim, self.v_dim,
                                         self.q_norm_w, self.k_norm_w, self.eps, inp.positions, self.rot_dims,
                                         self.rot_base, kc, vc, inp.slot_mapping, None if self.step_angles
                                         else self.freqs, self.mag, self.unit_qk, ang, v_ang, self.whole_norm,
                                         self.q_temp, v_mix)
            gate = proj[:, self.n_in - self.n_out:self.n_in] if self.out_gate else None
            return Fn.masked_attention(q, kc, vc, inp, self.scale, self.heads, self.dim, self.v_dim, self.window,
                                       self.chunk, self.sink, out_scale, out, self.softcap,
                                       (self.r1, self.r2) if self.r1 is not None else None, gate, v_ang,
                                       self.dist_table)
        q = Fn.qk_norm_rope_kv_write(proj, self.heads, self.kv_heads if own else 0, self.dim, self.v_dim,
                                     self.q_norm_w, self.k_norm_w, self.eps, inp.positions, self.rot_dims,
                                     self.rot_base, kc, vc, inp.slot_mapping, self.freqs, self.mag)
        return Fn.masked_attention(q, kc, vc, inp, self.scale, self.heads, self.dim, self.v_dim, self.window,
                                   self.chunk, self.sink, out_scale, out, self.softcap)

    def load_extra(self, reader, pre, put):
        if self.q_norm_w is not None:
            put(self.q_norm_w, reader.get(pre + "q.norm"))
            put(self.k_norm_w, reader.get(pre + "k.norm"))
        if getattr(self, "r1", None) is not None:
            put(self.r1, reader.get(pre + "r1").float())
            put(self.r2, reader.get(pre + "r2").float())
        if self.vmix is not None:
            put(self.vmix, reader.get(pre + "vmix").float().reshape(1))
        if self.dist_table is not None:
            rel = reader.get(pre + "rel")
            assert rel.shape[0] == self.dist_rows, (tuple(rel.shape), self.dist_rows)
            put(self.dist_table, rel.float()[torch.tensor(self.buckets)])
