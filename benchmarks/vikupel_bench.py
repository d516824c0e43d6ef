"""Side benchmark of the Vikupel design (`python bench.py --design vikupel`): prefill / decode throughput through
`LLM.generate` with random weights beside Saritar (the closest design: recurrent mixers and windowed attention on an
fp32 stream) and Qwen3 at equal width and depth, and the device time of the kernels the design added or extended
beside the like kernels of the existing paths. Helpers and conventions are those of design_bench.py."""
from __future__ import annotations

import json

import torch

from benchmarks.design_bench import _qwen3_cfg, _saritar_cfg, _throughput, _time


def vikupel_cfg(width, n_quads, vocab, head=128, window=1024):
    heads = max(width // head, 1)
    kv = max(heads // 4, 1)
    ff = {"kind": "dense", "ff": 3 * width // 2}
    mam = {"type": "mamba2", "mlp": ff,
           "mixer": {"heads": 2 * width // 64, "groups": min(8, 2 * width // 64), "state": 128, "vdim": 64, "conv": 4,
                     "norm_groups": min(8, 2 * width // 64)}}
    att = {"heads": heads, "kv_heads": kv, "dim": head, "vdim": head, "scale": head ** -0.5}
    win = {"type": "attention", "mlp": ff, "mixer": {**att, "mask": {"size": window}}}
    rot = {"base": 5e5, "dims": head, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    full = {"type": "attention_2", "mlp": ff, "mixer": {**att, "rot": rot}}
    return {"architecture": "Vikupel", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "residual_mult": 0.5,
            "token_side": {"dim": 128}, "layers": [mam, win, mam, full] * n_quads}


def _meta(qlens, ctx, ps, dev):
    B = len(qlens)
    qsl = torch.tensor([0] + torch.tensor(qlens).cumsum(0).tolist(), dtype=torch.int32, device=dev)
    sl = torch.tensor([q + ctx for q in qlens], dtype=torch.int32, device=dev)
    npp = (max(qlens) + ctx + ps - 1) // ps
    bt = torch.arange(B * npp, dtype=torch.int32, device=dev).reshape(B, npp)
    pos = torch.cat([torch.arange(ctx, ctx + q) for q in qlens]).to(torch.int32).to(dev)
    seqi = torch.cat([torch.full((q,), i) for i, q in enumerate(qlens)]).to(dev)
    slots = (bt[seqi, (pos // ps).long()] * ps + pos % ps).to(torch.int32)
    return B, qsl, sl, npp, bt, pos, slots


def kernels(peaks):
    from gllm_b200.ops import ref, sm100, sm100_seq as S, sm100_ssd as K
    dev, bf = "cuda", torch.bfloat16
    hbm = float(peaks.get("hbm_gbs", 6650.0))
    out = []

    def row(name, ms, nbytes, like=None, flops=None):
        r = {"kernel": name, "ms": round(ms, 4), "gbs": round(nbytes / ms / 1e6, 1),
             "frac_hbm": round(nbytes / ms / 1e6 / hbm, 3)}
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 2)
        if like:
            r["like"] = like
        out.append(r)

    # -- stream, token side ------------------------------------------------------------------------------------
    T, W, V = 8192, 4096, 32000
    x = torch.randn(T, W, device=dev)
    y, w1 = torch.randn(T, W, device=dev).to(bf), torch.ones(W, device=dev).to(bf)
    row("resid_norm, multiplier, no norm, emits the stream in bf16 8192 x 4096",
        _time(lambda: S.resid_norm(x, y, None, None, None, 1e-5, bf, True, y_mul=0.5)), T * W * (4 + 4 + 2 + 2))
    row("resid_norm, side norm + multiplier + next norm 8192 x 4096",
        _time(lambda: S.resid_norm(x, y, w1, None, w1, 1e-5, bf, y_mul=0.5)), T * W * (4 + 4 + 2 + 2))
    res = torch.randn(T, W, device=dev).to(bf)
    row("rmsnorm + residual (existing bf16 path)", _time(lambda: sm100.rmsnorm(y, w1, 1e-5, res)), T * W * 8,
        like="resid_norm")
    ids = torch.randint(0, V, (T,), dtype=torch.int32, device=dev)
    table, g = torch.randn(V, 8 * 128, device=dev).to(bf), torch.randn(T, 128, device=dev).to(bf)
    row("gelu_gate_embed 8192 x 128", _time(lambda: K.gelu_gate_embed(g, ids, table, 256)), T * 128 * 6)
    gg = torch.cat([g, g], 1)
    row("silu_and_mul (existing, same output)", _time(lambda: sm100.silu_and_mul(gg)), T * 128 * 6,
        like="gelu_gate_embed")
    del x, y, res

    # -- Mamba-2 -----------------------------------------------------------------------------------------------
    H, G, N, P = 128, 8, 128, 64
    inner, bc = H * P, G * N
    C = inner + 2 * bc
    for label, qlens in (("prefill 4 x 2048", [2048] * 4), ("decode 256 x 1", [1] * 256)):
        B, qsl, sl, _, _, _, _ = _meta(qlens, 100, 16, dev)
        Tt = sum(qlens)
        rs = torch.arange(B, dtype=torch.int32, device=dev)
        proj = torch.randn(Tt, inner + C + H, device=dev).to(bf)
        cw, cb, cst = torch.randn(C, 4, device=dev), torch.randn(C, device=dev), torch.zeros(B, 3, C, device=dev).to(bf)
        row("conv + silu, %d channels, 4 taps %s" % (C, label),
            _time(lambda: S.causal_conv_silu(proj[:, inner:], C, cw, cb, cst, rs, sl, qsl)), Tt * C * 4 + B * 3 * C * 4)
        xbc = S.causal_conv_silu(proj[:, inner:], C, cw, cb, cst, rs, sl, qsl)
        na, db, dk = -torch.rand(H, device=dev), torch.randn(H, device=dev) - 3, torch.randn(H, device=dev)
        st = torch.zeros(B, H, N, P, device=dev)
        nbytes = Tt * (C * 2 + H * 2) + Tt * inner * 4 + B * H * N * P * 8
        args = (xbc[:, :inner], xbc[:, inner:inner + bc], xbc[:, inner + bc:], proj[:, inner + C:], na, db, dk, st, rs,
                sl, qsl, H, G, N, P)
        nd = B if qlens[0] == 1 else 0
        row("ssd_scan (%s) %s" % ("step" if nd else "chunked, tensor cores", label),
            _time(lambda: K.ssd_scan(*args, num_decode_seqs=nd, max_q_len=max(qlens)), iters=5), nbytes,
            flops=5.0 * Tt * H * N * P)
        row("linear_state_kernel (existing token-serial form, same recurrence) " + label,
            _time(lambda: K.ssd_scan(*args, force="serial"), iters=3), nbytes, like="ssd_scan",
            flops=5.0 * Tt * H * N * P)
        o, nw = torch.randn(Tt, inner, device=dev), torch.ones(inner, device=dev)
        row("gate_then_norm, 8 parts of 1024 " + label,
            _time(lambda: K.gate_then_norm(o, proj[:, :inner], nw, inner // 8, 1e-5)), Tt * inner * 8)
        row("gated_group_norm (existing, same groups) " + label,
            _time(lambda: S.gated_group_norm(o, proj[:, :inner], nw.to(bf), inner // 8, 1e-5, "silu")), Tt * inner * 8,
            like="gate_then_norm")
        C1, N1, R1 = 8192, 16, 256
        xz, p1 = torch.randn(Tt, 2 * C1, device=dev).to(bf), torch.randn(Tt, R1 + 2 * N1, device=dev).to(bf)
        xc, dtr = torch.randn(Tt, C1, device=dev).to(bf), torch.randn(Tt, C1, device=dev).to(bf)
        A, Dk, b1 = -torch.rand(C1, N1, device=dev), torch.randn(C1, device=dev), torch.randn(C1, device=dev)
        ss = torch.zeros(B, N1, C1, device=dev)
        row("selective_scan (existing, Mamba-1, 8192 x 16) " + label,
            _time(lambda: S.selective_scan(xc, dtr, p1, xz, A, Dk, b1, ss, rs, sl, qsl, C1, N1, R1), iters=5),
            Tt * C1 * 8 + B * N1 * C1 * 8, like="ssd_scan", flops=5.0 * Tt * C1 * N1)
        del st, o, proj, xbc, args

    # -- attention ---------------------------------------------------------------------------------------------
    H, G, D, ps, win = 32, 8, 128, 16, 1024
    r1, r2 = torch.rand(H, device=dev) + 0.5, torch.rand(H, device=dev)
    fr = ref.banded_rotary_frequencies(D, 5e5, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}).to(dev)
    fv = ref.banded_rotary_frequencies(D, 5e5).to(dev)
    for label, qlens, ctx in (("prefill 4 x 2048", [2048] * 4, 0), ("decode 256 x 1 at 2048", [1] * 256, 2047)):
        B, qsl, sl, npp, bt, pos, slots = _meta(qlens, ctx, ps, dev)
        Tt = sum(qlens)
        kc, vc = (torch.randn(ref.kv_cache_shape(B * npp + 1, G, D, ps), device=dev).to(bf) for _ in range(2))
        qkvg = torch.randn(Tt, (2 * H + 2 * G) * D, device=dev).to(bf)
        row("rotary_angles (one table of 64 pairs, once per step) " + label, _time(lambda: K.rotary_angles(pos, fr)),
            Tt * (4 + D * 4))
        ang, va = K.rotary_angles(pos, fr), K.rotary_angles(pos, fv)
        row("rotary write, unit norm, rotated values " + label,
            _time(lambda: S.qk_norm_rope_kv_write(qkvg, H, G, D, D, None, None, 1e-5, pos, D, 5e5, kc, vc, slots, None,
                                                  1.0, True, ang, va)), Tt * (H + 2 * G) * D * 4 + Tt * D * 8)
        row("cache write without rotation (windowed layers) " + label,
            _time(lambda: S.qk_norm_rope_kv_write(qkvg, H, G, D, D, None, None, 1e-5, pos, 0, 5e5, kc, vc, slots)),
            Tt * (H + 2 * G) * D * 4)
        cs, qn = torch.randn(8192, D, device=dev), torch.ones(D, device=dev).to(bf)
        qq, kk, vv = (qkvg[:, a * D:b * D].unflatten(1, (b - a, D)) for a, b in ((0, H), (H, H + G), (H + G, H + 2 * G)))
        row("rope_kv_write (existing: table rotary + q/k norm + cache write) " + label,
            _time(lambda: sm100.rope_kv_write(qq, kk, vv, pos, cs, D, True, qn, qn, 1e-5, kc, vc, slots)),
            Tt * (H + 2 * G) * D * 4, like="rotary write")
        q, gate = torch.randn(Tt, H * D, device=dev).to(bf), qkvg[:, (H + 2 * G) * D:]
        nd = B if qlens[0] == 1 else 0

        def att(**kw):
            w = kw.pop("window", None)
            return _time(lambda: S.window_attention(q, kc, vc, bt, sl, qsl, pos, D ** -0.5, H, D, w, kw.get("sink"),
                                                    num_decode_seqs=nd, max_q_len=max(qlens), v_dim=D,
                                                    **{k: v for k, v in kw.items() if k != "sink"}), iters=5)

        def arow(name, ms, w, like=None):
            keys = sum(min(p + 1, w or 1 << 30) for ql in qlens for p in range(ctx, ctx + ql))
            r = {"kernel": name + " " + label, "ms": round(ms, 4), "tflops": round(4.0 * keys * H * D / ms / 1e9, 2)}
            out.append({**r, "like": like} if like else r)

        arow("attention, window 1024, distance bias, output gate", att(window=win, dist_bias=(r1, r2), gate=gate), win)
        arow("window attention with a sink (existing design, same window)", att(window=win, sink=torch.zeros(H, device=dev)),
             win, like="attention, window")
        arow("window attention on the mma.sync kernels", att(window=win, sink=torch.zeros(H, device=dev), tc=False), win,
             like="attention, window")
        arow("attention, full causal, values turned back", att(v_turn=va), None)
        arow("paged_attention (existing, full causal)",
             _time(lambda: sm100.paged_attention(q, kc, vc, bt, sl, qsl, D ** -0.5, H, D, nd, B, max(qlens),
                                                 max(qlens) + ctx), iters=3), None, like="attention, full causal")
        del kc, vc
    return out


def run(args, peaks):
    vocab = 32000
    rows = kernels(peaks)
    torch.cuda.empty_cache()
    sizes = []
    for width, quads in ((1024, 2), (2048, 2), (4096, 1)):
        heads = width // 128
        kv = max(heads // 4, 1)
        sizes.append({"width": width, "layers": 4 * quads,
                      "vikupel": _throughput(vikupel_cfg(width, quads, vocab), vocab, args.warmup, args.steps),
                      "saritar": _throughput(_saritar_cfg(width, 2 * quads, heads, kv, 128, 1024, 4 * width, vocab),
                                             vocab, args.warmup, args.steps),
                      "qwen3": _throughput(_qwen3_cfg(width, 4 * quads, heads, kv, 128, 3 * width, vocab), vocab,
                                           args.warmup, args.steps)})
    line = {"design": "vikupel", "dtype": "bf16", "data": "synthetic", "warmup": args.warmup, "steps": args.steps,
            "timing": "wall clock around LLM.generate with synchronize (sizes); CUDA events, L2 flushed (kernels)",
            "peaks": peaks, "sizes": sizes, "kernels": rows}
    print(json.dumps(line))
    return line
