"""Side benchmark of the Liverax design (`python bench.py --design liverax`): prefill / decode throughput through
`LLM.generate` with random weights beside Qwen3 (the closest existing decoder: grouped-query attention and a gated dense
feed-forward) and Vikupel (the closest layer-list design) at equal width and depth, and the device time of the kernels the
design added or extended beside the like kernels of the existing paths. Helpers and conventions are those of
design_bench.py and vikupel_bench.py."""
from __future__ import annotations

import json

import torch

from benchmarks.design_bench import _qwen3_cfg, _throughput, _time
from benchmarks.vikupel_bench import _meta, vikupel_cfg


def liverax_cfg(width, n_quads, vocab, head=128, window=1024, latent=None):
    """[attention_2, attention, latent_attention, attention] x n_quads; `latent`: (q_rank, kv_rank, head size, rotated
    size) of the latent layers."""
    heads = max(width // head, 1)
    kv = max(heads // 4, 1)
    ff = {"kind": "dense", "ff": 3 * width}
    qr, kr, d, rd = latent or (max(width // 4, 384), 512, 128, 64)
    base = {"heads": heads, "kv_heads": kv, "dim": head, "vdim": head, "scale": head ** -0.5, "v_mix": True}
    far = {"type": "attention_2", "mlp": ff,
           "mixer": {**base, "bias_max": 1024, "q_temp": {"coef": 0.1, "every": 512}}}
    win = {"type": "attention", "mlp": ff,
           "mixer": {**base, "mask": {"size": window}, "rot": {"base": 1e5, "dims": head, "scaling": {"factor": 2.0}}}}
    lat = {"type": "latent_attention", "mlp": ff,
           "mixer": {"heads": heads, "dim": d, "rot_dim": rd, "vdim": d, "q_rank": qr, "kv_rank": kr,
                     "scale": (d + rd) ** -0.5, "rot": {"base": 1e4, "dims": rd}, "mask": {"size": window}}}
    return {"architecture": "Liverax", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "logit_softcap": 25.0,
            "layers": [far, win, lat, win] * n_quads}


def kernels(peaks):
    from gllm_b200.ops import ref, sm100, sm100_latent as Lt, sm100_seq as S, sm100_ssd as K
    dev, bf = "cuda", torch.bfloat16
    hbm = float(peaks.get("hbm_gbs", 6650.0))
    out = []

    def row(name, ms, nbytes=None, like=None, flops=None):
        r = {"kernel": name, "ms": round(ms, 4)}
        if nbytes:
            r.update(gbs=round(nbytes / ms / 1e6, 1), frac_hbm=round(nbytes / ms / 1e6 / hbm, 3))
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 2)
        if like:
            r["like"] = like
        out.append(r)

    # -- stream and feed-forward -------------------------------------------------------------------------------
    T, W = 8192, 4096
    x, w1 = torch.randn(T, W, device=dev), torch.ones(W, device=dev).to(bf)
    y, res = torch.randn(T, W, device=dev).to(bf), torch.randn(T, W, device=dev).to(bf)
    row("resid_norm, layer norm 8192 x 4096",
        _time(lambda: S.resid_norm(x, y, None, None, w1, 1e-5, bf, center=True)), T * W * (4 + 4 + 2 + 2))
    row("rmsnorm + residual (existing bf16 path)", _time(lambda: sm100.rmsnorm(y, w1, 1e-5, res)), T * W * 8,
        like="resid_norm")
    del x, res
    F = 12288
    gu = (torch.randn(2 * F, W, device=dev) * W ** -0.5).to(bf)
    for t in (8192, 256, 64, 16):
        flops = 4.0 * t * W * F
        nb = 4 * F * W + 2 * t * (W + F)
        row("gate / up product, gelu epilogue, %d x 4096 -> 12288" % t,
            _time(lambda: sm100.linear_silu_mul(y[:t], gu, act="gelu"), iters=5), nb, flops=flops)
        row("gate / up product, silu epilogue (existing) %d" % t,
            _time(lambda: sm100.linear_silu_mul(y[:t], gu), iters=5), nb, like="gelu epilogue", flops=flops)
    del gu
    H, D = 32, 128
    o, z = torch.randn(T, H * D, device=dev).to(bf), torch.randn(T, 2 * H * D, device=dev).to(bf)
    row("gate_rows 8192 x 4096", _time(lambda: Lt.gate_rows(o, z[:, :H * D])), T * H * D * 6)
    row("silu_and_mul (existing, same output)", _time(lambda: sm100.silu_and_mul(z)), T * H * D * 6, like="gate_rows")
    del o, z, y

    # -- attention over keys and values -------------------------------------------------------------------------
    G, ps, win = 8, 16, 1024
    table = torch.randn(len(ref.distance_buckets(32, 1024)), H, device=dev)
    short = torch.randn(len(ref.distance_buckets(32, 128)), H, device=dev)
    fr = ref.banded_rotary_frequencies(D, 1e5, {"factor": 2.0}).to(dev)
    lam, sink = torch.tensor([0.3], device=dev), torch.zeros(H, device=dev)
    for label, qlens, ctx in (("prefill 4 x 2048", [2048] * 4, 0), ("decode 256 x 1 at 2048", [1] * 256, 2047)):
        B, qsl, sl, npp, bt, pos, slots = _meta(qlens, ctx, ps, dev)
        Tt = sum(qlens)
        kc, vc = (torch.randn(ref.kv_cache_shape(B * npp + 1, G, D, ps), device=dev).to(bf) for _ in range(2))
        qkvg = torch.randn(Tt, (2 * H + 2 * G) * D, device=dev).to(bf)
        first = torch.randn(Tt, (H + 2 * G) * D, device=dev).to(bf)[:, (H + G) * D:]
        qn, kn = torch.ones(H * D, device=dev).to(bf), torch.ones(G * D, device=dev).to(bf)
        ang = K.rotary_angles(pos, fr)
        rw = Tt * (H + 2 * G) * D * 4
        row("write, whole norms, temperature, mixed values " + label,
            _time(lambda: S.qk_norm_rope_kv_write(qkvg, H, G, D, D, qn, kn, 1e-5, pos, 0, 1e5, kc, vc, slots,
                                                  whole_norm=True, q_temp=(0.1, 512), v_mix=(first, lam))),
            rw + Tt * G * D * 2)
        row("write, rotation, mixed values " + label,
            _time(lambda: S.qk_norm_rope_kv_write(qkvg, H, G, D, D, None, None, 1e-5, pos, D, 1e5, kc, vc, slots, None,
                                                  1.0, False, ang, None, v_mix=(first, lam))),
            rw + Tt * G * D * 2 + Tt * D * 4)
        cs, q1 = torch.randn(8192, D, device=dev), torch.ones(D, device=dev).to(bf)
        qq, kk, vv = (qkvg[:, a * D:b * D].unflatten(1, (b - a, D)) for a, b in ((0, H), (H, H + G), (H + G, H + 2 * G)))
        row("rope_kv_write (existing: table rotary + q/k norm + cache write) " + label,
            _time(lambda: sm100.rope_kv_write(qq, kk, vv, pos, cs, D, True, q1, q1, 1e-5, kc, vc, slots)), rw,
            like="write")
        q, gate = torch.randn(Tt, H * D, device=dev).to(bf), qkvg[:, (H + 2 * G) * D:]
        nd = B if qlens[0] == 1 else 0

        def att(window=None, sk=None, **kw):
            return _time(lambda: S.window_attention(q, kc, vc, bt, sl, qsl, pos, D ** -0.5, H, D, window, sk,
                                                    num_decode_seqs=nd, max_q_len=max(qlens), v_dim=D, **kw), iters=5)

        def arow(name, ms, w, like=None):
            keys = sum(min(p + 1, w or 1 << 30) for ql in qlens for p in range(ctx, ctx + ql))
            row(name + " " + label, ms, like=like, flops=4.0 * keys * H * D,
                nbytes=B * min(ctx + qlens[0], w or 1 << 30) * G * D * 4 if nd else None)

        arow("attention, full causal, distance table to 1024, output gate", att(dist_table=table, gate=gate), None)
        arow("attention, full causal, distance table to 128, output gate", att(dist_table=short, gate=gate), None)
        arow("the same on the mma.sync kernels (to 1024)", att(dist_table=table, gate=gate, tc=False), None)
        arow("paged_attention (existing, full causal)",
             _time(lambda: sm100.paged_attention(q, kc, vc, bt, sl, qsl, D ** -0.5, H, D, nd, B, max(qlens),
                                                 max(qlens) + ctx), iters=5), None, like="attention, full causal")
        arow("attention, window 1024", att(win), win)
        arow("window attention with a sink (existing design, same window)", att(win, sink), win, like="attention, window")
        del kc, vc

    # -- latent attention ----------------------------------------------------------------------------------------
    R, rot = 512, 64
    fr = ref.banded_rotary_frequencies(rot, 1e4).to(dev)
    sink = torch.randn(H, device=dev)
    for label, qlens, ctx in (("prefill 4 x 2048", [2048] * 4, 0), ("decode 256 x 1 at 2048", [1] * 256, 2047)):
        B, qsl, sl, npp, bt, pos, slots = _meta(qlens, ctx, ps, dev)
        Tt = sum(qlens)
        tok_seq = torch.cat([torch.full((n,), i) for i, n in enumerate(qlens)]).to(torch.int32).to(dev)
        lat = torch.randn(ref.kv_cache_shape(B * npp + 1, 1, R + rot, ps), device=dev).to(bf)
        q, dkv = torch.randn(Tt, H, 128 + rot, device=dev).to(bf), torch.randn(Tt, R + rot, device=dev).to(bf)
        full, nw = torch.randn(Tt, H, R + rot, device=dev).to(bf), torch.ones(R, device=dev).to(bf)
        ang = K.rotary_angles(pos, fr)
        nb = Tt * (H * rot * 4 + (R + rot) * 4)
        row("latent norm + half-split rotation + latent write " + label,
            _time(lambda: Lt.latent_norm_rope_write(q, dkv, R, rot, nw, 1e-5, pos, fr, 1.0, full, lat, slots, ang)),
            nb + Tt * rot * 4)
        fp = torch.rand(rot // 2, device=dev)
        row("latent norm + pair rotation + latent write (existing) " + label,
            _time(lambda: Lt.latent_norm_rope_write(q, dkv, R, rot, nw, 1e-5, pos, fp, 1.0, full, lat, slots)), nb,
            like="latent norm")

        def lrow(name, ms, w, like=None):
            keys = sum(min(p + 1, w or 1 << 30) for ql in qlens for p in range(ctx, ctx + ql))
            row(name + " " + label, ms, like=like, flops=2.0 * keys * H * (2 * R + rot),
                nbytes=keys * (R + rot) * 2 if qlens[0] == 1 else None)

        lrow("latent attention, window 1024, sink",
             _time(lambda: sm100.mla_attention(full, lat, bt, tok_seq, pos, 192 ** -0.5, window=win, sink=sink), iters=3),
             win)
        lrow("latent attention (existing, full causal)",
             _time(lambda: sm100.mla_attention(full, lat, bt, tok_seq, pos, 192 ** -0.5), iters=3), None,
             like="latent attention")
        del lat
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
                      "liverax": _throughput(liverax_cfg(width, quads, vocab), vocab, args.warmup, args.steps),
                      "qwen3": _throughput(_qwen3_cfg(width, 4 * quads, heads, kv, 128, 3 * width, vocab), vocab,
                                           args.warmup, args.steps),
                      "vikupel": _throughput(vikupel_cfg(width, quads, vocab), vocab, args.warmup, args.steps)})
    line = {"design": "liverax", "dtype": "bf16", "data": "synthetic", "warmup": args.warmup, "steps": args.steps,
            "timing": "wall clock around LLM.generate with synchronize (sizes); CUDA events, L2 flushed (kernels)",
            "peaks": peaks, "sizes": sizes, "kernels": rows}
    print(json.dumps(line))
    return line
