"""Vikupel on the sm_100a kernels: the kernels this design added or extended (Mamba-2 step and chunked scan, vectorised
convolution, gate before the grouped norm, per-layer token input, rotary rows, rotated values, distance bias, output
gate and window in the plain and tensor-core paged attention) against their unfused PyTorch forms, the mixers alone
against the plain oracle, and the engine scenarios of test_vikupel_cpu.py in fp32 (tight) and bf16 (rounding-sized)."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import vikupel_oracle as oracle
import vikupel_util as U
from test_vikupel_cpu import CONFIGS, MIXERS, PLAN, marked_key_probe, mixer_alone, toks

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL32 = 1e-3


def close(a, b, tol):
    a, b = a.float().cpu(), b.float().cpu()
    return (a - b).abs().max().item() <= tol * (b.abs().max().item() + 1e-9)


def _batch(qlens, ctx, ps, pages):
    """Batch metadata of unequal requests (context `ctx` + `qlens` new tokens each) on random pages."""
    qsl = torch.tensor([0] + np.cumsum(qlens).tolist(), dtype=torch.int32, device=DEV)
    sl = torch.tensor([c + q for c, q in zip(ctx, qlens)], dtype=torch.int32, device=DEV)
    per = max((c + q + ps - 1) // ps for c, q in zip(ctx, qlens))
    bt = torch.randperm(pages - 1)[: len(qlens) * per].reshape(len(qlens), per).to(torch.int32).to(DEV)
    pos = torch.cat([torch.arange(c, c + q) for c, q in zip(ctx, qlens)]).to(torch.int32).to(DEV)
    seqi = torch.cat([torch.full((q,), i) for i, q in enumerate(qlens)]).to(DEV)
    slots = (bt[seqi, (pos // ps).long()] * ps + pos % ps).to(torch.int32)
    ndec = next((i for i, q in enumerate(qlens) if q != 1), len(qlens))
    return SimpleNamespace(query_start_loc=qsl, seq_lens=sl, block_table=bt, positions=pos, slot_mapping=slots,
                           max_q_len=max(qlens), num_decode_seqs=ndec, num_seqs=len(qlens), padded_tokens=0,
                           rec_slots=torch.randperm(len(qlens) + 3)[: len(qlens)].to(torch.int32).to(DEV))


# -- kernels against their unfused forms ---------------------------------------------------------------------------
SSD = [  # heads, groups, nstate, v_dim
    (4, 2, 16, 32), (3, 1, 48, 24), (8, 8, 128, 64), (4, 2, 64, 128), (2, 1, 256, 64), (6, 3, 40, 72), (2, 2, 8, 8)]


@pytest.mark.parametrize("sizes", SSD)
def test_ssd_scan_chunked_and_step(sizes):
    from gllm_b200.ops import ref, sm100_ssd as K
    H, G, N, V = sizes
    torch.manual_seed(sum(sizes))
    qlens, ctx = [1, 1, 2, 63, 64, 65, 150, 7], [0, 9, 5, 0, 33, 1, 70, 0]
    b = _batch(qlens, ctx, 16, 128)
    t, inner, bc = sum(qlens), H * V, G * N
    for dt in (torch.bfloat16, torch.float32):
        row = torch.randn(t, inner + 2 * bc, device=DEV).to(dt)
        step = (torch.randn(t, H + 8, device=DEV) * 2).to(dt)[:, :H]
        neg_a, bias, d = -torch.exp(torch.randn(H, device=DEV)), torch.randn(H, device=DEV) - 1, torch.randn(H, device=DEV)
        state = torch.randn(len(qlens) + 3, H, N, V, device=DEV)
        args = lambda st, dev: [x.to(dev) for x in (row[:, :inner], row[:, inner:inner + bc], row[:, inner + bc:],  # noqa: E731
                                                    step, neg_a, bias, d)] + [st, b.rec_slots.to(dev),
                                                                              b.seq_lens.to(dev),
                                                                              b.query_start_loc.to(dev), H, G, N, V]
        sref = state.cpu().clone()
        want = ref.ssd_scan(*args(sref, "cpu"))
        kinds = ["auto", "serial"] + (["chunk"] if dt == torch.bfloat16 else [])
        for kind in kinds:
            st = state.clone()
            got = K.ssd_scan(*args(st, DEV), num_decode_seqs=b.num_decode_seqs, max_q_len=b.max_q_len,
                             force=None if kind == "auto" else kind)
            tol = 2e-4 if kind == "chunk" or dt == torch.bfloat16 else 2e-5
            assert close(got, want, tol), (kind, dt)
            used = b.rec_slots.long().cpu()
            assert close(st[used.to(DEV)], sref[used], tol), (kind, dt)
            rest = [i for i in range(len(qlens) + 3) if i not in used.tolist()]
            assert torch.equal(st[rest].cpu(), state[rest].cpu())       # other slots are untouched


def test_ssd_chunked_far_decays():
    """Decays from nothing to whole orders of magnitude per token in one chunk: weights of neighbours stay exact."""
    from gllm_b200.ops import ref, sm100_ssd as K
    H, G, N, V, t = 4, 1, 32, 32, 130
    torch.manual_seed(5)
    row = torch.randn(t, H * V + 2 * N, device=DEV).bfloat16()
    step = torch.randn(t, H, device=DEV).bfloat16()
    step[10] = 60.0                                   # one token wipes the state, small decays follow
    args = [row[:, :H * V], row[:, H * V:H * V + N], row[:, H * V + N:], step, -torch.tensor([16.0, 1.0, 1e-3, 4.0]),
            torch.zeros(H), torch.ones(H), None, None, torch.tensor([t], dtype=torch.int32),
            torch.tensor([0, t], dtype=torch.int32), H, G, N, V]
    to = lambda dev: [x.to(dev) if torch.is_tensor(x) else x for x in args]  # noqa: E731
    assert close(K.ssd_scan(*to(DEV), force="chunk"), ref.ssd_scan(*to("cpu")), 2e-4)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5])
def test_convolution_vectorised(taps):
    from gllm_b200.ops import ref, sm100_seq as K
    torch.manual_seed(taps)
    for qlens, ctx in (([1, 1, 2, 3, 70, 5], [4, 0, 1, 0, 2, 9]), ([700, 1900], [0, 3])):
        b = _batch(qlens, ctx, 16, 512)
        for C, off in ((40, 8), (1032, 16), (36, 3)):
            t = sum(qlens)
            xz = torch.randn(t, off + C + 5, device=DEV).bfloat16()
            xz = torch.nn.functional.pad(xz, (0, -xz.shape[1] % 8)).contiguous()
            w, bias = torch.randn(C, taps, device=DEV), torch.randn(C, device=DEV)
            for act, ib in (("silu", None), ("none", torch.randn(C, device=DEV))):
                st = torch.randn(len(qlens) + 3, max(taps - 1, 1), C, device=DEV).bfloat16()
                sref = st.cpu().clone()
                cpu = lambda x: None if x is None else x.cpu()  # noqa: E731
                want = ref.causal_conv_silu(xz[:, off:].cpu(), C, w.cpu(), bias.cpu(), sref, b.rec_slots.cpu(),
                                            b.seq_lens.cpu(), b.query_start_loc.cpu(), act, cpu(ib))
                got = K.causal_conv_silu(xz[:, off:], C, w, bias, st, b.rec_slots, b.seq_lens, b.query_start_loc, act, ib)
                assert close(got, want, 8e-3) and torch.equal(st.cpu(), sref), (C, act)


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-5), (torch.bfloat16, 8e-3)])
def test_gate_norm_token_side_stream_update(dt, tol):
    from gllm_b200.ops import ref, sm100_seq, sm100_ssd as K
    torch.manual_seed(2)
    for t, n, parts in ((3, 12, 4), (17, 96, 2), (5, 1024, 1), (9, 8192, 2), (3, 8192, 1), (2, 16384, 1), (4, 30, 3)):
        o, z, w = torch.randn(t, n, device=DEV), torch.randn(t, n + 8, device=DEV).to(dt), torch.rand(n, device=DEV)
        out = torch.zeros(t, n + 24, device=DEV).to(dt)
        K.gate_then_norm(o, z[:, :n], w, n // parts, 1e-5, out[:, 8:8 + n])
        assert close(out[:, 8:8 + n], ref.gate_then_norm(o, z[:, :n], w, n // parts, 1e-5), tol), (t, n, parts)
        assert out[:, :8].abs().max() == 0 and out[:, 8 + n:].abs().max() == 0
    for t, dim, layers in ((5, 3, 4), (130, 64, 3)):
        g, table = torch.randn(t, dim, device=DEV).to(dt) * 2, torch.randn(50, dim * layers, device=DEV).to(dt)
        ids = torch.randint(0, 50, (t,), dtype=torch.int32, device=DEV)
        for i in range(layers):
            assert close(K.gelu_gate_embed(g, ids, table, i * dim), ref.gelu_gate_embed(g, ids, table, i * dim), tol)
    for t, width in ((3, 20), (65, 1024)):
        x, y = torch.randn(t, width, device=DEV), torch.randn(t, width, device=DEV).to(dt)
        w1, w2 = torch.rand(width, device=DEV).to(dt), torch.rand(width, device=DEV).to(dt)
        for post, pre, plain in ((None, w2, False), (None, None, True), (w1, w2, False), (w1, None, False)):
            a, b = x.clone(), x.clone()
            p = sm100_seq.resid_norm(a, y, post, None, pre, 1e-5, dt, plain, y_mul=0.37)
            q = ref.resid_norm(b, y, post, None, pre, 1e-5, dt, plain, y_mul=0.37)
            assert close(a, b, 1e-5)
            assert (p is None) == (q is None) and (p is None or close(p, q, tol))
    pos = torch.tensor([0, 1, 77, 100000], dtype=torch.int32, device=DEV)
    f = ref.banded_rotary_frequencies(34, 1e4).to(DEV)
    assert (K.rotary_angles(pos, f) - ref.rotary_angles(pos, f)).abs().max() < 1e-6


ATT = [  # heads, kv heads, dim, vdim, window, page size
    (4, 2, 64, 64, 20, 16), (8, 2, 128, 128, 100, 16), (6, 1, 64, 64, None, 8), (8, 8, 128, 128, None, 16),
    (4, 1, 256, 256, 33, 16), (6, 3, 48, 40, 17, 16), (5, 1, 64, 32, None, 16), (16, 1, 64, 64, 130, 64),
    (4, 4, 128, 128, 1, 16)]


@pytest.mark.parametrize("sizes", ATT)
def test_attention_bias_gate_turned_values(sizes):
    """All kernels that take a shape (plain, mma.sync, tcgen05) with every combination of the options."""
    from gllm_b200.ops import ref, sm100_seq as K
    H, G, D, V, window, ps = sizes
    torch.manual_seed(D + H)
    qlens, ctx = [1, 1, 1, 2, 64, 130, 31, 200], [0, 63, 300, 5, 0, 77, 250, 0]
    b = _batch(qlens, ctx, ps, 1200 // ps * 3)
    t, pages = sum(qlens), 1200 // ps * 3
    for dt in (torch.float32, torch.bfloat16):
        shape = ref.kv_cache_shape
        kc = torch.randn(shape(pages, G, D, ps), device=DEV).to(dt)
        vc = torch.randn(shape(pages, G, V, ps), device=DEV).to(dt)
        q = torch.randn(t, H * D, device=DEV).to(dt)
        gate = torch.randn(t, H * V + 16, device=DEV).to(dt)[:, 8:8 + H * V]
        bias = (torch.rand(H, device=DEV) * 2, torch.rand(H, device=DEV))
        turn = ref.rotary_angles(b.positions, ref.banded_rotary_frequencies(V, 100.0).to(DEV))
        meta = (b.block_table, b.seq_lens, b.query_start_loc)
        for db, gt, vt in ((bias, gate, None), (None, None, turn), (bias, None, turn), (None, gate, turn)):
            want = ref.window_attention(q, kc, vc, *meta, 1.5 * D ** -0.5, H, D, window, None, v_dim=V, dist_bias=db,
                                        gate=gt, v_turn=vt)
            for kw in ({"simt": True}, {"tc": False}, {}):
                out = torch.full((t, H * V + 24), 9.0, device=DEV).to(dt)
                K.window_attention(q, kc, vc, *meta, b.positions, 1.5 * D ** -0.5, H, D, window, None,
                                   num_decode_seqs=b.num_decode_seqs, max_q_len=b.max_q_len, v_dim=V,
                                   out=out[:, 8:8 + H * V], dist_bias=db, gate=gt, v_turn=vt, **kw)
                assert close(out[:, 8:8 + H * V], want, 2e-5 if dt == torch.float32 else 1.2e-2), (kw, dt)
                assert (out[:, :8] == 9).all() and (out[:, 8 + H * V:] == 9).all()


@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-5), (torch.bfloat16, 8e-3)])
def test_rotary_write_unit_norm_and_rotated_values(dt, tol):
    from gllm_b200.ops import ref, sm100_seq as K
    torch.manual_seed(3)
    for H, G, D, V, rot in ((4, 2, 48, 40, 32), (8, 8, 128, 128, 128), (2, 1, 6, 10, 0), (3, 1, 64, 64, 64)):
        b = _batch([1, 9, 40], [100, 0, 31], 16, 40)
        qkv = torch.randn(50, H * D + G * (D + V) + 7, device=DEV).to(dt)
        ang = ref.rotary_angles(b.positions, ref.banded_rotary_frequencies(
            rot, 50.0, {"factor": 4.0, "high": 4.0, "low": 1.0, "original": 64}).to(DEV))
        va = ref.rotary_angles(b.positions, ref.banded_rotary_frequencies(V, 50.0).to(DEV))
        res = []
        for m in (K, ref):
            kc, vc = (torch.zeros(ref.kv_cache_shape(40, G, d, 16), device=DEV).to(dt) for d in (D, V))
            q = m.qk_norm_rope_kv_write(qkv, H, G, D, V, None, None, 1e-5, b.positions, rot, 50.0, kc, vc,
                                        b.slot_mapping, None, 1.0, True, ang if rot else None, va)
            res.append((q, kc, vc))
        for a, c in zip(*res):
            assert close(a, c, tol)


# -- mixers and models ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(MIXERS))
def test_mixer_alone(name):
    want, outs = mixer_alone(MIXERS[name], 40 + len(name), device=DEV)
    for o in outs:
        assert close(o, want, 1e-4)


BIG = {
    "mamba": U.mamba(heads=4, groups=2, state=64, vdim=32, conv=4, norm_groups=2, mlp=U.dense(128)),
    "window": U.window(heads=4, kv_heads=2, dim=64, vdim=64, size=70, scale=0.125, mlp=U.dense(256)),
    "turned": U.turned(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=64, base=1e4, scale=0.2, mlp=U.dense(128)),
}


@pytest.mark.parametrize("name", sorted(BIG))
def test_tensor_core_sized_mixer_alone(name):
    cuts = ((200,), (130, 1, 1, 2, 66), (64, 64, 65, 7), (5,) * 20 + (1,) * 100)
    want, outs = mixer_alone(BIG[name], 9, n=200, cuts=cuts, page_size=16, device=DEV, dtype=torch.bfloat16, width=128)
    ref_out = mixer_alone(BIG[name], 9, n=200, cuts=((200,),), page_size=16, dtype=torch.bfloat16, width=128)[1][0]
    rms = want.pow(2).mean().sqrt()
    noise = (ref_out - want).pow(2).mean().sqrt() / rms
    for o in outs:
        assert (o - want).pow(2).mean().sqrt() / rms < 2 * noise + 2e-3
        assert (o - want).abs().max() < 3 * (ref_out - want).abs().max() + 1e-2 * want.abs().max()


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_marked_keys_at_window_edges_and_page_borders(dt):
    tol = 1e-4 if dt == torch.float32 else 3e-2
    for kind, n, size, heads, kv, dim, vdim in (("turned", 331, None, 2, 2, 64, 64), ("window", 200, 65, 4, 2, 64, 64),
                                                ("window", 200, 48, 2, 2, 32, 4), ("turned", 200, None, 2, 1, 32, 8)):
        for back in ((0, 1, 15, 16, 17, 64, 199) if kind == "turned" else (1, size - 2, size - 1, size, size + 1)):
            want, outs, other = marked_key_probe(kind, n, back, size, 16, DEV, dt, heads, kv, dim, vdim)
            moved = (want[-1] - other[-1]).abs().max() / want[-1].abs().max()
            if back > 0:
                assert moved > 0.2 if kind == "turned" or back < size else moved == 0
            # in bf16 only a row that rests on one key is sharp: elsewhere large scores carry their operands' rounding
            for o in outs:
                if dt == torch.float32:
                    assert close(o, want, tol), (kind, back)
                elif back > 0 and moved > 0.2:
                    assert close(o[-1], want[-1], tol), (kind, back)


@pytest.fixture(scope="module")
def models():
    out = {}
    cfgs = dict(CONFIGS)
    cfgs["tensor_core"] = U.make_config([BIG["mamba"], BIG["window"], BIG["turned"], BIG["mamba"]], width=128, vocab=128,
                                        side=64, loop=(1, 3, 2))
    for i, (name, cfg) in enumerate(cfgs.items()):
        w = U.random_weights(cfg, seed=30 + i)
        out[name] = (cfg, w, U.save_model(cfg, w))
    return out


class Expect:
    """What a run is held to. fp32: the oracle, tightly. bf16: the error that rounding alone causes, measured by running
    the unfused PyTorch forms on the CPU with the same rounding points; the kernels may be twice as far."""

    def __init__(self, cfg, w, path, tokens, dtype):
        self.want, self.dtype = U.expected_logits(cfg, w, tokens), dtype
        if dtype == "bfloat16":
            s = U.session(path, "bfloat16", "cpu", max_tokens=max(256, len(tokens) + 64), page_size=16)
            self.noise = U.row_errs(U.run_chunks(s, "r", tokens, [len(tokens)]), self.want)

    def check(self, got):
        e = U.row_errs(got, self.want)
        if self.dtype == "float32":
            assert e.max() < TOL32 and np.median(e) < 1e-5, (e.max(), np.median(e))
        else:
            assert np.median(e) <= 2 * np.median(self.noise) + 1e-2, (np.median(e), np.median(self.noise))
            assert np.sort(e)[int(0.9 * (len(e) - 1))] <= 2 * np.sort(self.noise)[int(0.9 * (len(e) - 1))] + 2e-2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS) + ["tensor_core"])
def test_prompts_portions_and_decoding(models, name, dtype):
    cfg, w, path = models[name]
    t = toks(150 if name == "tensor_core" else 60, cfg["vocab"], 3)
    x = Expect(cfg, w, path, t, dtype)
    for cuts in ([len(t)], [len(t) // 2], [2, 3, 2, 17, 1, 1, 2], [1]):
        x.check(U.run_chunks(U.session(path, dtype, DEV, page_size=16), "a", t, cuts))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "state_only", "tensor_core"])
def test_mixed_batch_reuses_pages_and_slots(models, name, dtype):
    cfg, w, path = models[name]
    total = {}
    for step in PLAN:
        for k, n in step:
            total[k] = total.get(k, 0) + n
    reqs = {k: toks(n, cfg["vocab"], 50 + i) for i, (k, n) in enumerate(sorted(total.items()))}
    got = U.run_plan(U.session(path, dtype, DEV, max_tokens=128, page_size=16), reqs, PLAN)
    for k, t in reqs.items():
        Expect(cfg, w, path, t, dtype).check(got[k])


def test_generation_under_cuda_graphs(models):
    from gllm_b200.engine.llm_engine import LLM
    cfg, w, path = models["mixed"]
    llm = LLM(path, dtype="float32", page_size=16, maxp=32, maxd=8, num_gpu_pages=64, model_max_length=96,
              log_stats=False, device=DEV, num_state_slots=2)
    prompts, lens = [toks(21, cfg["vocab"], 31), toks(3, cfg["vocab"], 32), toks(40, cfg["vocab"], 33)], [7, 12, 5]
    seqs = llm.generate(tokens=prompts, output_lens=lens, temperature=0.0, top_k=1)
    for p, n, s in zip(prompts, lens, seqs):
        cur = list(p)
        for _ in range(n):
            cur.append(int(oracle.forward(cfg, w, cur)[-1].argmax()))
        assert s.token_ids == cur
