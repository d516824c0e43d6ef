"""Liverax on the sm_100a kernels: the kernels this design added or extended (layer norm in the stream update, norms over
whole projections, query temperature and mixed values in the rotary write, distance table in the plain and tensor-core
paged attention, window and sink in both latent attention kernels, half-split latent rotation, row gate, tanh-gelu gated
products) against their unfused PyTorch forms, the mixers alone against the plain oracle, and the engine scenarios of
test_liverax_cpu.py in fp32 (tight) and bf16 (rounding-sized)."""
import numpy as np
import pytest
import torch

import liverax_oracle as oracle
import liverax_util as U
from test_liverax_cpu import CONFIGS, MIXERS, PLAN, marked_key_probe, mixer_alone, toks
from test_vikupel_gpu import _batch, close

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL32 = 1e-3
DTYPES = [(torch.float32, 2e-5), (torch.bfloat16, 8e-3)]


# -- kernels against their unfused forms ---------------------------------------------------------------------------
@pytest.mark.parametrize("dt,tol", DTYPES)
def test_stream_update_with_a_layer_norm(dt, tol):
    from gllm_b200.ops import ref, sm100_seq as K
    torch.manual_seed(1)
    for t, width in ((3, 20), (65, 1024), (9, 2056), (5, 4096), (2, 8192), (4, 10000)):
        x, y = torch.randn(t, width, device=DEV) + 25.0, torch.randn(t, width, device=DEV).to(dt)
        w1, w2 = torch.rand(width, device=DEV).to(dt), torch.rand(width, device=DEV).to(dt)
        for branch, post in ((y, None), (None, None), (y, w1)):
            a, b = x.clone(), x.clone()
            p = K.resid_norm(a, branch, post, None, w2, 1e-5, dt, center=True)
            q = ref.resid_norm(b, branch, post, None, w2, 1e-5, dt, center=True)
            assert close(a, b, 1e-5) and close(p, q, max(tol, 1e-4)), (t, width)


@pytest.mark.parametrize("dt,tol", DTYPES)
def test_rotary_write_whole_norm_temperature_mixed_values(dt, tol):
    from gllm_b200.ops import ref, sm100_seq as K
    torch.manual_seed(3)
    for H, G, D, V, rot in ((4, 2, 48, 40, 0), (8, 8, 128, 128, 0), (2, 1, 6, 10, 4), (3, 1, 64, 64, 64), (16, 2, 128, 64, 0),
                            (5, 5, 32, 128, 32)):
        b = _batch([1, 9, 40], [100, 0, 31], 16, 40)
        qkv = torch.randn(50, H * D + G * (D + V) + 8, device=DEV).to(dt)
        first = torch.randn(50, G * V + 5, device=DEV).to(dt)[:, 4:4 + G * V]
        qn, kn = (torch.rand(n * D, device=DEV).to(dt) + 0.5 for n in (H, G))
        ang = ref.rotary_angles(b.positions, ref.banded_rotary_frequencies(rot, 50.0, {"factor": 2.0}).to(DEV)) \
            if rot else None
        lam = torch.tensor([0.3], device=DEV)
        for whole, temp, mix in ((True, (0.7, 6), (first, lam)), (True, None, None), (False, (0.2, 1), None),
                                 (False, None, (first, lam))):
            res = []
            for m in (K, ref):
                kc, vc = (torch.zeros(ref.kv_cache_shape(40, G, d, 16), device=DEV).to(dt) for d in (D, V))
                q = m.qk_norm_rope_kv_write(qkv, H, G, D, V, qn if whole else None, kn if whole else None, 1e-5,
                                            b.positions, rot, 50.0, kc, vc, b.slot_mapping, None, 1.0, False, ang, None,
                                            whole, temp, mix)
                res.append((q, kc, vc))
            for a, c in zip(*res):
                assert close(a, c, tol), (H, D, V, whole, temp, mix is not None)


ATT = [  # heads, kv heads, dim, vdim, window, page size, table rows (distances)
    (4, 2, 64, 64, None, 16, 90), (8, 2, 128, 128, None, 16, 33), (6, 1, 64, 64, None, 8, 1), (8, 8, 128, 128, 100, 16, 500),
    (4, 1, 256, 256, None, 16, 70), (6, 3, 48, 40, None, 16, 41), (5, 1, 64, 32, 20, 16, 12), (32, 1, 64, 64, None, 64, 200),
    (24, 2, 128, 128, None, 16, 129), (4, 4, 128, 128, None, 16, 64)]


@pytest.mark.parametrize("sizes", ATT)
def test_attention_with_a_distance_table(sizes):
    """All kernels that take a shape (plain, mma.sync, tcgen05): far and near tiles, tables shorter and longer than the
    context, with gate, window and sink."""
    from gllm_b200.ops import ref, sm100_seq as K
    H, G, D, V, window, ps, rows = sizes
    torch.manual_seed(D + H)
    qlens, ctx = [1, 1, 1, 2, 64, 130, 31, 200], [0, 63, 300, 5, 0, 77, 250, 0]
    pages = 1200 // ps * 3
    b = _batch(qlens, ctx, ps, pages)
    t = sum(qlens)
    for dt in (torch.float32, torch.bfloat16):
        kc = torch.randn(ref.kv_cache_shape(pages, G, D, ps), device=DEV).to(dt)
        vc = torch.randn(ref.kv_cache_shape(pages, G, V, ps), device=DEV).to(dt)
        q = torch.randn(t, H * D, device=DEV).to(dt)
        gate = torch.randn(t, H * V + 16, device=DEV).to(dt)[:, 8:8 + H * V]
        table, sink = torch.randn(rows, H, device=DEV) * 2, torch.randn(H, device=DEV)
        meta = (b.block_table, b.seq_lens, b.query_start_loc)
        for gt, sk in ((gate, None), (None, sink), (gate, sink)):
            want = ref.window_attention(q, kc, vc, *meta, 1.5 * D ** -0.5, H, D, window, sk, v_dim=V, gate=gt,
                                        dist_table=table)
            for kw in ({"simt": True}, {"tc": False}, {}):
                out = torch.full((t, H * V + 24), 9.0, device=DEV).to(dt)
                K.window_attention(q, kc, vc, *meta, b.positions, 1.5 * D ** -0.5, H, D, window, sk,
                                   num_decode_seqs=b.num_decode_seqs, max_q_len=b.max_q_len, v_dim=V,
                                   out=out[:, 8:8 + H * V], gate=gt, dist_table=table, **kw)
                assert close(out[:, 8:8 + H * V], want, 2e-5 if dt == torch.float32 else 1.2e-2), (kw, dt)
                assert (out[:, :8] == 9).all() and (out[:, 8 + H * V:] == 9).all()


@pytest.mark.parametrize("dt,tol", DTYPES)
def test_latent_write_with_half_split_rotation(dt, tol):
    from gllm_b200.ops import ref, sm100_latent as K
    torch.manual_seed(4)
    for H, dim, rot, rank, qr in ((3, 6, 4, 9, 5), (16, 64, 64, 512, 128), (5, 8, 2, 62, 7)):
        b = _batch([1, 9, 40], [100, 0, 31], 16, 40)
        q = torch.randn(50, H, dim + rot, device=DEV).to(dt)
        dkv = torch.randn(50, qr + rank + rot + 3, device=DEV).to(dt)[:, qr:qr + rank + rot]
        nw = torch.rand(rank, device=DEV).to(dt)
        f = ref.banded_rotary_frequencies(rot, 77.0).to(DEV)
        ang = ref.rotary_angles(b.positions, f)
        res = []
        for m in (K, ref):
            full = torch.zeros(50, H, rank + rot, device=DEV).to(dt)
            cache = torch.zeros(ref.kv_cache_shape(40, 1, rank + rot, 16), device=DEV).to(dt)
            m.latent_norm_rope_write(q, dkv, rank, rot, nw, 1e-5, b.positions, f, 1.0, full, cache, b.slot_mapping, ang)
            res.append((full, cache))
        for a, c in zip(*res):
            assert close(a, c, tol), (H, rank)


@pytest.mark.parametrize("sizes", [(3, 9, 4, 16), (16, 512, 64, 16), (5, 512, 64, 64), (40, 512, 64, 8), (4, 130, 6, 16),
                                   (2, 96, 32, 4)])
def test_latent_attention_with_window_and_sink(sizes):
    from gllm_b200.ops import ref, sm100, sm100_latent as K
    H, rank, rot, ps = sizes
    torch.manual_seed(rank + H)
    qlens, ctx = [1, 1, 1, 2, 64, 130, 31, 200], [0, 63, 300, 5, 0, 77, 250, 0]
    pages = 1200 // ps * 3
    b = _batch(qlens, ctx, ps, pages)
    t = sum(qlens)
    b.tok_seq = torch.cat([torch.full((q,), i) for i, q in enumerate(qlens)]).to(torch.int32).to(DEV)
    sink = torch.randn(H, device=DEV) * 2
    for dt in (torch.float32, torch.bfloat16):
        cache = torch.randn(ref.kv_cache_shape(pages, 1, rank + rot, ps), device=DEV).to(dt)
        q = torch.randn(t, H, rank + rot, device=DEV).to(dt)
        for window in (None, 1, 2, 63, 64, 65, 129, 1000):
            for sk in (None, sink):
                want = ref.latent_attention(q, cache, b.block_table, b.seq_lens, b.query_start_loc,
                                            1.5 * (rank + rot) ** -0.5, rank, window, sk)
                got = K.latent_attention(q, cache, b, 1.5 * (rank + rot) ** -0.5, rank, window=window, sink=sk)
                assert close(got, want, 2e-5 if dt == torch.float32 else 1.2e-2), (window, dt)
                plain = K.latent_attention(q, cache, b, 1.5 * (rank + rot) ** -0.5, rank, plain=True, window=window,
                                           sink=sk)
                assert close(plain, want, 2e-5 if dt == torch.float32 else 1.2e-2), (window, dt)
                if rank == 512 and dt == torch.bfloat16:       # the keys split over several blocks, then merged
                    n = 4                                      # few tokens: the partials' workspace is bounded
                    split = sm100.mla_attention(q[:n].contiguous(), cache, b.block_table, b.tok_seq[:n].contiguous(),
                                                b.positions[:n].contiguous(), 1.5 * (rank + rot) ** -0.5, 3, window, sk)
                    assert close(split, want[:n], 1.2e-2), window


@pytest.mark.parametrize("dt,tol", DTYPES)
def test_row_gate_and_gated_gelu(dt, tol):
    from gllm_b200.ops import ref, sm100_latent, sm100_seq
    torch.manual_seed(5)
    for t, n in ((3, 12), (130, 512), (1, 7)):
        o = torch.randn(t, n + 8, device=DEV).to(dt)[:, 8:]
        gate = torch.randn(t, 2 * n + 8, device=DEV).to(dt)[:, 8:8 + n]
        want = ref.gate_rows(o.clone(), gate)
        assert close(sm100_latent.gate_rows(o, gate), want, tol)
    for t, f, block in ((3, 12, 0), (40, 256, 128), (9, 30, 5)):
        gu = (torch.randn(t, 2 * f + 8, device=DEV) * 3).to(dt)[:, :2 * f]
        assert close(sm100_seq.silu_mul(gu, None, block, "gelu"), ref.silu_mul(gu, block, "gelu"), tol)


@pytest.mark.parametrize("t", [1, 7, 32, 33, 64, 130, 700])
def test_gated_gelu_product(t):
    from gllm_b200.ops import ref, sm100
    torch.manual_seed(t)
    for k, f in ((128, 128), (192, 256), (1024, 1152)):
        x = torch.randn(t, k, device=DEV).bfloat16()
        w = (torch.randn(2 * f, k, device=DEV) * 2 * k ** -0.5).bfloat16()
        w[:f] *= 3                                             # gates far out on both sides
        wi = ref.interleave_gate_up(w, 128)
        for act in ("gelu", "silu"):
            got = sm100.linear_silu_mul(x, wi, act=act)
            want = ref.linear_silu_mul(x.float(), wi.float(), act=act)
            assert torch.isfinite(got).all() and close(got, want, 1e-2), (k, f, act)
    z = torch.tensor([[-300.0, -40.0, -8.0, -1.0, 0.0, 1.0, 8.0, 300.0]], device=DEV).bfloat16()
    x = z[:, :1].new_ones(t, 64)
    w = torch.zeros(256, 64, device=DEV).bfloat16()
    w[:8, 0], w[128:, 1] = z[0], 1.0
    got = sm100.linear_silu_mul(x, ref.interleave_gate_up(w, 128), act="gelu")[:, :8]
    assert close(got, oracle.gelu_tanh(z.cpu().double()).float().expand(t, 8), 8e-3)


# -- mixers and models ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(MIXERS))
def test_mixer_alone(name):
    want, outs = mixer_alone(MIXERS[name], 40 + len(name), device=DEV)
    for o in outs:
        assert close(o, want, 1e-4)


BIG = {
    "rotary": U.rotary(heads=4, kv_heads=2, dim=64, vdim=64, size=70, rot_dims=64, base=1e4, scale=0.12, v_mix=True,
                       mlp=U.dense(256)),
    "distance": U.distance(heads=4, kv_heads=2, dim=64, vdim=64, rows=24, bias_max=90, coef=0.2, every=20, scale=0.1,
                           v_mix=True, mlp=U.dense(128)),
    "latent": U.latent(heads=4, dim=64, rot_dim=64, vdim=64, q_rank=96, kv_rank=512, size=75, base=1e4, scale=0.08,
                       mlp=U.dense(128)),
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
    for kind, n, size, heads, kv, dim, vdim, rank in (
            ("distance", 331, None, 2, 2, 64, 64, None), ("rotary", 200, 65, 4, 2, 64, 64, None),
            ("rotary", 200, 48, 2, 2, 32, 4, None), ("distance", 200, None, 2, 1, 32, 8, None),
            ("latent", 200, 65, 3, 0, 64, 64, 512), ("latent", 200, 48, 2, 0, 32, 8, None)):
        for back in ((0, 1, 15, 16, 17, 64, 199) if kind == "distance" else (1, size - 2, size - 1, size, size + 1)):
            want, outs, other = marked_key_probe(kind, n, back, size, 16, DEV, dt, heads, kv, dim, vdim, rank=rank)
            moved = (want[-1] - other[-1]).abs().max() / want[-1].abs().max()
            if back > 0:
                assert moved > 0.1 if kind == "distance" or back < size else moved == 0, (kind, back, moved)
            # in bf16 only a row that rests on one key is sharp: elsewhere large scores carry their operands' rounding
            for o in outs:
                if dt == torch.float32:
                    assert close(o, want, tol), (kind, back)
                elif back > 0 and moved > 0.1:
                    assert close(o[-1], want[-1], tol), (kind, back)


@pytest.fixture(scope="module")
def models():
    out = {}
    cfgs = dict(CONFIGS)
    cfgs["tensor_core"] = U.make_config([BIG["distance"], BIG["rotary"], BIG["latent"], BIG["rotary"]], width=128, vocab=128)
    for i, (name, cfg) in enumerate(cfgs.items()):
        w = U.random_weights(cfg, seed=70 + i)
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
@pytest.mark.parametrize("name", ["mixed", "latent_only", "tensor_core"])
def test_mixed_batch_reuses_pages(models, name, dtype):
    cfg, w, path = models[name]
    total = {}
    for step in PLAN:
        for k, n in step:
            total[k] = total.get(k, 0) + n
    reqs = {k: toks(n, cfg["vocab"], 50 + i) for i, (k, n) in enumerate(sorted(total.items()))}
    got = U.run_plan(U.session(path, dtype, DEV, max_tokens=128, page_size=16), reqs, PLAN)
    for k, t in reqs.items():
        Expect(cfg, w, path, t, dtype).check(got[k])


def test_long_decoding_tensor_core(models):
    """Decoding past the windows and the distance table on the tensor-core kernels."""
    cfg, w, path = models["tensor_core"]
    t = toks(330, cfg["vocab"], 6)
    Expect(cfg, w, path, t, "bfloat16").check(U.run_chunks(U.session(path, "bfloat16", DEV, max_tokens=384, page_size=16),
                                                           "a", t, [90, 2, 3]))


@pytest.mark.parametrize("name", ["mixed", "tensor_core"])
def test_generation_under_cuda_graphs(models, name):
    """fp32 against the oracle's own greedy choice at every position."""
    from gllm_b200.engine.llm_engine import LLM
    cfg, w, path = models[name]
    llm = LLM(path, dtype="float32", page_size=16, maxp=32, maxd=8, num_gpu_pages=64, model_max_length=96,
              log_stats=False, device=DEV)
    prompts, lens = [toks(21, cfg["vocab"], 31), toks(3, cfg["vocab"], 32), toks(40, cfg["vocab"], 33)], [7, 12, 5]
    seqs = llm.generate(tokens=prompts, output_lens=lens, temperature=0.0, top_k=1)
    for p, n, s in zip(prompts, lens, seqs):
        cur = list(p)
        for _ in range(n):
            cur.append(int(oracle.forward(cfg, w, cur)[-1].argmax()))
        assert s.token_ids == cur
