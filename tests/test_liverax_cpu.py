"""Liverax through the engine (scheduler bookkeeping, page manager, batch builder, runner) against the plain oracle in
liverax_oracle.py: mechanisms alone, chunking, batching, re-use of pages, far keys, page borders, window and distance-bucket
edges, mixed values, degenerate sizes, greedy generation. Runs on the CPU path in fp32; test_liverax_gpu.py repeats the
scenarios on the kernels."""
import math

import numpy as np
import pytest
import torch

import liverax_oracle as oracle
import liverax_util as U

TOL = 2e-4
EPS = 1e-5


def toks(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


CONFIGS = {
    # every mixer; the first value-mixing layer is a rotary one, a layer between two mixing ones does not mix; no ff once
    "mixed": U.make_config([U.latent(mlp=U.dense()), U.rotary(v_mix=True, mlp=U.dense(20)),
                            U.distance(v_mix=True, mlp=U.dense(16)), U.rotary(size=3, mlp=U.dense(9)), U.latent(size=11),
                            U.distance(heads=6, kv_heads=2, dim=10, rows=8, bias_max=40, every=3, v_mix=True),
                            U.rotary(heads=2, kv_heads=2, dim=6, rot_dims=6, v_mix=True, mlp=U.dense(7))]),
    # nothing is mixed, no cap, no query temperature, no linear scaling, values wider than keys, a window of two
    "plain": U.make_config([U.distance(heads=3, kv_heads=3, dim=4, vdim=10, coef=None, rows=4, bias_max=9),
                            U.rotary(heads=6, kv_heads=3, dim=10, vdim=12, size=2, factor=None, rot_dims=10, mlp=U.dense(8)),
                            U.latent(heads=4, dim=10, rot_dim=2, vdim=3, q_rank=4, kv_rank=16, size=30, mlp=U.dense(8))],
                           cap=None),
    # the only mixing layer is alone; one kind of layer
    "distance_only": U.make_config([U.distance(v_mix=True, mlp=U.dense()), U.distance(rows=32, bias_max=100)], cap=3.0),
    "latent_only": U.make_config([U.latent(), U.latent(heads=5, size=1, mlp=U.dense())]),
    # sizes of one, values that other models make equal or 1
    "ones": U.make_config([U.distance(heads=1, kv_heads=1, dim=1, vdim=1, rows=2, bias_max=2, every=1, scale=1.0,
                                      v_mix=True, mlp=U.dense(1)),
                           U.rotary(heads=1, kv_heads=1, dim=2, vdim=1, size=1, rot_dims=2, factor=1.0, scale=1.0,
                                    v_mix=True, mlp=U.dense(3)),
                           U.latent(heads=1, dim=1, rot_dim=2, vdim=1, q_rank=1, kv_rank=1, size=2, scale=1.0,
                                    mlp=U.dense(2))], width=8, vocab=17),
}


@pytest.fixture(scope="module")
def models():
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        w = U.random_weights(cfg, seed=70 + i)
        out[name] = (cfg, w, U.save_model(cfg, w))
    return out


# -- each mechanism alone, against its own oracle function -----------------------------------------------------
def mixer_alone(layer_cfg, seed, n=19, cuts=((19,), (7, 1, 1, 2, 8), (2,) * 9 + (1,), (1,) * 19), page_size=4,
                device="cpu", dtype=torch.float32, width=20):
    """Value-mixing mixers get another layer's values, rows of a wider buffer."""
    w = U.random_weights(U.make_config([layer_cfg], width=width), seed)
    mixer = U.build_mixer(layer_cfg, w, width, device, dtype)
    g = torch.Generator().manual_seed(seed)
    h = torch.randn(n, width, generator=g).bfloat16().float()
    m, first, prepare = layer_cfg["mixer"], None, None
    if m.get("v_mix"):
        kv, dv = m["kv_heads"], m["vdim"]
        first = torch.randn(n, kv * dv + 3, generator=g).bfloat16().float()
        buf = first.to(device=device, dtype=dtype)
        first = first[:, 2:2 + kv * dv]

        def prepare(inp, at, c):
            inp.first_values = buf[at:at + c, 2:2 + kv * dv]
        first = first.reshape(n, kv, dv)
    want = U.oracle_mixer(h, layer_cfg, w, first=first).float()
    return want, [U.drive_mixer(mixer, h, list(c), page_size, device, dtype, prepare=prepare) for c in cuts]


MIXERS = {
    "rotary": U.rotary(),
    "rotary_mixed_values": U.rotary(v_mix=True),
    "rotary_one_kv_head": U.rotary(heads=5, kv_heads=1, dim=6, vdim=9, size=1, rot_dims=2),
    "rotary_whole_unscaled": U.rotary(rot_dims=8, factor=None, size=500, v_mix=True),
    "distance": U.distance(),
    "distance_mixed_values": U.distance(v_mix=True),
    "distance_one_kv_head": U.distance(heads=5, kv_heads=1, dim=3, vdim=7, rows=4, bias_max=3),
    "distance_no_temperature": U.distance(coef=None, rows=2, bias_max=8),
    "distance_wide_table": U.distance(heads=2, kv_heads=2, rows=64, bias_max=900, every=1, coef=1.5),
    "latent": U.latent(),
    "latent_wide_values": U.latent(heads=2, dim=4, rot_dim=6, vdim=12, q_rank=22, kv_rank=30, size=1),
    "latent_window_wider_than_all": U.latent(heads=5, size=400),
}


@pytest.mark.parametrize("name", sorted(MIXERS))
def test_mixer_alone(name):
    want, outs = mixer_alone(MIXERS[name], 40 + len(name))
    for o in outs:
        assert torch.allclose(o, want, atol=1e-4, rtol=1e-4), (o - want).abs().max()


def test_layer_norm_with_a_mean_far_from_zero():
    from gllm_b200.layers import functional as Fn
    g = torch.Generator().manual_seed(1)
    x, y, w = torch.randn(5, 12, generator=g) + 300.0, torch.randn(5, 12, generator=g), torch.rand(12, generator=g)
    a = x.clone()
    out = Fn.resid_norm(a, y, None, None, w, EPS, torch.float32, center=True)
    want = oracle.layer_norm(x.double() + y.double(), w.double(), EPS).float()
    assert torch.allclose(a, x + y) and torch.allclose(out, want, atol=2e-4)


def test_distance_buckets():
    """Expanded rows equal the formula at every distance, also where a logarithmic step falls on a whole number, and
    beyond the end of the expansion."""
    from gllm_b200.ops import ref
    for rows, dmax in ((2, 2), (2, 50), (4, 9), (10, 29), (8, 64), (16, 128), (32, 256), (32, 300), (64, 1000), (6, 4)):
        got = ref.distance_buckets(rows, dmax)
        assert got[-1] == rows - 1 and got == sorted(got)
        for n in range(3 * dmax + 5):
            assert got[min(n, len(got) - 1)] == oracle.bucket(n, rows, dmax), (rows, dmax, n)
    assert ref.distance_buckets(32, 256)[31:33] == [19, 20] and ref.distance_buckets(32, 256)[64] == 24


def test_query_temperature_steps():
    from gllm_b200.ops import ref
    for coef, every in ((0.3, 7), (1.0, 1), (0.05, 64)):
        pos = torch.arange(400, dtype=torch.int32)
        want = oracle.temperature(400, {"coef": coef, "every": every}).float()
        got = ref.query_temperature(pos, coef, every)
        assert torch.allclose(got, want, rtol=1e-6)
        assert got[every - 2] == 1.0 if every > 1 else got[0] > 1.0
        assert got[every - 1] > 1.0 and (got[1:] >= got[:-1]).all()


def test_linear_scaling_of_the_angles():
    from gllm_b200.ops import ref
    f = ref.banded_rotary_frequencies(12, 700.0, {"factor": 5.0})
    assert torch.allclose(f, torch.tensor(oracle.frequencies({"dims": 12, "base": 700.0, "scaling": {"factor": 5.0}}),
                                          dtype=torch.float64), rtol=1e-12)
    assert math.isclose(float(f[0]), 0.2)


def test_gated_gelu():
    from gllm_b200.layers import functional as Fn
    from gllm_b200.ops import ref
    gu = torch.randn(4, 12, generator=torch.Generator().manual_seed(3)) * 3
    want = oracle.gelu_tanh(gu[:, :6].double()) * gu[:, 6:].double()
    assert torch.allclose(Fn.silu_mul(gu, act="gelu"), want.float(), atol=1e-6)
    alt = torch.cat([gu[:, :3], gu[:, 6:9], gu[:, 3:6], gu[:, 9:]], 1)
    assert torch.allclose(Fn.silu_mul(alt, block=3, act="gelu"), want.float(), atol=1e-6)
    x, w = torch.randn(5, 8), torch.randn(512, 8)
    want = oracle.gelu_tanh(x.double() @ w[:256].double().T) * (x.double() @ w[256:].double().T)
    got = Fn.linear_silu_mul(x, ref.interleave_gate_up(w, 128), act="gelu")
    assert torch.allclose(got, want.float(), atol=1e-4)


@pytest.mark.parametrize("name", ["vmix", "rel", "q.norm", "k.norm", "q.b", "k.b", "v.b", "g"])
def test_every_part_of_the_distance_attention_shows(name):
    layer = U.distance(v_mix=True)
    w = U.random_weights(U.make_config([layer]), 7)
    h = torch.randn(16, 20, generator=torch.Generator().manual_seed(7))
    first = torch.randn(16, 2, 6, generator=torch.Generator().manual_seed(8))
    base = U.oracle_mixer(h, layer, w, first=first)
    w2 = dict(w)
    w2["l0.mix." + name] = w["l0.mix." + name].flip(0) if w["l0.mix." + name].dim() else w["l0.mix." + name] * 0.25
    want = U.oracle_mixer(h, layer, w2, first=first)
    assert (want - base).abs().max() > 0.05

    def prepare(inp, at, c):
        inp.first_values = first.reshape(16, -1)[at:at + c]

    got = U.drive_mixer(U.build_mixer(layer, w2, 20), h, [5, 1, 2, 8], prepare=prepare)
    assert torch.allclose(got, want.float(), atol=1e-4)


def test_sink_shows_and_counts_once():
    """A large sink takes the result to zero, a very negative one leaves the plain softmax; one key only: the weight is
    the logistic function of score minus sink."""
    layer = U.latent(size=1)
    w = U.random_weights(U.make_config([layer]), 9)
    h = torch.randn(6, 20, generator=torch.Generator().manual_seed(9))
    outs = {}
    for s in (-40.0, 0.5, 60.0):
        w2 = {**w, "l0.mix.sink": torch.full((3,), s)}
        want = U.oracle_mixer(h, layer, w2).float()
        got = U.drive_mixer(U.build_mixer(layer, w2, 20), h, [4, 1, 1])
        assert torch.allclose(got, want, atol=1e-4)
        outs[s] = want
    assert outs[60.0].abs().max() < 1e-3 * outs[-40.0].abs().max()
    assert (outs[0.5] - outs[-40.0]).abs().max() > 0.05


# -- whole models ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_matches_oracle(models, name):
    cfg, w, path = models[name]
    t = toks(37, cfg["vocab"], 1)
    got = U.run_chunks(U.session(path), "a", t, [len(t)])
    assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL


def test_residual_stream_after_every_layer(models):
    cfg, w, path = models["mixed"]
    t = toks(15, cfg["vocab"], 2)
    s = U.session(path)
    s.runner.model.trace = []
    U.run_chunks(s, "a", t, [len(t)])
    want = []
    U.expected_logits(cfg, w, t, want)
    assert len(want) == len(s.runner.model.trace) == 7
    for a, b in zip(s.runner.model.trace, want):
        assert torch.allclose(a, b.float(), atol=1e-3, rtol=1e-4)


def test_values_are_mixed_with_the_first_mixing_layer(models):
    """Not with the first layer, not with the one before, and the first one keeps its own."""
    cfg, w, path = models["mixed"]
    t = toks(12, cfg["vocab"], 5)
    base = U.expected_logits(cfg, w, t)
    for i, layer in enumerate(cfg["layers"]):
        name = "l%d.mix.vmix" % i
        if name not in w:
            continue
        moved = U.rel_err(U.expected_logits(cfg, {**w, name: w[name] * 0.0}, t), base)
        assert (moved > 0.01) == (bool(layer["mixer"].get("v_mix")) and i != 1), i
    model = U.session(path).runner.model
    assert [getattr(L.mixer.cores[0], "vmix", None) is not None if hasattr(L.mixer, "cores") else False
            for L in model.layers] == [False, True, True, False, False, True, True]


def test_cache_layout_and_no_state_slots(models):
    cfg, w, path = models["mixed"]
    s = U.session(path)
    lay = s.runner.model.cache_layout()
    assert [e["kind"] for e in lay] == ["latent", "kv", "kv", "kv", "latent", "kv", "kv"]
    assert lay[0]["dim"] == 9 + 4 and (lay[5]["heads"], lay[5]["dim"], lay[5]["vdim"]) == (2, 10, 6)
    assert not s.runner.model.has_state and s.runner.num_state_slots == 0


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_token_by_token_equals_prefill(models, name):
    cfg, w, path = models[name]
    t = toks(26, cfg["vocab"], 3)
    got = U.run_chunks(U.session(path), "a", t, [])
    assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL


@pytest.mark.parametrize("cuts", [(2,) * 20, (3, 2, 5, 2, 2, 9, 2), (16, 1, 1, 2, 17), (1, 36, 2)])
def test_portions(models, cuts):
    for name in ("mixed", "plain", "ones"):
        cfg, w, path = models[name]
        t = toks(40, cfg["vocab"], 4)
        got = U.run_chunks(U.session(path), "a", t, list(cuts))
        assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL, name


PLAN = [[("a", 13)], [("a", 1), ("b", 7)], [("a", 2), ("b", 1), ("c", 11)], [("a", 4), ("c", 1)],
        [("d", 2), ("b", 3), ("c", 2)], [("c", 1), ("d", 1)], [("e", 9), ("d", 6), ("c", 1)],
        [("e", 1), ("f", 14), ("d", 1)], [("e", 2), ("f", 1)], [("g", 5), ("f", 2), ("e", 1)], [("g", 1)]]


def test_mixed_batch_equals_alone_and_reuses_pages(models):
    """Portions beside decoded tokens, requests left out of steps, pages of finished requests used again."""
    for name in ("mixed", "latent_only", "plain"):
        cfg, w, path = models[name]
        total = {}
        for step in PLAN:
            for k, n in step:
                total[k] = total.get(k, 0) + n
        reqs = {k: toks(n, cfg["vocab"], 50 + i) for i, (k, n) in enumerate(sorted(total.items()))}
        s = U.session(path, max_tokens=72, page_size=4)
        got = U.run_plan(s, reqs, PLAN)
        for k, t in reqs.items():
            assert U.rel_err(got[k], U.expected_logits(cfg, w, t)) < TOL, (name, k)
        mm = s.scheduler.mm
        assert mm.get_num_free_pages() == mm.usable_pages or mm.id_allocator.get_num_used_ids() <= 1


def test_stale_page_contents_do_not_leak(models):
    cfg, w, path = models["mixed"]
    s = U.session(path, max_tokens=64, page_size=4)
    for group in (s.runner.kv_cache.k_cache, s.runner.kv_cache.v_cache):
        for x in group:
            if x is not None:
                x.fill_(37.0)
    t = toks(22, cfg["vocab"], 8)
    assert U.rel_err(U.run_chunks(s, "a", t, [1, 2, 5]), U.expected_logits(cfg, w, t)) < TOL


def test_first_tokens_of_a_sequence(models):
    for name in CONFIGS:
        cfg, w, path = models[name]
        s = U.session(path)
        for n in (1, 2, 3, 4, 5):
            t = toks(n, cfg["vocab"], 60 + n)
            for cuts in ([n], [1] * n, [max(n - 1, 1)]):
                got = U.run_chunks(s, "r%d%s" % (n, len(cuts)), t, cuts)
                assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL, (name, n, cuts)


def marked_key_probe(kind, n, back, size, page_size, device="cpu", dtype=torch.float32, heads=2, kv_heads=2, dim=32,
                     vdim=4, cuts=None, rank=None):
    """One mixer in which the last query singles out one key. The query map is the key map after a permutation of the
    input, the key maps are orthogonal, inputs have unit length and the scale is large; the last token's input is the
    permuted input of the token `back` places before it.
    -> (oracle, [outputs for several ways of cutting], the oracle with the marked token's input replaced)."""
    g = torch.Generator().manual_seed(back * 7 + page_size)
    width = dim

    def orth(k):
        return torch.linalg.qr(torch.randn(k, k, generator=g))[0]

    perm = torch.roll(torch.arange(width), 5)                  # query(h) = key(h') with h'[perm] = h
    if kind == "latent":
        # the latents are an orthogonal map of the input (padded with zeros when the latent is wider)
        rank = rank or width
        layer = U.latent(heads, dim, 2 if rank != 512 else 64, vdim, width, rank, size, scale=70.0 / width)
        w = U.random_weights(U.make_config([layer], width=width), 99)
        rd, v = layer["mixer"]["rot_dim"], orth(width)
        w["l0.mix.dkv"][:rank] = 0
        w["l0.mix.dkv"][:width] = v
        w["l0.mix.dq"] = v[:, perm]
        w["l0.mix.dq.norm"], w["l0.mix.dkv.norm"] = torch.ones(width), torch.ones(rank) * (width / rank) ** 0.5
        uq, uk = torch.zeros(heads, dim + rd, width), torch.zeros(heads, dim, rank)
        for a in range(heads):                                 # the rotated entries stay out of the scores
            uq[a, :dim] = orth(width)
            uk[a, :, :width] = uq[a, :dim]
        w["l0.mix.uq"], w["l0.mix.uk"] = uq.reshape(-1, width), uk.reshape(-1, rank)
        w["l0.mix.uv"][:, :width] *= (rank / width) ** 0.5
        w["l0.mix.sink"] = torch.full((heads,), 2.0)
    else:
        rot = 2 if kind == "rotary" else 0
        if kind == "rotary":
            layer = U.rotary(heads, kv_heads, dim, vdim, size, rot, 500.0, 2.0, scale=70.0)
        else:                                                  # whole-projection norms: entries of root mean square 1
            layer = U.distance(heads, kv_heads, dim, vdim, rows=12, bias_max=100, coef=0.1, every=50, scale=70.0 / dim)
        w = U.random_weights(U.make_config([layer], width=width), 99)
        wk = torch.stack([orth(dim) for _ in range(kv_heads)])
        wk[:, :rot] = 0                                        # the rotated entries stay out of the scores
        w["l0.mix.k"] = wk.reshape(-1, width)
        w["l0.mix.q"] = wk.repeat_interleave(heads // kv_heads, 0).reshape(-1, width)[:, perm]
        if kind == "distance":
            for a in ("q", "k"):
                w["l0.mix.%s.b" % a] *= 0
                w["l0.mix.%s.norm" % a] = torch.ones_like(w["l0.mix.%s.norm" % a])
    w = {k: t.bfloat16().float() for k, t in w.items()}
    m = U.build_mixer(layer, w, width, device, dtype)
    h = torch.randn(n, width, generator=g)
    h = h / h.norm(dim=-1, keepdim=True)
    tgt = n - 1 - back
    h[n - 1] = h[tgt][perm]                                    # the last query equals the marked token's key
    h = h.bfloat16().float()
    want = U.oracle_mixer(h, layer, w).float()
    h2 = h.clone()
    if back > 0:
        x = torch.randn(width, generator=g)
        h2[tgt] = x / x.norm()
    other = U.oracle_mixer(h2, layer, w).float()
    outs = []
    for c in cuts or [[n], [n - 1, 1], [n - back - 1, 1] + [back] * (back > 0), [max(n - 40, 1)] + [2] * 19]:
        c = [x for x in c if x > 0]
        rest = n - sum(c)
        outs.append(U.drive_mixer(m, h, c + [1] * rest, page_size, device, dtype, pool=1024))
    return want, outs, other


@pytest.mark.parametrize("page_size", [4, 16])
def test_far_keys_and_page_borders(page_size):
    n = 331
    for back in (0, 1, page_size - 1, page_size, page_size + 1, 63, 64, 65, 99, 100, 200, 329, 330):
        want, outs, other = marked_key_probe("distance", n, back, None, page_size)
        if back > 0:          # the oracle's last row rests on the marked key
            assert (want[-1] - other[-1]).abs().max() > 0.05 * want[-1].abs().max(), back
        for o in outs:
            assert torch.allclose(o, want, atol=1e-4 * want.abs().max().item(), rtol=2e-4), (page_size, back)


@pytest.mark.parametrize("kind", ["rotary", "latent"])
@pytest.mark.parametrize("size", [1, 2, 33, 64, 100])
def test_window_edges(kind, size):
    """A key just inside the window decides the last row, one just outside does not touch it."""
    n = 150
    for back in (size - 2, size - 1, size, size + 1):
        if back < 0:
            continue
        want, outs, other = marked_key_probe(kind, n, back, size, 16)
        moved = (want[-1] - other[-1]).abs().max() / want[-1].abs().max()
        if back > 0:
            assert (moved > 0.05) if back < size else (moved == 0), (size, back, moved)
        for o in outs:
            assert torch.allclose(o, want, atol=1e-4 * want.abs().max().item(), rtol=2e-4), (size, back)


def test_long_decoding(models):
    """A long prompt, then hundreds of single tokens: every window and the whole distance table are passed."""
    cfg, w, path = models["mixed"]
    t = toks(260, cfg["vocab"], 11)
    got = U.run_chunks(U.session(path, max_tokens=512, page_size=16), "a", t, [60, 3, 2])
    e = U.row_errs(got, U.expected_logits(cfg, w, t))
    assert np.median(e) < 1e-5 and e.max() < 1e-3       # a few of so many rows amplify fp32 rounding


@pytest.mark.parametrize("prefix", [False, True])
def test_greedy_generation_through_the_engine(models, prefix):
    """Prompts that share their first pages: with the prefix cache the mixed values and latents of those are reused."""
    from gllm_b200.engine.llm_engine import LLM
    cfg, w, path = models["mixed"]
    llm = LLM(path, dtype="float32", page_size=4, maxp=16, maxd=8, num_cpu_pages=64, model_max_length=96,
              log_stats=False, device="cpu", enable_prefix_caching=prefix)
    head = toks(17, cfg["vocab"], 30)
    prompts = [head + toks(4, cfg["vocab"], 31), toks(3, cfg["vocab"], 32), head + toks(9, cfg["vocab"], 33)]
    lens = [7, 12, 5]
    for _ in range(2):
        seqs = llm.generate(tokens=prompts, output_lens=lens, temperature=0.0, top_k=1)
        for p, n, s in zip(prompts, lens, seqs):
            cur = list(p)
            for _ in range(n):
                cur.append(int(oracle.forward(cfg, w, cur)[-1].argmax()))
            assert s.token_ids == cur


def test_side_benchmark_configuration_is_served():
    """The layer-like configuration of `bench.py --design liverax` (scaled down) is a valid model of this design: it
    builds with random weights and generates through the engine."""
    import os
    import sys
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    from benchmarks.liverax_bench import liverax_cfg
    from gllm_b200.engine.llm_engine import LLM
    cfg = liverax_cfg(128, 1, 97, window=12, latent=(24, 32, 16, 16))
    assert [L["type"] for L in cfg["layers"]] == ["attention_2", "attention", "latent_attention", "attention"]
    cfg["torch_dtype"] = "float32"
    llm = LLM(cfg, load_format="dummy", page_size=4, maxp=16, maxd=4, num_cpu_pages=32, model_max_length=64,
              log_stats=False, device="cpu")
    seqs = llm.generate(tokens=[toks(9, 97, 1), toks(4, 97, 2)], output_lens=[3, 2], temperature=0.0, top_k=1)
    assert [len(s.token_ids) for s in seqs] == [12, 6]
