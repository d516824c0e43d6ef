"""Helpers of the Vikupel tests: small configurations, random checkpoints on disk, comparisons. The replay session and
the portion / plan drivers are the ones the other layer-list designs' tests use."""
import json
import os

import torch

import vikupel_oracle as oracle
from bevovik_util import DictReader, drive_mixer, rel_err, row_errs, run_chunks, run_plan, session  # noqa: F401
from conftest import scratch_dir

BANDS = {"factor": 3.0, "high": 5.0, "low": 1.5, "original": 40}


def dense(ff=24):
    return {"kind": "dense", "ff": ff}


def mamba(heads=4, groups=2, state=8, vdim=6, conv=4, norm_groups=2, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim,
                                                    "conv": conv, "norm_groups": norm_groups}}


def window(heads=4, kv_heads=2, dim=8, vdim=6, size=7, scale=0.4, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                                       "scale": scale, "mask": {"size": size}}}


def turned(heads=4, kv_heads=2, dim=8, vdim=6, rot_dims=4, base=90.0, scaling=BANDS, scale=0.6, mlp=None):
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(scaling)
    return {"type": "attention_2", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim,
                                                         "vdim": vdim, "scale": scale, "rot": rot}}


def make_config(layers, vocab=61, width=20, eps=1e-5, mult=0.6, side=5, loop=None):
    cfg = {"architecture": "Vikupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
           "residual_mult": mult}
    if side:
        cfg["token_side"] = {"dim": side}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed=0):
    """name -> bf16-representable fp32 tensor, in checkpoint naming."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    wd, v, n = cfg["width"], cfg["vocab"], len(cfg["layers"])
    side = (cfg.get("token_side") or {}).get("dim", 0)

    def rnd(name, *shape, std=1.0, mean=0.0):
        w[name] = torch.randn(*shape, generator=g) * std + mean

    def uni(name, lo, hi, *shape):
        w[name] = torch.rand(*shape, generator=g) * (hi - lo) + lo

    def lin(name, out, inp, gain=1.0):
        rnd(name, out, inp, std=gain * inp ** -0.5)

    rnd("embed", v, wd)
    lin("head", v, wd, 3.0)
    rnd("final.norm", wd, std=0.2, mean=1.0)
    if side:
        rnd("side.embed", v, n * side)
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        q = p + "mix."
        rnd(p + "norm1", wd, std=0.2, mean=1.0)
        if L["type"] == "mamba2":
            h, inner, bc = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
            lin(q + "in", 2 * inner + 2 * bc + h, wd, 1.5)
            rnd(q + "conv", inner + 2 * bc, m["conv"], std=0.6)
            rnd(q + "conv.b", inner + 2 * bc, std=0.3)
            uni(q + "dt_bias", -3.0, 1.0, h)
            uni(q + "A_log", -2.0, 1.0, h)
            rnd(q + "D", h)
            rnd(q + "norm", inner, std=0.2, mean=1.0)
            lin(q + "o", wd, inner, 2.0)
        else:
            h, kv, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            lin(q + "q", h * d, wd, 2.0)
            lin(q + "k", kv * d, wd, 2.0)
            lin(q + "v", kv * dv, wd, 2.0)
            lin(q + "o", wd, h * dv, 2.0)
            if L["type"] == "attention":
                uni(q + "r1", 0.2, 1.5, h)
                uni(q + "r2", 0.05, 2.0, h)
                lin(q + "g", h * dv, wd, 2.0)
        if L["mlp"]:
            f = L["mlp"]["ff"]
            lin(p + "mlp.gate", f, wd, 1.5)
            lin(p + "mlp.up", f, wd, 1.5)
            lin(p + "mlp.down", wd, f, 2.0)
        if side:
            lin(p + "side.gate", side, wd)
            lin(p + "side.proj", wd, side, 2.0)
            rnd(p + "side.norm", wd, std=0.2, mean=0.7)
    return {k: t.bfloat16().float() for k, t in w.items()}     # exactly what the bf16 checkpoint holds


def save_model(cfg, weights):
    from safetensors.torch import save_file
    d = scratch_dir("vikupel_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.bfloat16().contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


def expected_logits(cfg, weights, tokens, trace=None):
    return oracle.forward(cfg, weights, tokens, trace).float().numpy()


def build_mixer(layer_cfg, w, width, device="cpu", dtype=torch.float32, eps=1e-5, pre="l0."):
    """The layer's mixer (with its feed-forward as a branch, when it has one) from checkpoint tensors."""
    from gllm_b200.models.hybrid import HybridSpec, make_parallel_mixer
    spec = HybridSpec("vikupel", width, 61, eps, 1.0, [layer_cfg], dtype=dtype, block="parallel", ff_act="silu_gate")
    mlp = layer_cfg["mlp"]
    m = make_parallel_mixer(layer_cfg["type"], dict(layer_cfg["mixer"]), int(mlp["ff"]) if mlp else 0, spec, device)

    def put(p, t):
        assert tuple(p.shape) == tuple(t.shape)
        p.data.copy_(t) if isinstance(p, torch.nn.Parameter) else p.copy_(t)

    m.load(DictReader(w), pre + "mix.", put, pre + "mlp.")
    return m


def oracle_mixer(h, layer_cfg, w, eps=1e-5, pre="l0."):
    h = h.double()
    y = oracle.MIXERS[layer_cfg["type"]](h, layer_cfg["mixer"], w, pre + "mix.", eps)
    return y + oracle.feed_forward(h, w, pre + "mlp.") if layer_cfg["mlp"] else y
