"""Helpers of the Liverax tests: small configurations, random checkpoints on disk, comparisons. The replay session and
the portion / plan drivers are the ones the other layer-list designs' tests use."""
import json
import os

import torch

import liverax_oracle as oracle
from bevovik_util import DictReader, drive_mixer, rel_err, row_errs, run_chunks, run_plan, session  # noqa: F401
from conftest import scratch_dir


def dense(ff=24):
    return {"kind": "dense", "ff": ff}


def rotary(heads=4, kv_heads=2, dim=8, vdim=6, size=7, rot_dims=4, base=90.0, factor=3.0, scale=0.5, v_mix=False, mlp=None):
    rot = {"base": base, "dims": rot_dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot, "mask": {"size": size}}
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mlp": mlp, "mixer": m}


def distance(heads=4, kv_heads=2, dim=8, vdim=6, rows=10, bias_max=29, coef=0.4, every=5, scale=0.4, v_mix=False,
             mlp=None):
    """`rows` is the number of rows of the checkpoint's distance table; config.json does not hold it."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
         "_rows": rows}
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention_2", "mlp": mlp, "mixer": m}


def latent(heads=3, dim=6, rot_dim=4, vdim=5, q_rank=10, kv_rank=9, size=6, base=300.0, scale=0.6, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot_dim}, "mask": {"size": size}}}


def make_config(layers, vocab=61, width=20, eps=1e-5, cap=12.0):
    cfg = {"architecture": "Liverax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


def random_weights(cfg, seed=0):
    """name -> bf16-representable fp32 tensor, in checkpoint naming."""
    g = torch.Generator().manual_seed(seed)
    w, wd, v = {}, cfg["width"], cfg["vocab"]

    def rnd(name, *shape, std=1.0, mean=0.0):
        w[name] = torch.randn(*shape, generator=g) * std + mean

    def lin(name, out, inp, gain=1.0):
        rnd(name, out, inp, std=gain * inp ** -0.5)

    rnd("embed", v, wd)
    w["embed"] += 0.7                                  # a mean that only a layer norm takes off
    lin("head", v, wd, 3.0)
    rnd("final.norm", wd, std=0.2, mean=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        q, h, d, dv = p + "mix.", m["heads"], m["dim"], m["vdim"]
        rnd(p + "norm1", wd, std=0.2, mean=1.0)
        if L["type"] == "latent_attention":
            r, k, rd = m["q_rank"], m["kv_rank"], m["rot_dim"]
            lin(q + "dq", r, wd, 2.0)
            rnd(q + "dq.norm", r, std=0.3, mean=1.0)
            lin(q + "uq", h * (d + rd), r, 2.0)
            lin(q + "dkv", k + rd, wd, 2.0)
            rnd(q + "dkv.norm", k, std=0.3, mean=1.0)
            lin(q + "uk", h * d, k, 2.0)
            lin(q + "uv", h * dv, k, 2.0)
            rnd(q + "sink", h, std=1.0, mean=1.0)
        else:
            kv = m["kv_heads"]
            lin(q + "q", h * d, wd, 2.0)
            lin(q + "k", kv * d, wd, 2.0)
            lin(q + "v", kv * dv, wd, 2.0)
            w[q + "vmix"] = torch.rand((), generator=g) * 0.6 + 0.2
        if L["type"] == "attention_2":
            for n, rows in (("q", h * d), ("k", kv * d), ("v", kv * dv)):
                rnd(q + n + ".b", rows, std=0.7)
            rnd(q + "q.norm", h * d, std=0.3, mean=1.0)
            rnd(q + "k.norm", kv * d, std=0.3, mean=1.0)
            rnd(q + "rel", m["_rows"], h, std=1.5)
        if L["type"] != "attention":
            lin(q + "g", h * dv, wd, 2.0)
        lin(q + "o", wd, h * dv, 2.0)
        if L["mlp"]:
            f = L["mlp"]["ff"]
            rnd(p + "norm2", wd, std=0.2, mean=1.0)
            lin(p + "mlp.gate", f, wd, 1.5)
            lin(p + "mlp.up", f, wd, 1.5)
            lin(p + "mlp.down", wd, f, 2.0)
    return {k: t.bfloat16().float() for k, t in w.items()}     # exactly what the bf16 checkpoint holds


def plain(cfg):
    """The configuration as config.json holds it."""
    return {**cfg, "layers": [{**L, "mixer": {k: v for k, v in L["mixer"].items() if not k.startswith("_")}}
                              for L in cfg["layers"]]}


def save_model(cfg, weights):
    from safetensors.torch import save_file
    d = scratch_dir("liverax_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(plain(cfg), f)
    save_file({k: v.bfloat16().contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


def expected_logits(cfg, weights, tokens, trace=None):
    return oracle.forward(cfg, weights, tokens, trace).float().numpy()


def build_mixer(layer_cfg, w, width, device="cpu", dtype=torch.float32, eps=1e-5, pre="l0."):
    from gllm_b200.models.hybrid import HybridSpec, make_mixer
    spec = HybridSpec("liverax", width, 61, eps, 1.0, [layer_cfg], dtype=dtype, block="prenorm", center_norm=True,
                      ff_act="gelu_gate")
    m = dict(layer_cfg["mixer"])
    if "_rows" in m:
        m["bias_rows"] = m.pop("_rows")
    mixer = make_mixer(layer_cfg["type"], m, spec, device)

    def put(p, t):
        assert tuple(p.shape) == tuple(t.shape)
        p.data.copy_(t) if isinstance(p, torch.nn.Parameter) else p.copy_(t)

    mixer.load(DictReader(w), pre + "mix.", put)
    return mixer


def oracle_mixer(h, layer_cfg, w, eps=1e-5, pre="l0.", first=None):
    return oracle.MIXERS[layer_cfg["type"]](h.double(), layer_cfg["mixer"], w, pre + "mix.", eps,
                                            {} if first is None else {"v": first.double()})
