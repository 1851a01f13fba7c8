"""Small Tibalorn configurations and random weights for the tests (shared by the CPU and GPU files)."""
import torch

from sneppx_alg_b200.models import ModelConfig, build_model, complete_config


def dense(ff):
    return ff and {"kind": "dense", "ff": ff}


def mamba2(heads, vdim, state, groups, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mlp": dense(ff),
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads, kv, dim, vdim, size, pool, rot, scale, base=10000.0, scaling=None, ff=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = scaling
    return {"type": "attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size, "pool": pool}, "rot": r, "scale": scale}}


def config(width, vocab, layers, eps=1e-5, scale=1.0, cap=20.0):
    return {"architecture": "Tibalorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_softcap": cap, "layers": layers}


# every size differs from its neighbours; a block longer than its window, odd sizes, conv 1 and 6, values wider than a tile
ODD = config(72, 101, [
    mamba2(6, 10, 20, 3, 4, 2, 40),
    attention(6, 2, 20, 14, 24, 5, 8, 0.3, 500.0, yarn(4.0, 64, 6.0, 1.0), 88),
    mamba2(2, 130, 5, 1, 6, 5),
    attention(3, 3, 17, 22, 7, 16, 16, 0.4, 1e4),
    mamba2(3, 7, 33, 1, 1, 3),
], eps=1e-3, scale=1.7, cap=9.0)
# sizes that the tensor-core kernels take; an epsilon at which rows that nearly cancel do not amplify bf16 rounding
TENSOR = config(128, 160, [
    mamba2(4, 64, 128, 2, 4, 4),
    attention(8, 2, 64, 64, 48, 8, 32, 0.2, 1e5, yarn(8.0, 256, 16.0, 2.0), 96),
    mamba2(2, 72, 40, 1, 3, 1, 64),
    attention(20, 1, 40, 72, 130, 3, 40, 0.25),
    mamba2(2, 32, 200, 2, 4, 2),
    attention(4, 2, 136, 128, 5, 2, 0, 0.1),
], eps=2e-2, scale=0.8)
CONFIGS = {"odd": ODD, "tensor": TENSOR}


def make_weights(cfg, seed=0):
    """Random checkpoint tensors (bf16-representable fp32) for a configuration."""
    gen = torch.Generator().manual_seed(seed)

    def rnd(*shape):
        return torch.randn(*shape, generator=gen)

    d = cfg["width"]
    W = {"embed": rnd(cfg["vocab"], d)}

    def lin(name, out, inp):
        W[name] = rnd(out, inp) / inp ** 0.5

    def norm(name):
        W[name], W[name + ".b"] = 1 + 0.2 * rnd(d), 0.2 * rnd(d)

    norm("final.norm")
    for i, s in enumerate(cfg["layers"]):
        p, m = f"l{i}.", s["mixer"]
        q = p + "mix."
        norm(p + "norm1")
        if s["type"] == "mamba2":
            H, inner = m["heads"], m["heads"] * m["vdim"]
            c = inner + 2 * m["groups"] * m["state"]
            lin(q + "in", inner + c + H, d)
            W[q + "conv"], W[q + "conv.b"] = rnd(c, m["conv"]) * 0.6, 0.3 * rnd(c)
            W[q + "dt_bias"], W[q + "A_log"], W[q + "D"] = rnd(H) - 1, 0.7 * rnd(H) - 0.5, 1 + 0.5 * rnd(H)
            W[q + "norm"] = 1 + 0.2 * rnd(inner)
            lin(q + "o", d, inner)
        else:
            H, G, k, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, r in (("q", H * k), ("k", G * k), ("v", G * v)):
                lin(q + n, r, d)
                W[q + n + ".b"] = 0.5 * rnd(r)
            W[q + "temp"], W[q + "sink"] = 1 + 0.4 * rnd(H), rnd(H)
            W[q + "temp"][-1] = -0.7
            lin(q + "g", H * v, d)
            lin(q + "o", d, H * v)
        if s["mlp"] is not None:
            norm(p + "norm2")
            lin(p + "mlp.up", s["mlp"]["ff"], d)
            lin(p + "mlp.down", d, s["mlp"]["ff"])
    return {k: t.bfloat16().float() for k, t in W.items()}


def make_model(cfg, W, dtype=torch.float32, device="cpu"):
    model = build_model(complete_config(ModelConfig.from_dict(cfg), W), dtype=dtype, device=device)
    model.load_reference_state_dict(W)
    return model
