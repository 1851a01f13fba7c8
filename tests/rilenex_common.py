"""Small Rilenex configurations and random weights for the tests (shared by the CPU and GPU files)."""
import torch

from sneppx_alg_b200.models import ModelConfig, build_model, complete_config


def hgrn2(heads, dim, vdim, ff=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": ff and {"kind": "dense", "ff": ff}}


def attn(heads, kv, dim, vdim, conv, size, rot, scale, base=10000.0):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": size},
            "rot": {"base": base, "dims": rot}, "scale": scale}


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(left, right, ls, rs, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": ls, "right_scale": rs},
            "mlp": ff and {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Rilenex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


RANKS = (5, 9)   # decay and gate ranks of the random weights

# every size differs from its neighbours; odd value sizes, a layer without feed-forward, unequal chunk lengths, conv 1 and 5
ODD = config(72, 101, [
    hgrn2(3, 20, 12, 40),
    parallel(attn(6, 2, 24, 20, 4, 24, 16, 0.3), delta(4, 2, 12, 21, 2), 0.7, -1.1, 88),
    hgrn2(2, 40, 9, None),
    parallel(attn(3, 3, 16, 40, 1, 40, 16, 0.4, 500.0), delta(3, 1, 36, 8, 5), 1.5, 0.6, None),
], eps=1e-3)
# sizes that the tensor-core kernels take
TENSOR = config(128, 160, [
    parallel(attn(8, 4, 64, 64, 3, 48, 32, 0.2), delta(4, 4, 64, 32, 4), 1.3, 0.8, 96),
    hgrn2(2, 64, 48, 96),
    parallel(attn(16, 2, 32, 72, 4, 200, 32, 0.25), delta(2, 2, 128, 72, 3), 0.9, 1.2, 64),
    hgrn2(2, 128, 16, None),
])
CONFIGS = {"odd": ODD, "tensor": TENSOR}


def make_weights(cfg, seed=0):
    """Random checkpoint tensors (bf16-representable fp32) for a configuration."""
    gen = torch.Generator().manual_seed(seed)

    def rnd(*shape):
        return torch.randn(*shape, generator=gen)

    W, d = {"embed": rnd(cfg["vocab"], cfg["width"]), "final.norm": 1 + 0.2 * rnd(cfg["width"]),
            "head": rnd(cfg["vocab"], cfg["width"]) / cfg["width"] ** 0.5}, cfg["width"]

    def lin(name, out, inp):
        W[name] = rnd(out, inp) / inp ** 0.5

    for i, s in enumerate(cfg["layers"]):
        p, m = f"l{i}.", s["mixer"]
        W[p + "norm1"] = 1 + 0.2 * rnd(d)
        if s["type"] == "hgrn2":
            H, k, v = m["heads"], m["dim"], m["vdim"]
            for n, r in (("q", H * k), ("f", H * k), ("v", H * v)):
                lin(p + "mix." + n, r, d)
            W[p + "mix.f.b"], W[p + "mix.lower"] = 1 + rnd(H * k), torch.rand(H * k, generator=gen) * 0.9
            W[p + "mix.norm"] = 1 + 0.2 * rnd(v)
            lin(p + "mix.o", d, H * v)
        else:
            a, q = m["left"], p + "mix.left."
            H, G, k, v, taps = a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["conv"]
            for n, r in (("q", H * k), ("k", G * k), ("v", G * v)):
                lin(q + n, r, d)
                W[q + n + ".conv"] = rnd(r, taps) * 0.6
            lin(q + "g", H, d)
            lin(q + "o", d, H * v)
            W[q + "q.norm"], W[q + "k.norm"] = 1 + 0.3 * rnd(k), 1 + 0.3 * rnd(k)
            W[q + "talk"] = torch.eye(H) * 0.8 + 0.3 * rnd(H, H)
            a, q = m["right"], p + "mix.right."
            H, G, k, v, taps = a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["conv"]
            for n, r in (("q", G * k), ("k", G * k), ("v", H * v)):
                lin(q + n, r, d)
                W[q + n + ".conv"] = rnd(r, taps) * 0.6
            lin(q + "b", H, d)
            lin(q + "a1", RANKS[0], d)
            lin(q + "a2", H * k, RANKS[0])
            lin(q + "g1", RANKS[1], d)
            lin(q + "g2", H * v, RANKS[1])
            lin(q + "o", d, H * v)
            W[q + "A_log"], W[q + "dt_bias"] = rnd(H) * 0.5, rnd(H * k) - 2
            W[q + "norm"] = 1 + 0.2 * rnd(v)
        if s["mlp"] is not None:
            W[p + "norm2"] = 1 + 0.2 * rnd(d)
            lin(p + "mlp.up", s["mlp"]["ff"], d)
            lin(p + "mlp.down", d, s["mlp"]["ff"])
            W[p + "mlp.act"] = rnd(2)
    return {k: t.bfloat16().float() for k, t in W.items()}


def make_model(cfg, W, dtype=torch.float32, device="cpu"):
    model = build_model(complete_config(ModelConfig.from_dict(cfg), W), dtype=dtype, device=device)
    model.load_reference_state_dict(W)
    return model
