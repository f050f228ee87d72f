"""Small random Migurax models for the tests of that class."""
import numpy as np

from revitar_cases import to_bf16


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def latent(heads, dim, rot, vdim, rank, q_rank, mlp, scale=None, base=10000.0):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                      "q_rank": q_rank, "scale": (dim + rot) ** -0.5 if scale is None else scale,
                      "rot": {"base": base, "dims": rot}}, "mlp": mlp}


def memory(heads, dim, vdim, mlp, cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": mlp}


def config(vocab, width, layers, alpha=1.6, eps=1e-5):
    return {"architecture": "Migurax", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "postln_alpha": alpha, "layers": layers}


# Every size differs from the others, layers differ from one another, and the values that are
# easily taken for granted (1, equal sizes, multiples of eight) are other values here.
MIXED = config(203, 88, [
    memory(3, 24, 40, moe(7, 3, 56)),
    latent(5, 18, 10, 26, 44, 36, dense(70), base=500.0),
    memory(2, 36, 12, None, cap=4.0),
    latent(4, 40, 24, 16, 64, 50, moe(5, 5, 33), scale=0.09),
    memory(1, 70, 66, dense(44), cap=15.0),
])
ONE = config(95, 64, [latent(1, 64, 64, 64, 128, 64, moe(1, 1, 64), base=1.0),
                      memory(1, 64, 64, dense(64), cap=1.0)], alpha=1.0)
UNEVEN = config(131, 52, [latent(3, 20, 2, 12, 10, 14, moe(3, 2, 10)),
                          memory(5, 6, 10, moe(4, 1, 18))], alpha=0.7, eps=3e-3)
ATTENTION = config(77, 72, [latent(6, 32, 16, 24, 40, 48, None), latent(2, 8, 8, 56, 72, 8,
                                                                         dense(96))])
MEMORY = config(101, 64, [memory(4, 16, 32, dense(50)), memory(2, 33, 31, moe(9, 4, 24))])
WIDE = config(301, 320, [latent(20, 72, 64, 136, 264, 150, moe(16, 4, 128)),
                         memory(3, 160, 200, dense(400)), memory(2, 270, 96, None)])
# nothing here is a multiple of four
ODD = config(67, 45, [memory(3, 7, 9, dense(21)), latent(3, 9, 6, 11, 13, 11, moe(5, 2, 19)),
                      memory(1, 35, 33, moe(3, 1, 13)), latent(1, 7, 2, 5, 9, 7, dense(17))])
# value columns beyond the prompt attention's, key columns beyond the chunks': other kernels step in
LARGE = config(90, 64, [latent(3, 24, 8, 200, 40, 32, dense(64)), memory(1, 530, 24, None),
                        latent(2, 360, 16, 16, 24, 16, None)])
MODELS = {"attention": ATTENTION, "large": LARGE, "odd": ODD, "memory": MEMORY, "mixed": MIXED, "one": ONE, "uneven": UNEVEN,
          "wide": WIDE}


def weights(cfg, seed):
    """Random tensors (float32, bfloat16 values). Queries are large, so that scores spread over
    several units and single keys matter. In the matrix memory a token's query leans towards its own
    key: a read-out next to zero is all rounding once its head's norm has made it one. The forget
    gates' biases spread from fading within a few tokens to keeping hundreds."""
    rng = np.random.Generator(np.random.PCG64(seed))
    W, V = cfg["width"], cfg["vocab"]
    n = lambda *s, std=1.0: to_bf16(rng.standard_normal(s) * std)
    lin = lambda rows, cols, std=1.0: n(rows, cols, std=std * cols ** -0.5)
    near1 = lambda k, c=1.0: to_bf16(c * (1 + 0.2 * rng.standard_normal(k)))
    w = {"embed": n(V, W), "head": lin(V, W), "final.norm": near1(W)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        x, H, D, DV = p + "mix.", m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = near1(W)
        w[x + "o"] = lin(W, H * DV)
        if l["type"] == "mlstm":
            w[x + "k"] = lin(H * D, W, 1.5)
            w[x + "q"] = to_bf16(0.6 * w[x + "k"] + lin(H * D, W, 1.2))
            w[x + "v"], w[x + "g"] = lin(H * DV, W), lin(H * DV, W, 2.0)
            w[x + "i"], w[x + "f"] = lin(H, W, 1.5), lin(H, W, 1.0)
            w[x + "i.b"] = to_bf16(rng.uniform(-2, 2, H))
            w[x + "f.b"] = to_bf16(rng.uniform(0.5, 6, H))
            w[x + "norm"] = near1(H * DV)
        else:
            R, RD, Q = m["kv_rank"], m["rot_dim"], m["q_rank"]
            w[x + "dq"], w[x + "dq.norm"] = lin(Q, W), near1(Q, 1.5)
            w[x + "uq"] = lin(H * (D + RD), Q)
            w[x + "dkv"], w[x + "dkv.norm"] = lin(R + RD, W, 1.5), near1(R, 1.3)
            w[x + "uk"], w[x + "uv"] = lin(H * D, R), lin(H * DV, R)
            w[x + "sink"] = to_bf16(rng.uniform(-2, 4, H))
        if not l["mlp"]:
            continue
        w[p + "norm2"] = near1(W)
        q = p + "mlp."
        if l["mlp"]["kind"] == "dense":
            F = l["mlp"]["ff"]
            w[q + "up"], w[q + "up.b"] = lin(F, W), n(F, std=0.5)
            w[q + "down"], w[q + "down.b"] = lin(W, F), n(W, std=0.5)
            continue
        E, F = l["mlp"]["router"]["experts"], l["mlp"]["expert"]["ff"]
        w[q + "router"], w[q + "router.b"] = lin(E, W, 2.0), n(E, std=0.7)
        for e in range(E):
            w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = lin(F, W), lin(W, F)
    return w
