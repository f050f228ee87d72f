"""A slow, plain statement of the Migurax decoder in numpy float64, one function per mechanism.

Used by the tests as the thing to compare with; it shares no code with the library. `cfg` is the
parsed config.json, `w` maps tensor names to arrays.
"""
import numpy as np


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def rotate(x, positions, base):
    """Pairs (2i, 2i+1) of the last axis of x [T, ..., dims] turned by position * base^(-2i/dims)."""
    dims = x.shape[-1]
    freq = float(base) ** (-np.arange(0, dims, 2) / dims)
    angle = np.asarray(positions, np.float64)[:, None] * freq
    angle = angle.reshape((angle.shape[0],) + (1,) * (x.ndim - 2) + (angle.shape[1],))
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * np.cos(angle) - v * np.sin(angle)
    out[..., 1::2] = v * np.cos(angle) + u * np.sin(angle)
    return out


def sink_softmax(score, sink):
    """Softmax over the last axis of score [H, T, S] (minus infinity: not seen) whose denominator
    also holds exp(sink[h])."""
    top = np.maximum(score.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(score - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - top))


def latent_attention_core(q, q_rot, c, k_rot, uk, uv, q_pos, k_pos, scale, sink):
    """q [T,H,dim], q_rot [T,H,rot], c [S,rank], k_rot [S,rot], uk [H,dim,rank], uv [H,vdim,rank]
    -> [T,H,vdim]; a query sees the keys at its own position and before it."""
    k = np.einsum("hdr,sr->shd", uk, c)
    v = np.einsum("hdr,sr->shd", uv, c)
    score = (np.einsum("thd,shd->hts", q, k) + np.einsum("thd,sd->hts", q_rot, k_rot)) * scale
    seen = k_pos[None, :] <= q_pos[:, None]
    weight = sink_softmax(np.where(seen[None], score, -np.inf), sink)
    return np.einsum("hts,shd->thd", weight, v)


def latent_attention(h, w, p, mixer, eps):
    """The whole mixer on one sequence from its start: h [T, width] -> [T, width]."""
    T, H = h.shape[0], mixer["heads"]
    D, RD, DV, R = mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    pos, base = np.arange(T), mixer["rot"]["base"]
    q = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T
    q = q.reshape(T, H, D + RD)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    o = latent_attention_core(q[:, :, :D], rotate(q[:, :, D:], pos, base), c,
                              rotate(down[:, R:], pos, base), w[p + "uk"].reshape(H, D, R),
                              w[p + "uv"].reshape(H, DV, R), pos, pos, mixer["scale"],
                              w[p + "sink"])
    return o.reshape(T, -1) @ w[p + "o"].T


def mlstm_state(heads, dim, vdim):
    """(S [H,dim,vdim], n [H,dim], m [H]) before the first token."""
    return np.zeros((heads, dim, vdim)), np.zeros((heads, dim)), np.zeros(heads)


def mlstm_step(state, q, k, v, i, f):
    """One token: q, k [H,dim], v [H,vdim], log gates i, f [H] -> (state, o [H,vdim])."""
    S, n, m = state
    top = np.maximum(f + m, i)
    keep, take = np.exp(f + m - top), np.exp(i - top)
    S = keep[:, None, None] * S + take[:, None, None] * k[:, :, None] * v[:, None, :]
    n = keep[:, None] * n + take[:, None] * k
    den = np.maximum(np.abs(np.sum(n * q, axis=1)), np.exp(-top)) + 1e-6
    return (S, n, top), np.einsum("hdv,hd->hv", S, q) / den[:, None]


def mlstm_core(q, k, v, i, f, state=None):
    """[T,H,...] -> (o [T,H,vdim], state)"""
    state = state or mlstm_state(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        state, o = mlstm_step(state, q[t], k[t], v[t], i[t], f[t])
        out.append(o)
    return np.stack(out), state


def head_norm_gate(o, gate, weight, eps):
    """o [T,H,vdim], each head over its own root mean square, then the weight of all heads' size
    and the sigmoid gate [T, H*vdim]."""
    o = o / np.sqrt(np.mean(o * o, axis=-1, keepdims=True) + eps)
    return o.reshape(o.shape[0], -1) * weight * sigmoid(gate)


def mlstm(h, w, p, mixer, eps):
    T, H, D, DV, cap = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"], mixer["gate_cap"]
    q = (h @ w[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, DV)
    i = soft_cap(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w[p + "f"].T + w[p + "f.b"], cap))
    o, _ = mlstm_core(q, k, v, i, f)
    return head_norm_gate(o, h @ w[p + "g"].T, w[p + "norm"], eps) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm}


def dense(h, w, p):
    return relu_squared(h @ w[p + "up"].T + w[p + "up.b"]) @ w[p + "down"].T + w[p + "down.b"]


def route(h, router, bias, top):
    """(chosen [T, top], weight [T, top]): the largest logits, a softmax over those alone."""
    logit = h @ router.T + bias
    chosen = np.argsort(-logit, axis=-1, kind="stable")[:, :top]
    z = np.take_along_axis(logit, chosen, axis=-1)
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return chosen, e / e.sum(axis=-1, keepdims=True)


def expert(h, up, down):
    return relu_squared(h @ up.T) @ down.T


def moe(h, w, p, mlp):
    chosen, weight = route(h, w[p + "router"], w[p + "router.b"], mlp["router"]["top"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, j = np.nonzero(chosen == e)
        if t.size:
            y = expert(h[t], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
            np.add.at(out, t, weight[t, j][:, None] * y)
    return out


def feed_forward(h, w, p, mlp):
    return dense(h, w, p) if mlp["kind"] == "dense" else moe(h, w, p, mlp)


def walk(cfg, w, tokens):
    """Yields (the residual stream after the mixer's half, after the layer) of every layer of one
    sequence, each [T, width]; first (None, the embedding)."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][np.asarray(tokens)]
    yield None, x
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixed = MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps)
        mid = x = rms_norm(alpha * x + mixed, w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = rms_norm(alpha * x + feed_forward(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"],
                         eps)
        yield mid, x


def doubles(w):
    return {k: np.asarray(v, np.float64) for k, v in w.items()}


def logits(cfg, w, tokens):
    """[T, vocab]"""
    w = doubles(w)
    x = list(walk(cfg, w, tokens))[-1][1]
    return rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T


def routing_margin(cfg, w, tokens):
    """[T]: how far each row's choice of experts is from another one, the least over the layers,
    as a share of the spread of its router's logits (infinite where nothing is left out)."""
    w = doubles(w)
    out = np.full(len(tokens), np.inf)
    for i, (mid, _) in enumerate(walk(cfg, w, tokens)):
        mlp, p = (cfg["layers"][i - 1].get("mlp") if i else None), f"l{i - 1}."
        if not mlp or mlp["kind"] != "moe" or mlp["router"]["top"] == mlp["router"]["experts"]:
            continue
        logit = mid @ w[p + "mlp.router"].T + w[p + "mlp.router.b"]
        s, top = np.sort(logit, axis=1)[:, ::-1], mlp["router"]["top"]
        out = np.minimum(out, (s[:, top - 1] - s[:, top]) / np.std(logit))
    return out
