"""GPU: the mechanisms of the Migurax class one by one, and whole models in prompts, portions,
decoding, batches and greedy generation, against the plain float64 statement."""
import ctypes
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import plain_migurax as plain
from conftest import ROOT, rel_err
from migurax_cases import MODELS, weights
from revitar_cases import to_bf16, write_model
from test_revitar_gpu import BF16, F32, Case, compute, padded, to_dev, u32, up8  # noqa: F401

pytestmark = pytest.mark.gpu
f32 = lambda a: np.ascontiguousarray(a, np.float32)
f64 = lambda a: np.asarray(a, np.float64)


def dev(torch, a):
    return torch.from_numpy(f32(a)).cuda()


def guarded(torch, rows, cols):
    """Room for `rows` results and a guard row of NaN behind them."""
    return torch.full((rows + 1, cols), float("nan"), device="cuda")


def unguard(ctx, t):
    ctx.sync()
    a = t.float().cpu().numpy()
    assert np.isnan(a[-1]).all()  # nothing past the last row
    return a[:-1]


# ----------------------------------------------------- products, experts, residual step ----
@pytest.mark.parametrize("compute", [F32, BF16])
@pytest.mark.parametrize("rows, cols", [(50, 72), (300, 200), (130, 518)])
def test_linear_with_bias_and_squared_relu(ctx, torch_cuda, compute, rows, cols):
    torch = torch_cuda
    rng = np.random.Generator(np.random.PCG64(rows))
    w, b = to_bf16(rng.standard_normal((rows, cols))), f32(rng.standard_normal(rows) * 5)
    wd, bd = to_dev(torch, padded(w, up8(cols)), compute), dev(torch, b)
    for T in (1, 2, 3, 40, 200):
        x = to_bf16(rng.standard_normal((T, cols)))
        xd = to_dev(torch, padded(x, up8(cols)), compute)
        ref = f64(x) @ f64(w).T + b
        for path in (1, 2):
            if path == 1 and (T > 2 or compute == F32 and cols % 8):
                continue
            for relu2 in (0, 1):
                y = guarded(torch, T, rows)
                ctx.call("kanso_cuda_dense_linear_act", compute, wd.data_ptr(), xd.data_ptr(),
                         bd.data_ptr(), relu2, y.data_ptr(), T, rows, cols, path)
                want = plain.relu_squared(ref) if relu2 else ref
                assert rel_err(unguard(ctx, y), want) <= 4e-6, (T, path, relu2)


@pytest.mark.parametrize("compute", [F32, BF16])
@pytest.mark.parametrize("experts, top, width, ff", [(5, 2, 72, 40), (1, 1, 64, 24), (40, 7, 52, 33),
                                                     (6, 6, 200, 130), (130, 3, 128, 64)])
def test_experts(ctx, torch_cuda, compute, experts, top, width, ff):
    torch = torch_cuda
    rng = np.random.Generator(np.random.PCG64(experts * 31 + top))
    w = {"router": to_bf16(rng.standard_normal((experts, width)) * 2 * width ** -0.5),
         "router.b": f32(rng.standard_normal(experts))}
    for e in range(experts):
        w[f"e{e}.up"] = to_bf16(rng.standard_normal((ff, width)) * width ** -0.5)
        w[f"e{e}.down"] = to_bf16(rng.standard_normal((width, ff)) * ff ** -0.5)
    stack = lambda n, ld: to_dev(torch, padded(np.stack([w[f"e{e}.{n}"] for e in range(experts)]),
                                               up8(ld)), compute)
    router, bias = dev(torch, padded(w["router"], up8(width))), dev(torch, w["router.b"])
    up, down = stack("up", width), stack("down", ff)
    w64 = plain.doubles(w)
    mlp = {"router": {"experts": experts, "top": top}}
    for T, paths in ((1, (1, 2)), (2, (1, 2)), (40, (2,)), (333, (2,))):
        # inputs whose choice of experts is not a close call
        x = to_bf16(rng.standard_normal((8 * T, width)))
        s = np.sort(f64(x) @ w64["router"].T + w64["router.b"], axis=1)[:, ::-1]
        gap = s[:, top - 1] - s[:, top] if top < experts else np.ones(len(s))
        x = x[np.argsort(-gap)[:T]]
        ref = plain.moe(f64(x), w64, "", mlp)
        xd = dev(torch, x)
        for path in paths:
            y = guarded(torch, T, width)
            ctx.call("kanso_cuda_moe_relu2", compute, xd.data_ptr(), router.data_ptr(),
                     bias.data_ptr(), up.data_ptr(), down.data_ptr(), y.data_ptr(), T, width, ff,
                     experts, top, path)
            assert rel_err(unguard(ctx, y), ref) <= (4e-6 if compute == F32 else 1e-2), (T, path)


@pytest.mark.parametrize("width", [64, 50, 1000])
def test_residual_step(ctx, torch_cuda, width):
    torch = torch_cuda
    rng = np.random.Generator(np.random.PCG64(width))
    x, y, w = rng.standard_normal((7, width)), rng.standard_normal((7, width)), rng.standard_normal(width)
    x, y, w = f32(x), f32(y), f32(w)
    for eps in (1e-6, 0.5):
        for after, ref in ((1, plain.rms_norm(1.7 * f64(x) + y, f64(w), eps)),
                           (0, x + 1.7 * plain.rms_norm(f64(y), f64(w), eps))):
            xd = guarded(torch, 7, width)
            xd[:7] = dev(torch, x)
            yd, wd = dev(torch, y), dev(torch, w)
            ctx.call("kanso_cuda_residual_norm", xd.data_ptr(), yd.data_ptr(), wd.data_ptr(), eps,
                     1.7, after, 7, width)
            assert rel_err(unguard(ctx, xd), ref) <= 1e-6, (after, eps)


# ------------------------------------------------------------------- latent attention ----
class LatentCase:
    """One sequence's latents and rotated key parts in a pool with permuted pages, stored from down
    projections through kanso_cuda_latent_store. `raw` [n][rank + rot] is what is projected."""

    def __init__(self, kb, ctx, torch, rng, raw, c_norm, rank, base, bs, compute, first=0, spare=3,
                 eps=1e-5):
        self.kb, self.ctx, self.torch, self.compute = kb, ctx, torch, compute
        n, rot = raw.shape[0], raw.shape[1] - rank
        self.n, self.rank, self.rot, self.base = n, rank, rot, base
        self.first, self.nb = first, (first + n + bs - 1) // bs
        layers = np.array([[1, rank + rot, 0, 0, 0, 0]], np.uint32)
        self.pool = kb.KvPool.of_layers(ctx, layers, self.nb + spare, bs,
                                        kb.KV_F32 if compute == F32 else kb.KV_BF16)
        self.tables = u32(torch, rng.permutation(self.nb + spare)[:self.nb])
        q_rank, q_norm = 13, f32(rng.standard_normal(13))
        down = f32(np.concatenate([rng.standard_normal((n, q_rank)), raw], axis=1))
        cq = torch.full((n + 1, up8(q_rank)), float("nan"), device="cuda",
                        dtype=torch.float32 if compute == F32 else torch.bfloat16)
        pos, seq = u32(torch, first + np.arange(n)), u32(torch, np.zeros(n))
        p = self.params(n, 1, 1, 1.0, None)
        keep = [dev(torch, a) for a in (down, q_norm, c_norm)]
        ctx.call("kanso_cuda_latent_store", self.pool.h, 0, keep[0].data_ptr(), q_rank,
                 keep[1].data_ptr(), keep[2].data_ptr(), eps, pos.data_ptr(), seq.data_ptr(),
                 self.tables.data_ptr(), ctypes.byref(p), cq.data_ptr())
        got = unguard(ctx, cq)
        want = plain.rms_norm(f64(down[:, :q_rank]), f64(q_norm), eps)
        assert rel_err(got[:, :q_rank], want) <= (1e-6 if compute == F32 else 5e-3)
        assert (got[:, q_rank:] == 0).all()
        self.c = plain.rms_norm(f64(f32(raw[:, :rank])), f64(f32(c_norm)), eps)
        self.k_rot = plain.rotate(f64(f32(raw[:, rank:])), first + np.arange(n), base)

    def params(self, rows, heads, dim, scale, sink):
        return self.kb.LatentAttentionParams(rows, heads, self.nb, dim, self.rot, 1, self.rank,
                                             scale, self.base,
                                             None if sink is None else sink.ctypes.data)

    def attend(self, q_lat, q, positions, scale, sink, path):
        torch, (T, H) = self.torch, q_lat.shape[:2]
        sink = f32(sink)
        out = guarded(torch, T, H * self.rank)
        pos, seq = u32(torch, positions), u32(torch, np.zeros(T))
        p = self.params(T, H, q.shape[2] - self.rot, scale, sink)
        ql, qq = dev(torch, q_lat), dev(torch, q)
        self.ctx.call("kanso_cuda_latent_attention", self.pool.h, 0, ql.data_ptr(), qq.data_ptr(),
                      pos.data_ptr(), seq.data_ptr(), self.tables.data_ptr(), out.data_ptr(),
                      ctypes.byref(p), path)
        return unguard(self.ctx, out).reshape(T, H, self.rank)

    def reference(self, q_lat, q, positions, scale, sink):
        """The plain attention with the identity for both projections of the latent."""
        T, H = q_lat.shape[:2]
        eye = np.broadcast_to(np.eye(self.rank), (H, self.rank, self.rank))
        rot = plain.rotate(f64(f32(q))[:, :, -self.rot:], positions, self.base)
        return plain.latent_attention_core(f64(f32(q_lat)), rot, self.c, self.k_rot, eye, eye,
                                           np.asarray(positions), self.first + np.arange(self.n),
                                           scale, f64(f32(sink)))


@pytest.mark.parametrize("compute, path", [(F32, 1), (BF16, 1), (BF16, 2)])
@pytest.mark.parametrize("H, rank, rot, bs, n, scale, base", [
    (6, 44, 10, 16, 150, 0.15, 500.0),
    (1, 8, 2, 5, 40, 1.0, 10000.0),
    (16, 128, 32, 16, 300, 0.1, 20000.0),
    (19, 130, 64, 8, 200, 0.07, 1e6),
    (33, 264, 6, 32, 333, 0.05, 50.0),
    (5, 512, 64, 16, 700, 0.04, 10000.0),
    (3, 640, 16, 16, 129, 0.03, 3.0),
    (4, 40, 24, 64, 500, 0.1, 700.0),
])
def test_latent_attention(kb, ctx, torch_cuda, compute, path, H, rank, rot, bs, n, scale, base):
    torch = torch_cuda
    rng = np.random.Generator(np.random.PCG64(H * 1000 + rank + n))
    case = LatentCase(kb, ctx, torch, rng, rng.standard_normal((n, rank + rot)) * 2,
                      rng.uniform(0.5, 1.5, rank), rank, base, bs, compute)
    sink = rng.uniform(-3, 6, H)
    if path == 2 and bs == 5:  # pages that do not make up a tile
        with pytest.raises(kb.KansoError) as e:
            case.attend(np.zeros((1, H, rank)), np.zeros((1, H, 7 + rot)), [n - 1], scale, sink, path)
        assert e.value.code == kb.ERR_UNSUPPORTED
        return
    for rows in (np.arange(n), [n - 1], [0, 1, n // 2], np.arange(60, 70) % n):
        rows = np.asarray(rows)
        q_lat = rng.standard_normal((len(rows), H, rank)) * 3
        q = rng.standard_normal((len(rows), H, 7 + rot)) * 3
        got = case.attend(q_lat, q, rows, scale, sink, path)
        ref = case.reference(q_lat, q, rows, scale, sink)
        assert rel_err(got, ref) <= (1e-5 if compute == F32 else 2e-2), len(rows)
    case.pool.destroy()


@pytest.mark.parametrize("compute, path", [(F32, 1), (BF16, 1), (BF16, 2)])
def test_one_loud_latent_at_every_edge(kb, ctx, torch_cuda, compute, path):
    """One key of hundreds answers the query: every later row sees it, no earlier one does, at page
    and tile borders, at the sequence's start and with the keys shared out over many CTAs."""
    torch = torch_cuda
    rng = np.random.Generator(np.random.PCG64(5))
    n, rank, rot = 700, 16, 4
    for at in (0, 1, 15, 16, 17, 31, 32, 63, 64, 65, 127, 128, 300, 511, 512):
        raw = np.zeros((n, rank + rot))
        raw[:, 1] = 4.0
        raw[at, :2] = 4.0, 0.0
        case = LatentCase(kb, ctx, torch, rng, raw, np.ones(rank), rank, 100.0, 16, compute)
        rows = np.unique([r for r in (at - 1, at, at + 1, at + 63, at + 64, at + 65, n - 1)
                          if 0 <= r < n])
        q_lat = np.zeros((len(rows), 2, rank))
        q_lat[:, :, 0], q_lat[:, :, 1] = 30.0, -30.0
        got = case.attend(q_lat, np.zeros((len(rows), 2, 3 + rot)), rows, 0.2, [-50.0, 20.0], path)
        seen = rows >= at  # the loud key's latent is (4, 0, ...), the others' (0, 4, ...)
        assert (got[seen, 0, 0] > 3.9).all() and (got[seen, 0, 1] < 0.01).all(), (at, rows)
        assert (got[~seen, 0, 0] == 0).all() and (got[~seen, 0, 1] > 3.9).all(), (at, rows)
        # its score is 24: next to a sink of 20 it keeps most of the weight, the others nothing
        assert np.allclose(got[seen, 1, 0], 4 / (1 + np.exp(20 - 24)), rtol=2e-2)
        assert (got[~seen, 1] < 1e-6).all()
        case.pool.destroy()


@pytest.mark.parametrize("compute, path", [(F32, 1), (BF16, 1), (BF16, 2)])
def test_rotation_depends_on_the_distance_alone(kb, ctx, torch_cuda, compute, path):
    """A key's rotated part answers a query's at one distance: found near and far from the start."""
    torch = torch_cuda
    rng = np.random.Generator(np.random.PCG64(6))
    n, rank, rot, base = 200, 8, 16, 64.0
    for first in (0, 100000):
        raw = rng.standard_normal((n, rank + rot)) * 0.1
        part = rng.standard_normal(rot) * 4
        raw[40, rank:] = part
        case = LatentCase(kb, ctx, torch, rng, raw, np.ones(rank), rank, base, 16, compute, first)
        if first:  # pages in front of the stored rows hold zeros: rows with no part in the sum
            case.c = np.concatenate([np.zeros((first, rank)), case.c])
            case.k_rot = np.concatenate([np.zeros((first, rot)), case.k_rot])
            case.n, case.first = first + n, 0
        rows = first + np.array([40, 55, 120, 199])
        # the part turned back: aligned with the key at a distance of 15
        q = np.zeros((4, 1, 2 + rot))
        q[:, 0, 2:] = plain.rotate(part[None], [-15], base)[0]
        got = case.attend(np.zeros((4, 1, rank)), q, rows, 0.5, [0.0], path)
        ref = case.reference(np.zeros((4, 1, rank)), q, rows, 0.5, [0.0])
        assert rel_err(got, ref) <= (2e-5 if compute == F32 else 3e-2), first
        case.pool.destroy()


def prefill(kb, ctx, torch, q, q_rot, k, v, k_rot, pos0, scale, sink):
    """kanso_cuda_softmax_prefill on padded bfloat16 arrays."""
    (T, H, D), DV, RD = q.shape, v.shape[2], k_rot.shape[1]
    b = lambda a: to_dev(torch, padded(a, up8(a.shape[-1])), BF16)
    ds = [b(a) if a.size else None for a in (q, q_rot, k, v, k_rot)]
    out = guarded(torch, T, H * DV).to(torch.bfloat16)
    s = None if sink is None else f32(sink)
    p = kb.LatentAttentionParams(T, H, 0, D, RD, DV, 1, scale, 1.0,
                                 None if s is None else s.ctypes.data)
    ctx.call("kanso_cuda_softmax_prefill", *(None if d is None else d.data_ptr() for d in ds),
             out.data_ptr(), pos0, ctypes.byref(p))
    return unguard(ctx, out).reshape(T, H, DV)


def prefill_reference(q, q_rot, k, v, k_rot, pos0, scale, sink):
    T, n = q.shape[0], k.shape[0]
    score = (np.einsum("thd,shd->hts", f64(q), f64(k)) +
             np.einsum("thd,sd->hts", f64(q_rot), f64(k_rot))) * scale
    seen = np.arange(n)[None] <= pos0 + np.arange(T)[:, None]
    sink = np.full(q.shape[1], -1e30) if sink is None else f64(f32(sink))
    w = plain.sink_softmax(np.where(seen[None], score, -np.inf), sink)
    return np.einsum("hts,shd->thd", w, f64(v))


@pytest.mark.parametrize("H, D, RD, DV, T, pos0", [
    (3, 24, 10, 40, 150, 0), (2, 128, 64, 128, 300, 77), (1, 8, 0, 8, 16, 0), (5, 40, 2, 72, 129, 64),
    (2, 72, 64, 136, 200, 63), (4, 64, 32, 192, 64, 500), (1, 192, 64, 48, 130, 1),
    (2, 20, 6, 12, 17, 47), (1, 16, 16, 16, 1, 1000),
])
def test_prompt_attention(kb, ctx, torch_cuda, H, D, RD, DV, T, pos0):
    rng = np.random.Generator(np.random.PCG64(H * 100 + D + T))
    n = pos0 + T
    r = lambda *s, std=1.0: to_bf16(rng.standard_normal(s) * std)
    scale = (D + RD) ** -0.5
    for std, sink in ((1.5, rng.uniform(-2, 5, H)), (4.0, None)):
        a = (r(T, H, D, std=std), r(T, H, RD, std=std), r(n, H, D), r(n, H, DV), r(n, RD))
        got = prefill(kb, ctx, torch_cuda, *a, pos0, scale, sink)
        assert rel_err(got, prefill_reference(*a, pos0, scale, sink)) <= 1.5e-2


@pytest.mark.parametrize("step", [0.4, -0.4, 9.0])
def test_prompt_attention_with_moving_maxima(kb, ctx, torch_cuda, step):
    """Scores that rise or fall along the keys by far more than one reference maximum covers."""
    rng = np.random.Generator(np.random.PCG64(9))
    T, D, DV = 390, 16, 24
    k, q = np.zeros((T, 1, D)), np.zeros((T, 1, D))
    k[:, 0, 0], k[:, 0, 1] = np.arange(T) // 64, np.arange(T) % 64  # exact in bfloat16
    q[:, 0, 0], q[:, 0, 1] = 64 * step, step
    v = to_bf16(rng.standard_normal((T, 1, DV)))
    a = (to_bf16(q), np.zeros((T, 1, 0)), k, v, np.zeros((T, 0)))
    got = prefill(kb, ctx, torch_cuda, *a, 0, 1.0, [3.0])
    assert rel_err(got, prefill_reference(*a, 0, 1.0, [3.0])) <= 1.5e-2


def test_one_loud_key_in_a_prompt(kb, ctx, torch_cuda):
    """As with the latents, on the prompt kernel: every row against one loud key at a time."""
    T, D = 420, 16
    for at in (0, 1, 15, 16, 63, 64, 65, 127, 128, 129, 255, 256, 383, 419):
        k, v = np.zeros((T, 1, D)), np.zeros((T, 1, 8))
        k[:, 0, 1], v[:, 0, 1] = 1.0, 1.0
        k[at, 0, :2], v[at, 0, :2] = (1.0, 0.0), (1.0, 0.0)
        q = np.zeros((T, 1, D))
        q[:, 0, 0], q[:, 0, 1] = 20.0, -20.0
        got = prefill(kb, ctx, torch_cuda, q, np.zeros((T, 1, 0)), k, v, np.zeros((T, 0)), 0, 1.0,
                      [-40.0])[:, 0]
        seen = np.arange(T) >= at
        assert (got[seen, 0] > 0.99).all() and (got[~seen, 0] == 0).all(), at
        assert (got[~seen, 1] > 0.99).all(), at


def test_prompt_attention_refuses_what_it_cannot(kb, ctx, torch_cuda):
    z = lambda *s: np.zeros(s)
    for D, DV, scale in ((16, 200, 1.0), (512, 16, 1.0), (16, 16, -1.0)):
        with pytest.raises(kb.KansoError) as e:
            prefill(kb, ctx, torch_cuda, z(20, 1, D), z(20, 1, 0), z(20, 1, D), z(20, 1, DV),
                    z(20, 0), 0, scale, None)
        assert e.value.code == kb.ERR_UNSUPPORTED


# ---------------------------------------------------------------------- matrix memory ----
class Memory:
    """A pool of one recurrent layer with a few slots, all of them full of garbage at first."""

    def __init__(self, kb, ctx, torch, H, D, V, cap, slots=3):
        self.kb, self.ctx, self.torch, self.cap = kb, ctx, torch, cap
        self.H, self.D, self.V = H, D, V
        layers = np.array([[0, 0, 0, H, D, V]], np.uint32)
        self.pool = kb.KvPool.of_layers(ctx, layers, 1, 16, kb.KV_F32, slots)
        self.zero = dev(torch, np.zeros(H))
        rng = np.random.Generator(np.random.PCG64(1))
        for s in range(slots):
            self.run(*self.inputs(rng, 20), s, 0, 1)

    def inputs(self, rng, T, i=None, f=None):
        """(q, k, v, gate, z_i, z_f): bfloat16 values, gates before the cap."""
        H, D, V = self.H, self.D, self.V
        r = lambda *s: to_bf16(rng.standard_normal(s))
        return (r(T, H, D) * 2, r(T, H, D), r(T, H, V), r(T, H * V),
                f32(rng.standard_normal((T, H)) * 3 if i is None else i),
                f32(rng.standard_normal((T, H)) * 3 + 2 if f is None else f))

    def run(self, q, k, v, g, zi, zf, slot, pos0, path):
        T = q.shape[0]
        y = np.concatenate([a.reshape(T, -1) for a in (q, k, v, g, zi, zf)], axis=1)
        out = guarded(self.torch, T, self.H * self.V)
        p = self.kb.MlstmParams(T, pos0, slot, self.cap)
        yd = dev(self.torch, y)
        self.ctx.call("kanso_cuda_mlstm", self.pool.h, 0, yd.data_ptr(), self.zero.data_ptr(),
                      self.zero.data_ptr(), out.data_ptr(), ctypes.byref(p), path)
        return unguard(self.ctx, out).reshape(T, self.H, self.V)

    def reference(self, q, k, v, g, zi, zf):
        i = plain.soft_cap(f64(zi), self.cap)
        f = plain.log_sigmoid(plain.soft_cap(f64(zf), self.cap))
        return plain.mlstm_core(f64(q) * self.D ** -0.5, f64(k), f64(v), i, f)[0]

    def close(self, got, ref, tol):
        """Head by head: their sizes differ, and what follows divides them out."""
        size = np.sqrt(np.mean(ref ** 2, axis=2, keepdims=True)) + 1e-3
        return np.abs((got - ref) / size).max() <= tol


SHAPES = [(3, 24, 40), (1, 8, 8), (2, 20, 36), (4, 64, 32), (2, 130, 70), (2, 256, 64), (1, 300, 100),
          (1, 512, 96), (1, 33, 161)]


@pytest.mark.parametrize("H, D, V", SHAPES)
def test_memory_by_token_and_in_chunks(kb, ctx, torch_cuda, H, D, V):
    """Both kernels on whole prompts, in portions that hand the state from one to the other, and a
    token at a time; each in a slot that something else has used."""
    rng = np.random.Generator(np.random.PCG64(D))
    m = Memory(kb, ctx, torch_cuda, H, D, V, 7.0)
    n = 200
    a = m.inputs(rng, n)
    ref = m.reference(*a)
    for cuts in ([(n, 1)], [(n, 2)], [(64, 2), (64, 1), (72, 2)], [(1, 1), (63, 2), (2, 1), (65, 2), (69, 2)],
                 [(130, 2)] + [(1, 1)] * 70, [(17, 2)] * 11 + [(13, 1)]):
        got, at = [], 0
        for c, path in cuts:
            got.append(m.run(*(x[at:at + c] for x in a), 1, at, path))
            at += c
        # the denominator is the larger of two: near a crossing of zero it passes errors on
        assert m.close(np.concatenate(got), ref, 2e-4 if all(p == 1 for _, p in cuts) else 2e-3), cuts
    m.pool.destroy()


def test_memory_of_wide_heads(kb, ctx, torch_cuda):
    """A state too large for shared memory, and the range of the chunk kernel."""
    rng = np.random.Generator(np.random.PCG64(2))
    m = Memory(kb, ctx, torch_cuda, 1, 1700, 40, 5.0)
    a = m.inputs(rng, 30)
    got = [m.run(*(x[:29] for x in a), 0, 0, 0), m.run(*(x[29:] for x in a), 0, 29, 0)]
    assert m.close(np.concatenate(got), m.reference(*a), 2e-4)
    with pytest.raises(kb.KansoError) as e:
        m.run(*a, 0, 0, 2)
    assert e.value.code == kb.ERR_UNSUPPORTED
    with pytest.raises(kb.KansoError):
        m.run(*a, 7, 0, 1)
    m.pool.destroy()


@pytest.mark.parametrize("path", [1, 2])
def test_memory_keeps_one_token_for_long(kb, ctx, torch_cuda, path):
    """One token with an open input gate among closed ones and open forget gates: hundreds of
    tokens later a query that matches its key reads its value; before it nothing does. With the
    forget gate shut for a few tokens in between it is gone."""
    rng = np.random.Generator(np.random.PCG64(4))
    n, H, D, V = 500, 1, 40, 48
    m = Memory(kb, ctx, torch_cuda, H, D, V, 15.0)
    for at in (0, 3, 63, 64, 65, 127, 200):
        for shut in (None, 420):
            i, f = np.full((n, H), -30.0), np.full((n, H), 40.0)
            i[at] = 30.0
            if shut:
                f[shut:shut + 4] = -60.0
            q, k, v, g, zi, zf = m.inputs(rng, n, i, f)
            q = np.tile(k[at], (n, 1, 1)) * 4
            a = (to_bf16(q), k, v, g, zi, zf)
            got, pos = [], 0
            for c in (70, 230, 199, 1) if path == 2 else (300, 199, 1):
                got.append(m.run(*(x[pos:pos + c] for x in a), 2, pos, path if c > 1 else 1))
                pos += c
            got = np.concatenate(got)[:, 0]
            ref = m.reference(*a)[:, 0]
            near = lambda t: np.abs(got[t] - v[at, 0]).max() < 2e-2 * np.abs(v[at, 0]).max()
            seen = [at, at + 1, 300, 410] + ([] if shut else [450, n - 2, n - 1])
            assert all(near(t) for t in seen), (at, shut)
            assert not any(near(t) for t in ([at - 1] if at else []) + ([430, n - 1] if shut else []))
            # after the memory is gone the read-outs are made of what is left: tiny inputs
            live = np.arange(n) if shut is None else np.arange(shut)
            size = np.sqrt(np.mean(ref[live] ** 2, axis=1)) + 1e-3
            assert (np.abs(got[live] - ref[live]).max(axis=1) / size).max() < 5e-3
    m.pool.destroy()


def test_memory_first_token_and_the_denominators_floor(kb, ctx, torch_cuda):
    """The first token starts from a maximum of 0, not of minus infinity: a weak input leaves the
    read-out small instead of normalised."""
    m = Memory(kb, ctx, torch_cuda, 2, 16, 24, 10.0)
    rng = np.random.Generator(np.random.PCG64(8))
    a = m.inputs(rng, 20, np.full((20, 2), -4.0), np.full((20, 2), -1.0))
    ref = m.reference(*a)
    assert np.abs(ref[0]).max() < 0.5 * np.abs(a[2][0]).max()  # far below the value itself
    for path in (1, 2):
        assert rel_err(m.run(*a, 0, 0, path), ref) <= (1e-5 if path == 1 else 2e-4)
    one = tuple(x[:1] for x in a)
    assert rel_err(m.run(*one, 0, 0, 1), ref[:1]) <= 1e-5
    m.pool.destroy()


def test_head_norm_and_gate(ctx, torch_cuda):
    torch = torch_cuda
    rng = np.random.Generator(np.random.PCG64(10))
    T, H, D, V, eps = 5, 3, 4, 37, 0.2
    o, w = f32(rng.standard_normal((T, H, V)) * [[[0.1], [1], [5]]]), f32(rng.standard_normal(H * V))
    y = f32(rng.standard_normal((T, H * (2 * D + 2 * V + 2))) * 3)
    out = guarded(torch, T, H * V)
    od, yd, wd = (dev(torch, x) for x in (o, y, w))
    ctx.call("kanso_cuda_head_norm_gate", od.data_ptr(), yd.data_ptr(), wd.data_ptr(), eps,
             out.data_ptr(), T, H, D, V)
    gate = y[:, H * (2 * D + V):H * (2 * D + 2 * V)]
    assert rel_err(unguard(ctx, out), plain.head_norm_gate(f64(o), f64(gate), f64(w), eps)) <= 2e-6


# ----------------------------------------------------------------------- whole models ----
class MiguraxCase(Case):
    models, weights, plain_class = MODELS, staticmethod(weights), plain


@pytest.mark.parametrize("overlap", [1, 0])
@pytest.mark.parametrize("name", sorted(MODELS))
def test_prompt_portions_and_decoding(kb, torch_cuda, tmp_path, name, compute, overlap):
    ctx = kb.Context(0, torch_cuda.cuda.current_stream())
    ctx.set_option(kb.OPT_OVERLAP_WEIGHT_PREFETCH, overlap)
    c = MiguraxCase(kb, ctx, tmp_path, name, compute)
    n = 150
    tokens = c.tokens(n)
    ref = c.plain(tokens)
    e = kb.Engine(c.model, 4 * n, 4)
    free = e.free_blocks
    schedules = [[n], [1] * n] if not overlap else [
        [n], [1] * n, [2] * 75, [3] * 50, [7, 1, 1, 9, 8, 2] * 20, [16] * 10, [17] * 10, [64] * 3,
        [63, 2, 65, 1, 1, 100], [n - 40] + [1] * 40, [1, 2, 3, 5, 8, 13, 21, 34, 55, 89]]
    for i, cuts in enumerate(schedules):
        got = c.run(e, i, tokens, cuts)
        assert c.close(got, ref), cuts[:6]
        assert e.free_blocks == free
    e.destroy()
    c.done()
    ctx.close()


@pytest.mark.parametrize("name", ["memory", "mixed", "wide"])
def test_mixed_batches_against_each_alone(kb, ctx, torch_cuda, tmp_path, name, compute):
    """Steps of decoding requests, short and long portions together; the results in the order that
    was asked for."""
    c = MiguraxCase(kb, ctx, tmp_path, name, compute, seed=2)
    lens = [70, 3, 133, 1, 40, 18, 25, 61, 9, 12, 30]
    reqs = [c.tokens(n) for n in lens]
    refs = [c.plain(t) for t in reqs]
    e = kb.Engine(c.model, 2048, len(reqs))
    free = e.free_blocks
    at, got = [0] * len(reqs), [[] for _ in reqs]
    rng = np.random.Generator(np.random.PCG64(4))
    while any(a < n for a, n in zip(at, lens)):
        entries = []
        for i in rng.permutation(len(reqs)):
            k = min(int(rng.choice([1, 1, 1, 2, 3, 20, 66])), lens[i] - at[i])
            if k and rng.random() < 0.7:
                entries.append((int(i), reqs[i][at[i]:at[i] + k], list(range(k))[::-1]))
        if not entries:
            continue
        r = np.frombuffer(e.step(entries, c.V), np.float32).reshape(-1, c.V)
        row = 0
        for i, part, w in entries:
            got[i].append(r[row:row + len(w)][::-1].copy())
            row += len(w)
            at[i] += len(part)
            if at[i] == lens[i]:
                e.end(i)
    for g, ref in zip(got, refs):
        assert c.close(np.concatenate(g), ref)
    assert e.free_blocks == free
    e.destroy()
    c.done()


@pytest.mark.parametrize("name", ["mixed", "memory"])
def test_pages_and_slots_are_used_again(kb, ctx, torch_cuda, tmp_path, name, compute):
    """Few pages and two slots: requests one after the other, and two at a time, in the pages and
    the states of those before them."""
    c = MiguraxCase(kb, ctx, tmp_path, name, compute, seed=3)
    e = kb.Engine(c.model, 200, 2)
    for n in (100, 33, 180, 1, 64, 2):
        t = c.tokens(n)
        assert c.close(c.run(e, 5, t, [n // 2 + 1] + [1] * n), c.plain(t))
    a, b = c.tokens(60), c.tokens(35)
    ra, rb = c.plain(a), c.plain(b)
    e.step([(1, a[:20], []), (2, b[:30], [])], c.V)
    e.end(1)
    got = [e.step([(2, b[30:31], [0]), (3, a[:41], [])], c.V)]
    with pytest.raises(kb.KansoError) as ex:  # no slot is left
        e.step([(4, b[:2], [])], c.V)
    assert ex.value.code == kb.ERR_SHAPE
    got += [e.step([(3, a[41:42], [0]), (2, b[31:32], [0])], c.V)]
    got = np.concatenate([np.frombuffer(g, np.float32).reshape(-1, c.V) for g in got])
    margin = None if compute == F32 else np.array([rb.margin[30], ra.margin[41], rb.margin[31]])
    assert c.close(got, np.stack([rb[30], ra[41], rb[31]]), margin)
    e.end(2)
    e.end(3)
    # too much at once is an error and leaves the engine usable
    with pytest.raises(kb.KansoError) as ex:
        e.step([(7, c.tokens(400), [])], c.V)
    assert ex.value.code == kb.ERR_SHAPE
    e.end(7)
    t = c.tokens(50)
    assert c.close(c.run(e, 8, t, [50]), c.plain(t))
    e.destroy()
    c.done()


def test_long_decoding(kb, ctx, torch_cuda, tmp_path, compute):
    c = MiguraxCase(kb, ctx, tmp_path, "mixed", compute, seed=4)
    t = c.tokens(600)
    e = kb.Engine(c.model, 600, 1)
    assert c.close(c.run(e, 0, t, [40] + [1] * 560), c.plain(t))
    e.destroy()
    c.done()


def test_arguments_and_tensors_are_checked(kb, ctx, torch_cuda, tmp_path):
    c = MiguraxCase(kb, ctx, tmp_path, "uneven", BF16)
    a = lambda *x: np.array(x, np.uint32)
    out = np.empty((2, c.V), np.float32)
    pool = c.model.create_pool(8, 3)
    for slots in (a(0, 0), a(1, 3)):  # one slot twice; a slot that the pool does not have
        with pytest.raises(kb.KansoError) as ex:
            c.model.forward_step(pool, a(1, 2), a(1, 1), a(1, 1), a(0, 1), 1, a(0, 1), out, slots)
        assert ex.value.code == kb.ERR_SHAPE and "slot" in ex.value.message
    with pytest.raises(kb.KansoError):  # a pool of another geometry
        c.model.forward_step(kb.KvPool.of_layers(ctx, np.array([[1, 8, 8, 0, 0, 0]] * 2, np.uint32),
                                                 8, 16, kb.KV_BF16), a(1), a(1), a(1), a(0), 1, a(0),
                             out)
    with pytest.raises(kb.KansoError) as ex:  # a state needs slots
        c.model.create_pool(8, 0)
    assert ex.value.code == kb.ERR_CONFIG
    assert pool.state_bytes == 4 * 5 * (6 * 32 + 8 + 4) and pool.bytes_per_token == 2 * 16
    pool.destroy()
    for change in (lambda w: w.pop("l0.mix.sink"), lambda w: w.update({"l0.mix.uk": w["l0.mix.uv"]}),
                   lambda w: w.pop("l1.mix.f.b"), lambda w: w.pop("l1.mlp.router.b")):
        w = dict(c.w)
        change(w)
        with pytest.raises(kb.KansoError):
            kb.Model.from_dir(ctx, write_model(tmp_path / "bad", c.cfg, w), BF16)
    c.done()


@pytest.mark.parametrize("B", [2, 5])
def test_decode_step_and_forward_step_agree(kb, ctx, torch_cuda, tmp_path, compute, B):
    """The pool-level calls: a ragged step fills pages and slots, then the decode step of the other
    models' hosts gives what the plain model gives, also replayed from a captured graph (from the
    same state) and with the slots given."""
    torch = torch_cuda
    c = MiguraxCase(kb, ctx, tmp_path, "wide", compute, seed=6)
    bs, lens = 16, [40, 17, 33, 2, 64][:B]
    reqs = [c.tokens(n) for n in lens]
    refs = [c.plain(t) for t in reqs]
    perm = c.rng.permutation(16)
    maxb = 4
    tables = np.zeros((B, maxb), np.uint32)
    used = 0
    for i, n in enumerate(lens):
        nb = (n + bs - 1) // bs
        tables[i, :nb] = perm[used:used + nb]
        used += nb
    a = lambda x: np.array(x, np.uint32)
    heads = [t[:-1] for t in reqs]
    ends = np.cumsum([len(h) for h in heads]) - 1
    margin = lambda i: None if compute == F32 else np.array([r.margin[i] for r in refs])
    want, logits = np.stack([r[-1] for r in refs]), np.empty((B, c.V), np.float32)
    pos = a([n - 1 for n in lens])
    slots = a([tables[i, p // bs] * bs + p % bs for i, p in enumerate(pos)])
    last = a([t[-1] for t in reqs])
    for state_slots in (None, a([6, 0, 3, 2, 5][:B])):
        pool = c.model.create_pool(16, 7)

        def prompt():
            c.model.forward_step(pool, a(sum(heads, [])), a([len(h) for h in heads]),
                                 a([len(h) for h in heads]), tables, maxb, a(ends), logits,
                                 state_slots)
        prompt()
        assert c.close(logits, np.stack([r[-2] for r in refs]), margin(-2))
        if state_slots is None:
            c.model.decode_step(pool, last, pos, slots, tables, a(lens), maxb, logits)
            assert c.close(logits, want, margin(-1))
        d = [u32(torch, x) for x in (last, pos, slots, tables, a(lens))]
        ds = None if state_slots is None else u32(torch, state_slots)
        out = torch.zeros((B, c.V), device="cuda")
        step = lambda: c.model.decode_step_device(pool, *d, B, maxb, max(lens), out, state_slots=ds)
        prompt()
        step()
        ctx.sync()
        assert c.close(out.cpu().numpy(), want, margin(-1))
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, stream=torch.cuda.current_stream()):
            step()
        for _ in range(2):
            prompt()
            out.zero_()
            g.replay()
            ctx.sync()
            assert c.close(out.cpu().numpy(), want, margin(-1))
        del g
        pool.destroy()
    c.done()


@pytest.mark.parametrize("name", ["mixed", "memory"])
def test_greedy_generation(kb, ctx, torch_cuda, tmp_path, name):
    """Continuous batching over more prompts than may run at a time, prompts cut by the step's
    token budget; every request's tokens are those of the plain model."""
    c = MiguraxCase(kb, ctx, tmp_path, name, F32, seed=7)
    new, prompts, refs = 10, [], []
    for n in (5, 61, 1, 30, 90, 2, 17):
        while True:  # a prompt whose continuation has no close call
            t, margin = c.tokens(n), 1.0
            for _ in range(new):
                row = c.plain(t)[-1]
                margin = min(margin, np.diff(np.sort(row)[-2:])[0])
                t.append(int(np.argmax(row)))
            if margin > 1e-3:
                break
        prompts.append(t[:n])
        refs.append(t[n:])
    for max_tokens, max_seqs, budget in ((2000, 16, 0), (160, 3, 24), (2000, 2, 7)):
        e = kb.Engine(c.model, max_tokens, max_seqs)
        free = e.free_blocks
        assert e.generate(prompts, new, budget) == refs
        assert e.free_blocks == free
        e.destroy()
    c.done()


def test_trace_replay_command(kb, ctx, torch_cuda, tmp_path, compute):
    c = MiguraxCase(kb, ctx, tmp_path / "m", "uneven", compute, seed=9)
    a, b = c.tokens(50), c.tokens(20)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[30:49], "want": [18]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[49:], "want": [0]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b[:2], "want": [1]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", c.folder, "--dtype",
                        "float32" if compute == F32 else "bfloat16", "--out", str(out),
                        "--max-tokens", "70"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=600,
                       env={**os.environ, "PYTHONPATH": os.pathsep.join(sys.path)})
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l] == [f"done {i}" for i in range(5)]
    read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, c.V)
    ra, rb = c.plain(a), c.plain(b)
    margin = None if compute == F32 else np.append(ra.margin[[0, 29, 48, 49]], rb.margin[1])
    assert c.close(np.concatenate([read(0), read(2), read(3), read(4)]),
                   np.concatenate([ra[[0, 29, 48, 49]], rb[[1]]]), margin)
    c.done()
