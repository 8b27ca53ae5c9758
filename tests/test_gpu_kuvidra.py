"""The Kuvidra design in the engine against its plain implementation (``plain_kuvidra``): each mechanism alone, then whole
models under every way of cutting the work, in float32 and bfloat16.

The configurations are small and differ from one another in every size and constant: a repeated stretch of layers of one,
two and three passes (and none), latents that the tensor-core kernel takes as they are and filled up and latents it refuses,
matrix memories whose sizes the chunked and the single-token kernels take and refuse, gate caps of 4 to 25, routers that
choose one, several and all experts, with and without a shared expert, layers without a feed-forward.  Where random
weights would hide a fault the inputs are made so that it shows: queries are scaled until single far keys stand out, a
memory's head never forgets, another forgets everything between two tokens, input gates stay so low that the running
maximum's start at 0 decides the denominator.
"""
import json
import os
import random

import numpy as np
import pytest
import torch

import helpers as H
import plain_kuvidra as pk
from test_gpu_mumazen import _bound_part, check, cuts, f64, i32, load_plain, make_ctx, step_meta

pytestmark = pytest.mark.gpu


def _lat(heads, dim, vdim, kv_rank, q_rank, scale):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}}


def _mem(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _dense(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def _moe(layer, experts, top, ff, shared):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return dict(layer, mlp=mlp)


def _none(layer):
    return dict(layer, mlp=None)


CONFIGS = {
    # two passes over layers 1..2; a latent of 80 (filled up to 128); three of seven experts
    "A": {"architecture": "Kuvidra", "vocab": 301, "width": 96, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2}, "layers": [
        _dense(_mem(3, 16, 32, 10.0), 120), _moe(_lat(6, 24, 16, 80, 56, 0.3), 7, 3, 40, 48),
        _none(_mem(2, 48, 16, 4.0)), _moe(_lat(6, 24, 16, 80, 56, 0.3), 4, 2, 24, 0)]},
    # no loop; sizes that no tensor-core, vector or single-token kernel takes: width 90, latent 30, values of 10 and 7
    "B": {"architecture": "Kuvidra", "vocab": 203, "width": 90, "norm": {"eps": 3e-6}, "layers": [
        _moe(_lat(3, 11, 10, 30, 21, 0.25), 3, 3, 20, 27), _dense(_mem(2, 13, 7, 25.0), 50), _none(_lat(1, 40, 30, 12, 9, 0.2))]},
    # sizes of the tensor-core kernels; three passes over everything; one expert of sixteen
    "C": {"architecture": "Kuvidra", "vocab": 512, "width": 128, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 3}, "layers": [
        _moe(_mem(4, 64, 128, 15.0), 16, 1, 64, 96), _dense(_lat(8, 64, 64, 128, 96, 0.125), 256)]},
    # matrix memories only (no paged cache group); a loop of one pass; a state of 160 rows and one of 20 columns
    "D": {"architecture": "Kuvidra", "vocab": 130, "width": 64, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 2, "times": 1}, "layers": [
        _dense(_mem(1, 160, 48, 8.0), 72), _moe(_mem(5, 8, 20, 12.0), 5, 5, 16, 8), _none(_mem(2, 32, 208, 6.0))]},
    # attention only, the latent wider than the model; a loop of two passes over the last layer
    "E": {"architecture": "Kuvidra", "vocab": 222, "width": 72, "norm": {"eps": 1e-6}, "loop": {"start": 1, "stop": 2, "times": 2}, "layers": [
        _dense(_lat(5, 16, 40, 200, 64, 0.25), 88), _moe(_lat(2, 32, 8, 64, 40, 0.18), 6, 4, 32, 40)]},
}
PAGE = {"A": 16, "B": 8, "C": 16, "D": 16, "E": 32}
LENGTHS = {"A": [1, 9, 50, 150], "B": [2, 20, 77], "C": [5, 70, 200], "D": [3, 40, 140], "E": [2, 33, 130]}
SHARP = {"A": 3.0, "B": 4.0, "C": 2.5, "D": 1.0, "E": 3.0}          # queries times this: single keys, near and far, stand out
FP32_TOL, BF16_TOL = 1e-4, 5e-2
DTYPES = [("float32", FP32_TOL), ("bfloat16", BF16_TOL)]


def tokens(which, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, CONFIGS[which]["vocab"], n)]


CLASSES = 16         # leading channels of a well-conditioned model's stream: the token's class; behind them one constant channel


def _well_conditioned(cfg, tensors):
    """A model in which bfloat16 rounding stays rounding.  The first channels of the stream hold the token's class and a
    constant and nothing else (no branch writes them, a pass's product hands them on).  A router's scores are a well-spaced table
    over the classes plus a small random part, so no choice is close.  A memory's q and k share a direction that the constant
    feeds, so n . q stays away from zero, where o would change its sign."""
    W, C = cfg["width"], CLASSES + 1
    for name, t in tensors.items():
        t = t.float()
        if name == "embed":
            t[:, :C] = 0.0
            t[torch.arange(t.shape[0]), torch.arange(t.shape[0]) % CLASSES] = 3.0
            t[:, CLASSES] = 3.0
        elif name == "loop.in":
            t[:C] = 0.0
            t[torch.arange(C), W + torch.arange(C)] = 1.0
        elif name == "loop.step":
            t[:, :C] = 0.0
        elif name.endswith("mix.o") or name.endswith("down"):
            t[:C] = 0.0
        elif name.endswith("mix.q") or name.endswith("mix.k"):
            t[:, CLASSES] = 0.6 * (1.0 - 2.0 * (torch.arange(t.shape[0]) % 3 % 2))
        elif name.endswith("router"):
            E = t.shape[0]
            t *= 0.1
            t[:, :CLASSES] = (torch.arange(E)[:, None] + torch.arange(CLASSES)[None, :]) % E * (2.0 / E) - 1.0
        tensors[name] = t.to(torch.bfloat16)


def write_model(folder, cfg, seed, sharp=1.0, conditioned=True):
    """A random model folder with the attention's queries scaled; ``conditioned``: see above."""
    from aien_sovereign_core_mv_b200 import model_spec_for
    from aien_sovereign_core_mv_b200.models.decoder import Decoder
    from aien_sovereign_core_mv_b200.weights.random_init import random_tensor
    from aien_sovereign_core_mv_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    cat = Decoder(model_spec_for(cfg)[1]).catalog()
    out = {}
    for name, (shape, kind) in cat.items():
        t = random_tensor(name, tuple(shape), kind, seed)
        out[name] = (t.float() * sharp).to(torch.bfloat16) if name.endswith("mix.uq") else t
    if conditioned:
        _well_conditioned(cfg, out)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), out)
    return folder


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("kuvidra")
    out = {}
    for i, which in enumerate(CONFIGS):
        d = write_model(os.path.join(str(root), which), CONFIGS[which], 40 + i, SHARP[which])
        cfg, tensors = load_plain(d)
        reqs = {j + 1: tokens(which, n, 100 * i + n) for j, n in enumerate(LENGTHS[which])}
        want = {rid: pk.forward(cfg, tensors, toks) for rid, toks in reqs.items()}
        out[which] = (d, reqs, want)
    return out


# ------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 90, 256, 1000, 2052, 9000])
def test_pending_terms_and_norm(dtype, width):
    """Up to three terms (whole, in parts, times a gate per token), a vector for every token, added to the stream or in its place."""
    from aien_sovereign_core_mv_b200 import kernels as K
    g = torch.Generator().manual_seed(width)
    T, eps = 7, 1e-5
    x0 = torch.randn(T, width, generator=g)
    a, parts = torch.randn(T, width, generator=g), torch.randn(3, T, width, generator=g)
    low = torch.randn(2, T, width, generator=g).to(torch.bfloat16)
    z, bias = torch.randn(T, 5, generator=g) * 2.0, torch.randn(width, generator=g).to(torch.bfloat16)
    w = (torch.rand(width, generator=g) + 0.5).to(dtype)
    sg = pk.sigmoid(f64(z[:, 3]))[:, None]
    zc = z.cuda()
    cases = [((), None, False, f64(x0)), (((a, None),), None, False, f64(x0) + f64(a)),
             (((parts, None), (low, None), (a, 3)), bias, False, f64(x0) + f64(parts).sum(0) + f64(low).sum(0) + sg * f64(a) + f64(bias)),
             (((parts, None),), bias, True, f64(parts).sum(0) + f64(bias)), (((low[0].contiguous(), 3), (a, None)), None, True, sg * f64(low[0]) + f64(a))]
    for terms, b, replace, want in cases:
        x = x0.clone().cuda()
        if replace:
            x.fill_(float("nan"))                                    # what was there must not be read
        h = torch.zeros(T, width, dtype=dtype).cuda()
        dev = tuple((t.cuda(), None if c is None else zc[:, c]) for t, c in terms)
        K.sum_terms_rmsnorm(x, dev, None if b is None else b.cuda(), replace, w.cuda(), eps, h)
        H.assert_close(x.cpu().numpy(), want, 2e-6, "the stream after the sum")
        H.assert_close(h.float().cpu().numpy(), pk.rms(want, eps) * f64(w), 2e-6 if dtype == torch.float32 else 6e-3, "the norm")
        if not replace:
            y = x0.clone().cuda()
            K.sum_terms_rmsnorm(y, dev, None if b is None else b.cuda(), False, None, 0.0, None)
            H.assert_close(y.cpu().numpy(), want, 2e-6, "the sum alone")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,width", [(1, 64), (5, 90), (40, 128)])
def test_pass_input_projects_the_stream_and_the_embedding(dtype, T, width):
    """In bfloat16 the stream must enter the product with more than 8 bits: the bound is far below what one rounding gives."""
    from aien_sovereign_core_mv_b200.parts.base import SumTerms, add_to_residual
    part, W = _bound_part("pass_input", "step_projection", 11, dtype, hidden_size=width, times=3)
    g = torch.Generator().manual_seed(T)
    x0 = torch.randn(T, width, generator=g) * 10.0
    e = torch.randn(T, width, generator=g).to(torch.bfloat16).float()
    d = torch.randn(T, width, generator=g)
    names = {"loop.in": W["in_proj"], "loop.step": W["steps"]}
    for t, pending in ((0, None), (2, SumTerms(((d.cuda(), None),)))):
        ctx = make_ctx(dtype, list(range(T)), [0] * T, [0, T], [T])
        x = x0.clone().cuda()
        out = part.forward(ctx, x, e.cuda(), t, pending)
        add_to_residual(ctx, x, out)
        want = pk.pass_input(names, f64(x0) + (f64(d) if pending is not None else 0.0), f64(e), t)
        H.assert_close(x.cpu().numpy(), want, 3e-6 if dtype == torch.float32 else 3e-5, f"pass {t}")


def _memory_inputs(heads, D, V, cap, lens, seed):
    g = torch.Generator().manual_seed(seed)
    off = 8
    rows = [(torch.randn(n, off + 2 * heads * D + 2 * heads * V, generator=g)).to(torch.bfloat16).float() for n in lens]
    z = [torch.randn(n, 2 * heads + 3, generator=g) * 2.0 for n in lens]
    bi, bf = torch.randn(heads, generator=g) * 0.3, torch.rand(heads, generator=g) * 3.0 + 2.0
    for a in rows:
        a[:, off:off + D].abs_()                                     # head 0: q . k never near zero, where one bit of S would turn o
        a[:, off + heads * D:off + heads * D + D].abs_()
    bf[0] = 60.0                                                     # head 0 keeps (almost) everything: a cap away from the first token
    for s, n in enumerate(lens):
        z[s][:, 0] = -60.0                                           # ... and takes little, so that its maximum stays near its start at 0
        z[s][0, 0] = 60.0 if s == 0 else -60.0                       # except request 0's first token, which must show to the end
        z[s][n // 2, heads + heads - 1] = -60.0                      # the last head forgets everything in the middle
    return off, rows, z, bi, bf


def _memory_want(off, rows, z, bi, bf, heads, D, V, cap, w, eps):
    n = rows.shape[0]
    q = f64(rows[:, off:off + heads * D]).reshape(n, heads, D) * D ** -0.5
    k = f64(rows[:, off + heads * D:off + 2 * heads * D]).reshape(n, heads, D)
    v0 = off + 2 * heads * D
    v = f64(rows[:, v0:v0 + heads * V]).reshape(n, heads, V)
    gate = f64(rows[:, v0 + heads * V:])
    i, f = pk.mlstm_gates(f64(z[:, :heads]) + f64(bi), f64(z[:, heads:2 * heads]) + f64(bf), cap)
    o, state = pk.mlstm_recurrence(q, k, v, i, f)
    return pk.rms(o, eps).reshape(n, heads * V) * f64(w) * pk.sigmoid(gate), state


@pytest.mark.parametrize("form", ["walk", "token", "chunks"])
@pytest.mark.parametrize("heads,D,V,cap", [(4, 16, 16, 15.0), (3, 48, 80, 6.0), (2, 64, 128, 15.0), (2, 128, 64, 30.0), (1, 256, 256, 9.0), (3, 20, 12, 15.0), (2, 7, 9, 12.0), (1, 300, 8, 15.0)])
def test_matrix_memory_cut_any_way(form, heads, D, V, cap):
    """Whole, in portions down to one token, beside one another: the same rows and states as token by token in float64.
    A used slot must not leak into a new request, and slots of others stay as they are."""
    from aien_sovereign_core_mv_b200 import kernels as K
    bf16 = form == "chunks"
    if bf16 and not K.matrix_memory_chunks_supports(torch.bfloat16, D, V):
        assert D % 16 or V % 16
        return
    if form == "token" and not K.matrix_memory_token_supports(D, V):
        assert V % 4
        return
    lens = [200, 70] if D * V <= 8192 else [140, 66]
    eps, den = 1e-5, pk.DENOMINATOR_EPS
    off, rows, z, bi, bf = _memory_inputs(heads, D, V, cap, lens, heads * 100 + D)
    g = torch.Generator().manual_seed(D + V)
    w = torch.rand(heads * V, generator=g) + 0.5
    want = [_memory_want(off, rows[s], z[s], bi, bf, heads, D, V, cap, w, eps) for s in (0, 1)]
    k0, v0 = off + heads * D, off + 2 * heads * D
    g0 = v0 + heads * V
    floats = K.matrix_memory_state_floats(heads, D, V)
    for sizes in ([[1]] if form == "token" else [[300], [64, 1], [2, 1, 63, 7, 33, 65], [128, 3]]):
        state = torch.full((4, floats), 7.0).cuda()
        got = [[], []]
        for step in cuts(lens, sizes):
            pos, sot, q_start = step_meta(step)
            cat = lambda src: torch.cat([src[s][p0:p0 + n] for s, p0, n in step]).cuda()
            T, S = len(pos), len(step)
            proj, zz = cat(rows), cat(z)
            meta = (state, i32([2 - s for s, _, _ in step]), i32(q_start), i32(pos))
            out = torch.zeros(T, heads * V, dtype=torch.bfloat16 if bf16 else torch.float32).cuda()
            if form == "token":
                K.matrix_memory_token(proj, off, k0, v0, g0, D ** -0.5, zz, 0, heads, bi.cuda(), bf.cuda(), cap, *meta, w.cuda(), eps, den, out, S, heads, D, V)
            else:
                gates = torch.zeros(T, 3 * heads).cuda()
                K.matrix_memory_gates(zz, 0, heads, bi.cuda(), bf.cuda(), cap, *meta, gates, S, heads, D, V)
                if bf16:
                    scratch = torch.full((K.matrix_memory_chunks_scratch(T, S, heads, D, V),), float("nan")).cuda()
                    K.matrix_memory_chunked(proj.to(torch.bfloat16), off, k0, v0, g0, D ** -0.5, gates, *meta, w.cuda(), eps, den, out, scratch, S, heads, D, V)
                else:
                    num, nq = torch.zeros(T, heads * V).cuda(), torch.zeros(T, heads).cuda()
                    K.matrix_memory_walk(proj, off, k0, v0, D ** -0.5, gates, *meta, num, nq, S, heads, D, V)
                    K.matrix_memory_finish(num, nq, gates, proj[:, g0:], w.cuda(), eps, den, out, heads, V)
            for i, (s, _, n) in enumerate(step):
                got[s].append(out[q_start[i]:q_start[i] + n].float().cpu().numpy())
        for s in (0, 1):
            H.assert_close(np.concatenate(got[s]), want[s][0], 1e-2 if bf16 else 1e-4, f"{form} {sizes}, request {s}")
            flat = state[2 - s].double().cpu().numpy()
            DV = heads * D * V
            m = flat[DV + heads * D:DV + heads * D + heads]
            H.assert_close(m, want[s][1][2], 1e-5, f"{form} {sizes}: m of request {s}")
            # S and n are relative to e^m, whatever m was rounded to; float32 in every form
            rel = np.exp(m - want[s][1][2])
            H.assert_close(flat[:DV] * np.repeat(rel, D * V), want[s][1][0].reshape(-1), 1e-5, f"{form} {sizes}: S of request {s}")
            H.assert_close(flat[DV:DV + heads * D] * np.repeat(rel, D), want[s][1][1].reshape(-1), 1e-5, f"{form} {sizes}: n of request {s}")
        assert float((state[0] - 7.0).abs().max()) == 0.0 and float((state[3] - 7.0).abs().max()) == 0.0


def test_the_running_maximum_starts_at_zero():
    """With input gates far below zero the denominator is e^0 = 1, not what a maximum that starts at the first gate gives:
    the rows before the norm then differ by a factor that the norm's eps makes visible."""
    from aien_sovereign_core_mv_b200 import kernels as K
    heads, D, V, cap = 1, 16, 16, 20.0
    rows = torch.randn(5, 2 * D + 2 * V, generator=torch.Generator().manual_seed(1))
    z = torch.full((5, 2), -9.0)
    z[:, 1] = 30.0
    state = torch.zeros(2, K.matrix_memory_state_floats(1, D, V)).cuda()
    gates, num, nq = torch.zeros(5, 3).cuda(), torch.zeros(5, V).cuda(), torch.zeros(5, 1).cuda()
    zero, w, eps = torch.zeros(1), torch.ones(V), 1e-6
    meta = (state, i32([0]), i32([0, 5]), i32(list(range(5))))
    K.matrix_memory_gates(z.cuda(), 0, 1, zero.cuda(), zero.cuda(), cap, *meta, gates, 1, 1, D, V)
    K.matrix_memory_walk(rows.cuda(), 0, D, 2 * D, D ** -0.5, gates, *meta, num, nq, 1, 1, D, V)
    out = torch.zeros(5, V).cuda()
    K.matrix_memory_finish(num, nq, gates, rows.cuda()[:, 2 * D + V:], w.cuda(), eps, pk.DENOMINATOR_EPS, out, 1, V)
    want, (_, _, m) = _memory_want(0, rows, z, zero, zero, 1, D, V, cap, w, eps)
    assert abs(m[0]) < 1e-3 and abs(float(gates[4, 2]) - m[0]) < 1e-6
    H.assert_close(out.cpu().numpy(), want, 1e-5, "rows")


@pytest.mark.parametrize("heads,r,rd,page,window", [(4, 96, 0, 16, 0), (3, 24, 8, 8, 0), (6, 40, 0, 16, 33), (2, 200, 16, 8, 0), (16, 320, 0, 16, 64), (5, 72, 24, 32, 0), (3, 128, 0, 16, 0)])
def test_latent_attention_of_any_latent_size(heads, r, rd, page, window):
    """The tensor-core kernel (latents filled up to its sizes; tiles of 64 and of 16 rows; keys dealt out to CTAs) and the
    plain one against float64.  The rows at position 0, at a page's and a block's border and just inside and outside the window
    are scaled so that single scores stand out; slots nobody needs hold NaN."""
    from aien_sovereign_core_mv_b200 import kernels as K
    assert K.latent_attention_tc_supports(torch.bfloat16, r, rd)
    g = torch.Generator().manual_seed(r + rd)
    D, n = r + rd, 150
    tab = torch.randperm(24, generator=g)[: (n + page - 1) // page].tolist()
    kv = torch.randn(n, D, generator=g) * 0.6
    for j in (0, page - 1, page, 63, 64, 127):
        kv[j] *= 4.0
    kv = kv.to(torch.bfloat16)
    cache = torch.full((24 * page, D), float("nan"), dtype=torch.bfloat16)
    for p in range(n):
        cache[tab[p // page] * page + p % page] = kv[p]
    bt = i32([tab])
    for q0, T in ((0, n), (n - 1, 1), (60, 37)):
        q = torch.randn(T, heads, D, generator=g).to(torch.bfloat16)
        pos = list(range(q0, q0 + T))
        scale = 2.0 * D ** -0.5
        see = lambda t: [j for j in range(pos[t] + 1) if window == 0 or pos[t] - j < window]
        want = np.zeros((T, heads, r))
        for t in range(T):
            js = see(t)
            for h in range(heads):
                s = f64(kv)[js] @ f64(q)[t, h] * scale
                p = np.exp(s - s.max())
                want[t, h] = (p / p.sum()) @ f64(kv)[js, :r]
        for small in ((False, True) if T == 1 and r > 64 else (False,)):
            for ksplit in (1, 3):
                out = torch.full((T, heads * r), float("nan"), dtype=torch.bfloat16).cuda()
                scratch = torch.full((max(1, K.latent_attention_tc_scratch(T, heads, r, ksplit)),), float("nan")).cuda()
                K.latent_attention_tc(q.view(T, -1).cuda(), cache.cuda(), bt, len(tab), i32([0, T]), i32(pos), out, 1, heads, r, rd, page, window, scale,
                                      None, ksplit, scratch if ksplit > 1 else None, small)
                H.assert_close(out.float().cpu().numpy().reshape(T, heads, r), want, 1.5e-2, f"tensor cores, {T} tokens, split {ksplit}, small {small}")
        out = torch.full((T, heads * r), float("nan"), dtype=torch.float32).cuda()
        K.latent_attention(q.view(T, -1).float().cuda(), cache.cuda(), bt, len(tab), i32([0] * T), i32(pos), out, heads, r, rd, page, window, scale, None)
        H.assert_close(out.cpu().numpy().reshape(T, heads, r), want, 1e-5, f"plain, {T} tokens")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,n,k", [(3, 10, 12), (5, 40, 96), (2, 130, 64)])
def test_products_per_head_with_a_gate(dtype, heads, n, k):
    from aien_sovereign_core_mv_b200 import kernels as K
    g = torch.Generator().manual_seed(n)
    T = 70
    a = torch.randn(T, heads * k, generator=g).to(dtype)
    w = (torch.randn(heads, n, k, generator=g) * k ** -0.5).to(dtype)
    z = torch.randn(T, heads + 4, generator=g) * 2.0
    out = torch.zeros(T, heads * n, dtype=dtype).cuda()
    K.head_project(a.cuda(), k, 0, w.cuda(), out, n, 0, gate=z.cuda()[:, 3:3 + heads])
    want = np.einsum("thk,hnk->thn", f64(a).reshape(T, heads, k), f64(w)) * pk.sigmoid(f64(z[:, 3:3 + heads]))[:, :, None]
    H.assert_close(out.float().cpu().numpy().reshape(T, heads, n), want, 1e-5 if dtype == torch.float32 else 8e-3, "gated product")


@pytest.mark.parametrize("E,top", [(5, 1), (7, 3), (4, 4), (40, 6)])
def test_router_of_sigmoid_scores(E, top):
    from aien_sovereign_core_mv_b200 import kernels as K
    g = torch.Generator().manual_seed(E)
    T = 60
    z = torch.randn(T, E + 3, generator=g) * 4.0
    z[::3, :E] += 30.0                                               # scores that all round to one: the order is that of z
    ids, wts = torch.zeros(T, top, dtype=torch.int32).cuda(), torch.zeros(T, top).cuda()
    counts = torch.zeros(E, dtype=torch.int32).cuda()
    K.moe_route_biased(z.cuda(), E, E, top, False, 0.0, None, ids, wts, None, counts, sigmoid=True)
    order = np.argsort(-f64(z[:, :E]), axis=-1, kind="stable")[:, :top]
    assert (np.sort(ids.cpu().numpy(), -1) == np.sort(order, -1)).all()
    assert counts.cpu().tolist() == np.bincount(ids.cpu().numpy().ravel(), minlength=E).tolist()
    H.assert_close(wts.cpu().numpy(), pk.sigmoid(np.take_along_axis(f64(z[:, :E]), ids.cpu().numpy().astype(np.int64), -1)), 1e-6, "weights")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,ff,shared", [(5, 3, 64, 72), (3, 1, 20, 0), (6, 6, 8, 40), (9, 2, 136, 24)])
def test_gated_experts_with_the_weight_on_their_input(dtype, E, top, ff, shared):
    """Few tokens (streamed products) and many (grouped products); router rows in the part's own product and handed in."""
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    for T in (1, 5, 150):
        g = torch.Generator().manual_seed(T)
        h = torch.randn(T, 128, generator=g).to(torch.bfloat16)
        ff_part, W = _bound_part("feed_forward", "routed_experts", 6, dtype, hidden_size=128, expert_ff=ff, num_experts=E, top=top, act="swiglu",
                                 score="sigmoid", weight_on_input=True, shared_ff=shared, shared_gate=bool(shared))
        Wt = {"router": W["router"]}
        for e in range(E):
            for m in ("gate", "up", "down"):
                Wt[f"e{e}.{m}"] = W[f"experts.{e}.{m}"]
        if shared:
            Wt.update({"shared.gate": W["shared.gate_proj"], "shared.up": W["shared.up"], "shared.down": W["shared.down"], "shared.sg": W["shared.gate"]})
        want = pk.moe_ff({"router": {"top": top}, "shared": {"ff": shared} if shared else None}, Wt, "", f64(h))
        rows = np.concatenate([W["router"]] + ([W["shared.gate"]] if shared else []), 0)
        z = torch.tensor(f64(h) @ rows.T, dtype=torch.float32)
        for riders in (None, z.cuda()):
            ctx = make_ctx(dtype, list(range(T)), [0] * T, [0, T], [T])
            total = 0.0
            for t, gate in ff_part.terms(ctx, h.to(dtype).cuda(), riders):
                t = t.float().sum(0) if t.dim() == 3 else t.float()
                total = total + f64(t) * (1.0 if gate is None else pk.sigmoid(f64(gate))[:, None])
            H.assert_close(total, want, tol, f"{T} tokens, riders {riders is not None}")


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_whole_prompts(models, which, dtype, tol):
    d, reqs, want = models[which]
    eng = H.engine_for(d, dtype, PAGE[which], 512)
    steps = [([(rid, toks, list(range(len(toks))))], [rid]) for rid, toks in reqs.items()]
    check(H.run_steps(eng, steps), want, tol, f"{which} {dtype} whole")
    assert eng.cache_state()["check"] == "" and eng.cache_state()["requests"] == 0


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_prefill_then_token_by_token(models, which, dtype, tol):
    d, reqs, want = models[which]
    eng = H.engine_for(d, dtype, PAGE[which], 512)
    rid = max(reqs, key=lambda r: len(reqs[r]))
    toks = reqs[rid]
    cut = len(toks) - 45
    steps = [([(rid, toks[:cut], [0, cut - 1])], [])] + [([(rid, [toks[i]], [0])], []) for i in range(cut, len(toks))]
    check(H.run_steps(eng, steps), want, tol, f"{which} {dtype} decode")
    assert eng.cache_state()["check"] == ""


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_first_tokens_one_by_one(models, which, dtype, tol):
    d, reqs, want = models[which]
    eng = H.engine_for(d, dtype, PAGE[which], 512)
    rid = max(reqs, key=lambda r: len(reqs[r]))
    steps = [([(rid, [t], [0])], []) for t in reqs[rid][:40]]
    check(H.run_steps(eng, steps), want, tol, f"{which} {dtype} from the first token")


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_changing_portions(models, which, dtype, tol):
    d, reqs, want = models[which]
    eng = H.engine_for(d, dtype, PAGE[which], 512)
    sizes = [7, 2, 13, 3, 2, 29, 5, 2, 16, 17, 1, 8, 64, 2, 131]
    for rid, toks in reqs.items():
        steps, at, k = [], 0, rid
        while at < len(toks):
            n = min(sizes[k % len(sizes)], len(toks) - at)
            steps.append(([(rid, toks[at:at + n], list(range(n)))], []))
            at += n
            k += 1
        steps[-1] = (steps[-1][0], [rid])
        check(H.run_steps(eng, steps), want, tol, f"{which} {dtype} portions of request {rid}")
    assert eng.cache_state()["check"] == "" and eng.cache_state()["requests"] == 0


def _side_by_side(reqs, rng, live_at_most):
    """Steps of portions beside single tokens, requests admitted as others end; a request may sit a step out."""
    at, waiting, live, steps = {r: 0 for r in reqs}, sorted(reqs, key=lambda r: (len(reqs[r]), r)), [], []
    while waiting or live:
        while waiting and len(live) < live_at_most:
            live.append(waiting.pop(0))
        entries, end = [], []
        for rid in list(live):
            left = len(reqs[rid]) - at[rid]
            n = min(left, 1 if rng.random() < 0.4 else rng.randint(2, 60))
            if rng.random() < 0.15 and len(live) > 1:
                continue
            entries.append((rid, reqs[rid][at[rid]:at[rid] + n], list(range(n))))
            at[rid] += n
            if at[rid] == len(reqs[rid]):
                end.append(rid)
                live.remove(rid)
        if entries:
            steps.append((entries, end))
    return steps


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_mixed_batches_on_few_pages_and_slots(models, which, dtype, tol):
    """Unequal requests side by side with three state slots and a pool so small that pages and slots are used again; every
    logit equals the request's alone."""
    d, reqs, want = models[which]
    page = PAGE[which]
    reqs = dict(reqs)
    reqs.update({rid + 10: toks[: max(1, len(toks) - 3)] for rid, toks in list(reqs.items())})          # more requests than slots
    want = dict(want)
    want.update({rid: want[rid - 10] for rid in reqs if rid > 10})
    longest = max(len(t) for t in reqs.values())
    pool = (3 * ((longest + page - 1) // page + 1) + 2) * page
    eng = H.engine_for(d, dtype, page, pool, max_requests=3)
    check(H.run_steps(eng, _side_by_side(reqs, random.Random(5), 3)), want, tol, f"{which} {dtype} mixed")
    state = eng.cache_state()
    assert state["check"] == "" and state["requests"] == 0


def test_long_decoding_bfloat16_graphs(models):
    """Some 140 decode-only steps (captured graphs): along the given tokens the logits stay with the plain implementation."""
    d, reqs, want = models["C"]
    eng = H.engine_for(d, "bfloat16", 16, 1024)
    a, b = reqs[3], reqs[2]
    steps = [([(3, a[:15], [14]), (2, b[:4], [3])], [])]
    for i in range(140):
        steps.append(([(3, [a[15 + i]], [0])] + ([(2, [b[4 + i]], [0])] if 4 + i < len(b) else []), []))
    check(H.run_steps(eng, steps), want, BF16_TOL, "C bfloat16 long decoding")
    assert len(eng._graphs) > 0


def test_the_plain_forms_can_be_pinned(models):
    """A bfloat16 engine on the plain kernels (no chunks, no tensor-core attention) gives the same logits."""
    from aien_sovereign_core_mv_b200 import kernels as K
    d, reqs, want = models["C"]
    saved = K._MATRIX_MEMORY_IMPL, K._LATENT_IMPL
    K._MATRIX_MEMORY_IMPL, K._LATENT_IMPL = "walk", "plain"
    try:
        eng = H.engine_for(d, "bfloat16", 16, 512)
        check(H.run_steps(eng, [([(3, reqs[3], list(range(len(reqs[3]))))], [3])]), want, BF16_TOL, "C on plain kernels")
    finally:
        K._MATRIX_MEMORY_IMPL, K._LATENT_IMPL = saved


def test_greedy_generation_through_the_entry_point(models):
    from aien_sovereign_core_mv_b200.engine.generate import generate
    from aien_sovereign_core_mv_b200.sampling import SamplingParams
    d, reqs, _ = models["A"]
    cfg, tensors = load_plain(d)
    prompts = [reqs[2], reqs[3][:30], reqs[1]]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(8):
            seq.append(int(np.argmax(pk.forward(cfg, tensors, seq)[-1])))
        want.append(seq[len(p):])
    eng = H.engine_for(d, "float32", 16, 512, prefill_chunk_size=16, max_prefill_tokens=32)
    got = generate(eng, prompts, SamplingParams(temperature=0.0, max_tokens=8, stop_token_ids=[]))
    assert got == want
    assert eng.cache_state()["requests"] == 0 and eng.cache_state()["check"] == ""


def test_sampling_and_the_command_line(models):
    import subprocess
    from aien_sovereign_core_mv_b200.engine.generate import Generator
    from aien_sovereign_core_mv_b200.sampling import SamplingParams
    d, reqs, _ = models["B"]
    eng = H.engine_for(d, "bfloat16", 8, 512)
    params = SamplingParams(temperature=0.8, top_p=0.9, top_k=40, max_tokens=12, stop_token_ids=[], seed=7)
    a = Generator(eng).generate([reqs[2], reqs[1]], params, request_ids=[5, 6])
    b = Generator(eng).generate([reqs[2], reqs[1]], params, request_ids=[5, 6])
    assert [r.tokens for r in a] == [r.tokens for r in b] and all(len(r.tokens) == 12 for r in a)
    cfg, tensors = load_plain(d)
    seq = list(reqs[1])
    for _ in range(5):
        seq.append(int(np.argmax(pk.forward(cfg, tensors, seq)[-1])))
    exe = os.path.join(H.ROOT, "bin", "aien-b200")
    out = subprocess.run([exe, "generate", "--model-dir", d, "--dtype", "float32", "--prompt-ids", ",".join(map(str, reqs[1])),
                          "--max-tokens", "5", "--temperature", "0", "--stop-token-ids", "", "--json"], capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert json.loads(out.stdout.strip().splitlines()[-1])["tokens"] == [seq[len(reqs[1]):]]
    info = subprocess.run([exe, "info", "--model-dir", d], capture_output=True, text=True, timeout=600)
    assert info.returncode == 0, info.stderr[-2000:]
    rec = json.loads(info.stdout.strip().splitlines()[-1])
    assert rec["architecture"] == "Kuvidra" and rec["layers"] == 3 and "full" in rec["cache_groups"] and "state" in rec["cache_groups"]


def test_trace_replay_from_the_command(models, tmp_path):
    d, reqs, want = models["A"]
    toks = reqs[3]
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:40], "want": [0, 39]}, {"id": 7, "tokens": reqs[1], "want": [0]}], "end": [7]},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[40:42], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[42:], "want": [len(toks) - 43]}], "end": ["x"]}]
    out = H.run_trace(d, "float32", str(tmp_path / "out"), 192, steps)
    assert sorted(out) == [0, 2]
    H.assert_close(out[0], np.stack([want[3][0], want[3][39], want[1][0]]), FP32_TOL, "trace step 0")
    H.assert_close(out[2], want[3][-1:], FP32_TOL, "trace step 2")


# ------------------------------------------------------------------ configurations drawn at random
def _random_config(rng):
    width = rng.choice([64, 72, 96, 128])
    layers = []
    for _ in range(rng.randint(2, 5)):
        if rng.random() < 0.5:
            dim = rng.choice([8, 16, 24, 40, 64])
            layer = _lat(rng.choice([1, 2, 3, 6]), dim, rng.choice([8, 16, 40, 64]), rng.choice([16, 36, 64, 96, 128, 184]), rng.choice([24, 50, 96]),
                         rng.choice([0.15, 0.4, dim ** -0.5]))
        else:
            layer = _mem(rng.choice([1, 2, 5]), rng.choice([8, 16, 32, 48, 80]), rng.choice([8, 16, 48, 72, 112]), rng.choice([3.0, 10.0, 15.0, 30.0]))
        r = rng.random()
        if r < 0.2:
            layer = _none(layer)
        elif r < 0.5:
            layer = _dense(layer, rng.choice([24, 40, 96]))
        else:
            E = rng.choice([1, 2, 5, 9])
            layer = _moe(layer, E, rng.randint(1, E), rng.choice([12, 16, 64]), rng.choice([0, 20, 40]))
        layers.append(layer)
    cfg = {"architecture": "Kuvidra", "vocab": rng.choice([101, 256, 333]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}
    if rng.random() < 0.7:
        a = rng.randint(0, len(layers) - 1)
        cfg["loop"] = {"start": a, "stop": rng.randint(a + 1, len(layers)), "times": rng.randint(1, 3)}
    return cfg


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Whole prompts, portions of changing size and three requests side by side; float32 with random weights as they
    come, bfloat16 with well-conditioned ones."""
    for dtype, tol in (("float32", FP32_TOL), ("bfloat16", 2 * BF16_TOL)):
        rng = random.Random(seed)
        cfg = _random_config(rng)
        d = write_model(os.path.join(str(tmp_path), dtype), cfg, 4000 + seed, rng.choice([1.0, 2.0]), dtype == "bfloat16")
        c, tensors = load_plain(d)
        draw = np.random.default_rng(seed)
        reqs = {i + 1: [int(x) for x in draw.integers(0, cfg["vocab"], n)] for i, n in enumerate([rng.randint(1, 30), rng.randint(60, 100), rng.randint(130, 160)])}
        want = {r: pk.forward(c, tensors, t) for r, t in reqs.items()}
        portions = []
        for rid, t in reqs.items():
            at = 0
            while at < len(t):
                n = min(rng.choice([1, 2, 3, 7, 16, 33, 64, 129]), len(t) - at)
                portions.append(([(rid, t[at:at + n], list(range(n)))], [rid] if at + n == len(t) else []))
                at += n
        whole = [([(rid, t, list(range(len(t))))], [rid]) for rid, t in reqs.items()]
        for mode, steps in (("whole", whole), ("portions", portions), ("side by side", _side_by_side(reqs, rng, 3))):
            eng = H.engine_for(d, dtype, rng.choice([8, 16, 32]), 512, max_requests=4)
            check(H.run_steps(eng, steps), want, tol, f"seed {seed} {dtype} {mode}")
            assert eng.cache_state()["check"] == "" and eng.cache_state()["requests"] == 0
