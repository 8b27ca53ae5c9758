"""The Folavik design in the engine against its plain implementation (``plain_folavik``): each mechanism alone, then whole
models under every way of cutting the work, in float32 and bfloat16.

The configurations are small and differ from one another in every size and constant: value sizes below, equal to and above
the key size, sizes that the tensor-core, warp-wise and vector kernels take and refuse, one, several and as many key/value
heads as query heads, windows and chunks of a few tokens up to more than the prompt, frequency scalings whose ramps start and
end inside and outside the rotated pairs, a difference constant of zero, layers without a feed-forward, models of one kind of
mixer only.  Where random weights would hide a fault the inputs are made so that it shows: queries are scaled until single keys
stand out, keys at positions 0, at page borders and just inside and outside a window or chunk are made large.
"""
import json
import os
import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import helpers as H
import plain_folavik as pf
from test_gpu_kuvidra import _side_by_side
from test_gpu_mumazen import _bound_part, check, f64, i32, load_plain, make_ctx

pytestmark = pytest.mark.gpu


def _dif(heads, kv, dim, vdim, window, cap, diff, scale, dims, base, factor, original, fast, slow):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "diff": diff,
                                             "mask": {"size": window}, "rot": {"base": base, "dims": dims, "scaling": {
                                                 "factor": factor, "original": original, "fast": fast, "slow": slow}}}}


def _att(heads, kv, dim, vdim, chunk, scale, dims, base, factor, low, high, original):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk},
                                           "rot": {"base": base, "dims": dims, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}}}


def _lat(heads, dim, vdim, kv_rank, scale):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}}


def _ff(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff} if ff else None)


CONFIGS = {
    # every mixer; windows and chunks across pages; a layer without a feed-forward
    "A": {"architecture": "Folavik", "vocab": 301, "width": 96, "norm": {"eps": 1e-5}, "logit_scale": 0.5, "logit_softcap": 12.0, "layers": [
        _ff(_dif(6, 2, 16, 24, 37, 20.0, 0.3, 0.3, 12, 1000.0, 3.0, 64, 8.0, 1.0), 136), _ff(_lat(5, 24, 16, 72, 0.25), 0),
        _ff(_att(6, 3, 24, 40, 45, 0.2, 16, 5000.0, 5.0, 1.0, 4.0, 90), 64), _ff(_dif(4, 4, 8, 64, 20, 6.0, 0.7, 0.5, 8, 300.0, 2.0, 40, 4.0, 2.0), 40)]},
    # sizes that no tensor-core, warp-wise or vector kernel takes: width 90, heads of 10 and 7, a latent of 30; difference constant 0
    "B": {"architecture": "Folavik", "vocab": 203, "width": 90, "norm": {"eps": 3e-6}, "logit_scale": 1.0, "logit_softcap": 30.0, "layers": [
        _ff(_lat(3, 11, 10, 30, 0.3), 50), _ff(_dif(3, 1, 10, 7, 9, 15.0, 0.0, 0.4, 4, 50.0, 4.0, 30, 2.0, 0.5), 0),
        _ff(_att(2, 2, 14, 9, 13, 0.3, 6, 100.0, 2.0, 0.5, 2.0, 20), 33)]},
    # sizes of the wide kernels; two differential layers that share a cache group; a window beyond the prompt, chunks of a page
    "C": {"architecture": "Folavik", "vocab": 512, "width": 128, "norm": {"eps": 1e-6}, "logit_scale": 2.0, "logit_softcap": 20.0, "layers": [
        _ff(_dif(8, 2, 64, 128, 150, 30.0, 0.5, 0.125, 64, 10000.0, 4.0, 512, 32.0, 1.0), 256),
        _ff(_dif(8, 2, 64, 128, 150, 50.0, 0.2, 0.15, 20, 500.0, 8.0, 128, 16.0, 4.0), 96), _ff(_lat(8, 64, 64, 128, 0.125), 256),
        _ff(_att(4, 1, 128, 64, 16, 0.09, 128, 500000.0, 8.0, 1.0, 4.0, 256), 64), _ff(_att(8, 8, 32, 32, 128, 0.18, 32, 2000.0, 2.0, 1.0, 8.0, 100), 128)]},
    # differential attention only, one map group, a window of one page and of three tokens
    "D": {"architecture": "Folavik", "vocab": 130, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 0.25, "logit_softcap": 5.0, "layers": [
        _ff(_dif(1, 1, 48, 80, 16, 25.0, 0.8, 0.2, 24, 10000.0, 16.0, 256, 32.0, 1.0), 72), _ff(_dif(5, 5, 32, 16, 3, 3.0, 0.4, 0.3, 2, 10.0, 2.0, 8, 2.0, 1.0), 24)]},
    # latent attention only, the latent wider than the model
    "E": {"architecture": "Folavik", "vocab": 222, "width": 72, "norm": {"eps": 1e-6}, "logit_scale": 1.5, "logit_softcap": 8.0, "layers": [
        _ff(_lat(5, 16, 40, 160, 0.25), 88), _ff(_lat(2, 32, 8, 64, 0.3), 0)]},
}
PAGE = {"A": 16, "B": 8, "C": 16, "D": 16, "E": 32}
LENGTHS = {"A": [1, 9, 50, 150], "B": [2, 20, 77], "C": [5, 70, 200], "D": [3, 40, 140], "E": [2, 33, 130]}
SHARP = 2.0                                                          # queries times this: single keys, near and far, stand out
FP32_TOL, BF16_TOL = 1e-4, 5e-2
DTYPES = [("float32", FP32_TOL), ("bfloat16", BF16_TOL)]


def tokens(which, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, CONFIGS[which]["vocab"], n)]


def write_model(folder, cfg, seed, sharp=SHARP, half=False):
    """A random model folder: the attention's queries scaled; the difference's vectors scaled until lambda differs from layer
    to layer; biases and the embedding's mean well away from zero.  ``half``: lambda lies near 0.5 in every layer, so that two
    maps that see much the same do not cancel down to their rounding."""
    from aien_sovereign_core_mv_b200 import model_spec_for
    from aien_sovereign_core_mv_b200.models.decoder import Decoder
    from aien_sovereign_core_mv_b200.weights.random_init import random_tensor
    from aien_sovereign_core_mv_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    out = {}
    for name, (shape, kind) in Decoder(model_spec_for(cfg)[1]).catalog().items():
        t = random_tensor(name, tuple(shape), kind, seed).float()
        if name.endswith("mix.q"):
            t *= sharp
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t *= 10.0 * (shape[0] ** -0.25) * 0.7
        elif name.endswith(".b"):
            t *= 5.0
        elif name == "embed":
            t += 0.7
        out[name] = t.to(torch.bfloat16)
    for i, layer in enumerate(cfg["layers"]):
        if half and layer["type"] == "attention_2":                  # exp(0) - exp(ln(0.5 + diff)) + diff
            p = f"l{i}.mix."
            out[p + "lq1"] = torch.zeros_like(out[p + "lq1"])
            k2 = out[p + "lk2"].float()
            out[p + "lq2"] = (k2 * (np.log(0.5 + layer["mixer"]["diff"]) / float(k2 @ k2))).to(torch.bfloat16)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), out)
    return folder


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("folavik")
    out = {}
    for i, which in enumerate(CONFIGS):
        d = write_model(os.path.join(str(root), which), CONFIGS[which], 60 + i)
        cfg, tensors = load_plain(d)
        reqs = {j + 1: tokens(which, n, 100 * i + n) for j, n in enumerate(LENGTHS[which])}
        want = {rid: pf.forward(cfg, tensors, toks) for rid, toks in reqs.items()}
        out[which] = (d, reqs, want)
    return out


# ------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 90, 256, 1000, 2052, 5000, 9000])
def test_layer_norm_and_pending_sums(dtype, width):
    """The stream's mean is a thousand times its spread: sums of squares without the mean taken off first would lose it."""
    from aien_sovereign_core_mv_b200 import kernels as K
    g = torch.Generator().manual_seed(width)
    eps = 1e-5
    w = (torch.rand(width, generator=g) + 0.5).to(dtype)
    for T in (3, 200):
        x0 = torch.randn(T, width, generator=g) + torch.where(torch.arange(T) % 2 == 0, 1000.0, 0.0)[:, None]
        parts = torch.randn(3, T, width, generator=g)
        low = torch.randn(T, width, generator=g).to(torch.bfloat16)
        for delta in (None, low, parts, parts[0].contiguous()):
            x, h = x0.clone().cuda(), torch.zeros(T, width, dtype=dtype).cuda()
            K.add_layernorm(x, None if delta is None else delta.cuda(), w.cuda(), eps, h)
            new = f64(x0) + (0.0 if delta is None else (f64(delta).sum(0) if delta.dim() == 3 else f64(delta)))
            H.assert_close(x.cpu().numpy(), new, 2e-7 * 3, "the stream after the sum")
            want = pf.layer_norm(f64(x), f64(w), eps)
            H.assert_close(h.float().cpu().numpy(), want, 2e-4 if dtype == torch.float32 else 6e-3, "rows with a large mean")
            H.assert_close(h.float().cpu().numpy()[1::2], want[1::2], 3e-6 if dtype == torch.float32 else 6e-3, "the norm")
        x = x0.clone().cuda()
        h = torch.zeros(T, width, dtype=dtype).cuda()
        K.stream_norm_inplace(x, w.cuda(), eps, h=h, center=True)
        H.assert_close(x.cpu().numpy(), pf.layer_norm(f64(x0), f64(w), eps), 2e-4, "in place")
        H.assert_close(h.float().cpu().numpy(), f64(x), 1e-7 if dtype == torch.float32 else 5e-3, "its copy")


@pytest.mark.parametrize("yarn", [True, False])
@pytest.mark.parametrize("dims", [2, 12, 64])
def test_rotation_tables(yarn, dims):
    from aien_sovereign_core_mv_b200.registry import make_part
    rot = {"base": 3000.0, "dims": dims}
    if yarn:
        rot["scaling"] = {"factor": 6.0, "original": 300, "fast": 9.0, "slow": 1.0}
        freq, mult = pf.yarn_frequencies(rot)
        part = make_part("position", "rotary", head_dim=64, theta=3000.0, rotary_dim=dims, theta_as_float32=False, yarn=rot["scaling"])
    else:
        rot["scaling"] = {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 300}
        freq, mult = pf.smoothed_frequencies(rot), 1.0
        part = make_part("position", "rotary", head_dim=64, theta=3000.0, rotary_dim=dims, theta_as_float32=False, scaling={
            "factor": 6.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0, "original_max_position_embeddings": 300})
    pos = [0, 1, 2, 77, 299, 300, 4095, 131071]
    cos, sin, n = part.rotary(make_ctx(torch.float32, pos, list(range(8)), list(range(9)), [p + 1 for p in pos]))
    a = np.asarray(pos, dtype=np.float64)[:, None] * freq
    assert n == dims
    H.assert_close(cos.cpu().numpy(), np.cos(a) * mult, 1e-7, "cos")
    H.assert_close(sin.cpu().numpy(), np.sin(a) * mult, 1e-7, "sin")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,nv,hd,hdv,rot,bias,parts", [(3, 3, 3, 10, 14, 6, True, 1), (8, 4, 2, 16, 24, 16, True, 1), (6, 2, 2, 64, 32, 32, False, 3), (16, 8, 4, 64, 128, 64, True, 2),
                                                             (2, 1, 1, 40, 8, 12, True, 4), (5, 5, 5, 56, 104, 0, True, 1), (3, 1, 1, 128, 16, 128, False, 1)])
def test_bias_rotation_and_cache_write(dtype, nq, nkv, nv, hd, hdv, rot, bias, parts):
    """Rows in the compute dtype or as partial products, a bias per column, values with heads of their own; a token without a
    slot writes nothing."""
    from aien_sovereign_core_mv_b200 import kernels as K
    g = torch.Generator().manual_seed(hd * 7 + hdv)
    T, cols = 9, nq * hd + nkv * hd + nv * hdv
    proj = torch.randn(parts, T, cols, generator=g)
    proj = proj[0].to(dtype) if parts == 1 else proj
    b = torch.randn(cols, generator=g) if bias else None
    pos = [0, 1, 5, 17, 100, 1000, 33, 2, 8]
    freq, mult = np.array([0.7 ** i for i in range(rot // 2)]), 1.3
    a = np.asarray(pos, dtype=np.float64)[:, None] * freq
    cos, sin = (torch.tensor(np.cos(a) * mult, dtype=torch.float32).cuda(), torch.tensor(np.sin(a) * mult, dtype=torch.float32).cuda()) if rot else (None, None)
    slots = [4, 9, -1, 0, 11, 7, 2, 3, 10]
    kc, vc = torch.full((12, nkv, hd), 7.0, dtype=dtype).cuda(), torch.full((12, nv, hdv), 7.0, dtype=dtype).cuda()
    q = torch.zeros(T, nq * hd, dtype=dtype).cuda()
    K.rope_halves_value_write(proj.cuda(), 0, nq * hd, (nq + nkv) * hd, nq, nkv, hd, hdv, cos, sin, rot, i32(slots), q, kc, vc,
                              bias=None if b is None else b.cuda(), nv=nv)
    row = (f64(proj).sum(0) if parts > 1 else f64(proj)) + (0.0 if b is None else f64(b))
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    turn = lambda x: pf.rotate(x, pos, freq, mult) if rot else x
    H.assert_close(q.float().cpu().numpy().reshape(T, nq, hd), turn(row[:, :nq * hd].reshape(T, nq, hd)), tol, "q")
    wk, wv = np.full((12, nkv, hd), 7.0), np.full((12, nv, hdv), 7.0)
    for t, s in enumerate(slots):
        if s >= 0:
            wk[s] = turn(row[:, nq * hd:(nq + nkv) * hd].reshape(T, nkv, hd))[t]
            wv[s] = row[t, (nq + nkv) * hd:].reshape(nv, hdv)
    H.assert_close(kc.float().cpu().numpy(), wk, tol, "keys")
    H.assert_close(vc.float().cpu().numpy(), wv, tol, "values")


def _attention_case(dtype, page, heads, kv, maps, dim, vdim, window, chunk, cap, lens, seed):
    """Requests in one paged cache whose keys at the places that matter are large; slots nobody owns hold large numbers.
    Returns run(entries, call, want, tol): one step over the given (request, first position, count) through ``call``, against
    ``want`` of the plain maps."""
    from aien_sovereign_core_mv_b200 import kernels as K
    g = torch.Generator().manual_seed(seed)
    scale = 1.5 * dim ** -0.5
    size = window or chunk
    sees = pf.sees_window(window) if window else (pf.sees_chunk(chunk) if chunk else pf.sees_all)
    H2, G2 = heads * maps, kv * maps                                 # query heads, key heads; maps neighbouring key heads share a value head
    ks, vs, qs = [], [], []
    for n in lens:
        k = torch.randn(n, G2, dim, generator=g)
        places = {0, page - 1, page, n // 2, n - 1} | {p for e in range(0, n + 1, size or n) for p in (e - 1, e, e + 1)}
        for p in places:
            if 0 <= p < n:
                k[p] *= 2.5
        ks.append(k.to(dtype).float())
        vs.append((torch.randn(n, kv, vdim, generator=g) + 0.3 * torch.arange(n)[:, None, None] / n).to(dtype).float())
        qs.append(torch.randn(n, H2, dim, generator=g).to(dtype).float())
    pages = [(n + page - 1) // page for n in lens]
    order = torch.randperm(sum(pages) + 5, generator=g).tolist()
    width = max(pages) + 1
    total = (sum(pages) + 5) * page
    kc, vc = torch.full((total, G2, dim), 300.0, dtype=dtype), torch.full((total, kv, vdim), 300.0, dtype=dtype)
    bt = torch.full((len(lens), width), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(lens):
        tab = order[at:at + pages[s]]
        at += pages[s]
        bt[s, :pages[s]] = torch.tensor(tab)
        for p in range(n):
            kc[tab[p // page] * page + p % page], vc[tab[p // page] * page + p % page] = ks[s][p], vs[s][p]
    kc, vc = kc.cuda(), vc.cuda()

    def plain(s, p0, n):
        """[n, maps-major heads of every group, vdim]: per key/value head map 1's query heads, then map 2's."""
        return pf.softmax_attention(f64(qs[s][p0:p0 + n]), f64(ks[s]), np.repeat(f64(vs[s]), maps, 1), sees, scale, cap, list(range(p0, p0 + n)))

    def run(entries, call, want, tol, back=True):
        pos, sot, rows, q_start, ctx_len = [], [], [], [0], []
        table = torch.stack([bt[s] for s, _, _ in entries]).contiguous()
        for i, (s, p0, n) in enumerate(entries):
            pos += list(range(p0, p0 + n)); sot += [i] * n
            rows.append(qs[s][p0:p0 + n].reshape(n, H2 * dim))
            q_start.append(q_start[-1] + n); ctx_len.append(p0 + n)
            if back and size:                                        # pages behind the window or chunk are given back
                first = max(0, p0 - window + 1) if window else (p0 // chunk) * chunk
                table[i, :first // page] = -1
        ctx = make_ctx(dtype, pos, sot, q_start, ctx_len)
        if not ctx.decode_only:
            single = [q_start[i] for i, (_, _, n) in enumerate(entries) if n == 1]
            ts = sum([[i] * ((n + 127) // 128) for i, (_, _, n) in enumerate(entries) if n > 1], [])
            tq = sum([list(range(0, n, 128)) for _, _, n in entries if n > 1], [])
            ctx.prefill_tiles = (i32(ts or [0]), i32(tq or [0]), len(ts))
            ctx.single_tokens = (i32(single or [0]), len(single))
        group = SimpleNamespace(block_table=table.cuda(), max_blocks=width, page_size=page)
        got = call(K, ctx, torch.cat(rows).to(dtype).cuda(), kc, vc, group, scale)
        H.assert_close(got, np.concatenate([want(plain(s, p0, n)) for s, p0, n in entries]), tol, f"entries {entries}")

    return run


# (page, heads, kv, maps, dim, vdim, window, chunk, cap)
ATTENTIONS = [(8, 3, 3, 1, 10, 14, 23, 0, 0.0), (16, 6, 2, 1, 24, 40, 0, 45, 0.0), (16, 4, 1, 1, 56, 32, 0, 128, 0.0), (16, 8, 2, 1, 128, 64, 64, 0, 20.0),
              (16, 6, 3, 2, 48, 80, 120, 0, 9.0), (32, 6, 2, 2, 16, 24, 33, 0, 15.0), (16, 8, 1, 2, 64, 128, 100, 0, 30.0), (8, 3, 1, 2, 10, 7, 9, 0, 5.0),
              (16, 2, 1, 1, 64, 128, 0, 16, 12.0), (16, 5, 5, 2, 32, 64, 0, 70, 0.0), (64, 16, 1, 1, 64, 64, 0, 0, 8.0), (16, 12, 1, 2, 40, 120, 31, 0, 40.0),
              (8, 4, 4, 1, 200, 136, 50, 0, 0.0)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("page,heads,kv,maps,dim,vdim,window,chunk,cap", ATTENTIONS)
def test_attention_over_values_of_their_own(dtype, page, heads, kv, maps, dim, vdim, window, chunk, cap):
    """Whole prompts, portions, single tokens alone and beside portions; float32 results and results in the compute dtype;
    single tokens on every kernel that takes them."""
    from aien_sovereign_core_mv_b200 import kernels as K
    size = window or chunk or 100
    n = 300
    run = _attention_case(dtype, page, heads, kv, maps, dim, vdim, window, chunk, cap, [n, 41, 2], page + heads + dim)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    steps = [[(0, 0, n), (1, 0, 41), (2, 0, 2)], [(0, 130, 140), (1, 40, 1)], [(0, n - 1, 1), (1, 20, 1), (2, 1, 1)], [(1, 21, 2), (0, 127, 3), (2, 0, 1)]]
    steps += [[(0, p, 1)] for p in (0, size - 1, size, size + 1, 2 * size) if p < n] + [[(0, p - 1, 2)] for p in (size, size + 1) if p < n]
    for out_dtype in {torch.float32, dtype}:
        def call(K, ctx, q, kc, vc, group, scale):
            out = torch.full((q.shape[0], heads * maps * vdim), float("nan"), dtype=out_dtype).cuda()
            K.capped_attention(ctx, q, kc, vc, group, out, heads * maps, kv * maps, dim, vdim, window, scale, cap, chunk, v_share=maps)
            return out.float().cpu().numpy().reshape(q.shape[0], heads * maps, vdim)
        saved = K._DECODE_VALUES_IMPL
        try:
            for impl in ("warps", "direct"):
                K._DECODE_VALUES_IMPL = impl
                for entries in steps:
                    run(entries, call, lambda x: x, tol)
        finally:
            K._DECODE_VALUES_IMPL = saved


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("page,heads,kv,maps,dim,vdim,window,chunk,cap", [a for a in ATTENTIONS if a[3] == 2])
def test_difference_of_two_maps(dtype, page, heads, kv, maps, dim, vdim, window, chunk, cap):
    """Both forms (maps and difference in one kernel for single tokens, two kernels otherwise) against the plain difference;
    lambda so that the two maps neither cancel nor drown one another."""
    lam, diff, eps, per, n = 0.6, 0.25, 1e-5, heads // kv, 300
    run = _attention_case(dtype, page, heads, kv, maps, dim, vdim, window, chunk, cap, [n, 41], 3 * page + heads)

    def call(K, ctx, q, kc, vc, group, scale):
        out = torch.full((q.shape[0], heads * vdim), float("nan"), dtype=dtype).cuda()
        K.difference_attention(ctx, q, kc, vc, group, out, heads, kv, dim, vdim, window, scale, cap, chunk, lam, eps, 1.0 - diff)
        return out.float().cpu().numpy().reshape(q.shape[0], heads, vdim)

    def want(x):
        x = x.reshape(x.shape[0], kv, 2, per, vdim)
        return pf.combine_maps(x[:, :, 0], x[:, :, 1], lam, diff, eps).reshape(x.shape[0], heads, vdim)

    tol = 5e-5 if dtype == torch.float32 else 3e-2
    for entries in ([(0, 0, n), (1, 0, 41)], [(0, 130, 140), (1, 40, 1)], [(0, n - 1, 1), (1, 20, 1)], [(0, 0, 1)], [(1, 3, 1), (0, 140, 1)]):
        run(entries, call, want, tol)


@pytest.mark.parametrize("dim,vdim,maps,heads,kv,window,cap", [(64, 128, 2, 8, 2, 0, 30.0), (128, 128, 1, 16, 4, 0, 0.0), (32, 32, 1, 3, 3, 1500, 10.0), (128, 40, 2, 2, 1, 0, 6.0)])
def test_single_tokens_with_long_contexts(dim, vdim, maps, heads, kv, window, cap):
    """One, three and forty tokens a step over thousands of keys: the keys of a token are cut into many ranges, few, or one."""
    n = 2600
    run = _attention_case(torch.bfloat16, 16, heads, kv, maps, dim, vdim, window, 0, cap, [n, 700, 90], dim + heads)

    def call(K, ctx, q, kc, vc, group, scale):
        assert K.decode_warps_supports(heads * maps, kv * maps, dim, vdim, maps)
        out = torch.full((q.shape[0], heads * maps * vdim), float("nan"), dtype=torch.float32).cuda()
        K.capped_attention(ctx, q, kc, vc, group, out, heads * maps, kv * maps, dim, vdim, window, scale, cap, 0, v_share=maps)
        return out.cpu().numpy().reshape(q.shape[0], heads * maps, vdim)

    for entries in ([(0, n - 1, 1)], [(0, 2048, 1), (1, 699, 1), (2, 17, 1)], [(0, 2500 + i, 1) for i in range(0, 98, 7)] + [(1, 600 + i, 1) for i in range(20)] + [(2, i, 1) for i in range(6)]):
        run(entries, call, lambda x: x, 2e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H_,V,per", [(1, 4, 32, 2), (7, 6, 80, 3), (33, 3, 7, 1), (5, 8, 128, 8), (3, 2, 256, 1), (4, 5, 130, 5)])
def test_difference_and_norm_per_head(dtype, T, H_, V, per):
    from aien_sovereign_core_mv_b200 import kernels as K
    g = torch.Generator().manual_seed(V)
    a = torch.randn(T, 2 * H_ * V, generator=g)
    a[0] *= 1e-4                                                     # eps decides here
    lam, eps, mult = -0.7, 1e-5, 0.4
    out = torch.zeros(T, H_ * V, dtype=dtype).cuda()
    K.map_difference_norm(a.cuda(), out, H_, per, V, lam, eps, mult)
    x = f64(a).reshape(T, H_ // per, 2, per, V)
    want = pf.combine_maps(x[:, :, 0], x[:, :, 1], lam, 1.0 - mult, eps)
    H.assert_close(out.float().cpu().numpy().reshape(want.shape), want, 2e-6 if dtype == torch.float32 else 5e-3, "rows")
    H.assert_close(out.float().cpu().numpy()[0].reshape(want[0].shape), want[0], 2e-6 if dtype == torch.float32 else 5e-3, "the small row")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff", [(64, 96), (128, 256), (90, 33), (72, 40), (512, 1024)])
def test_gated_feed_forward_with_the_tanh_gelu(dtype, width, ff):
    """Streamed, tiled and persistent products with the activation in their epilogue, and the plain ones."""
    part, W = _bound_part("feed_forward", "swiglu", 9, dtype, hidden_size=width, intermediate_size=ff, act="gelu_tanh")
    Wt = {"gate": W["gate_proj"] , "up": W["up_proj"], "down": W["down_proj"]}
    for T in (1, 5, 12, 60, 300):
        g = torch.Generator().manual_seed(T)
        h = (torch.randn(T, width, generator=g) * 1.5).to(torch.bfloat16)
        y = part.forward(make_ctx(dtype, list(range(T)), [0] * T, [0, T], [T]), h.to(dtype).cuda())
        y = y.float().sum(0) if y.dim() == 3 else y.float()
        H.assert_close(y.cpu().numpy(), pf.dense_ff(Wt, "", f64(h)), 1e-5 if dtype == torch.float32 else 2e-2, f"{T} tokens")


def test_scaled_and_capped_logits():
    from aien_sovereign_core_mv_b200 import kernels as K
    v = torch.randn(7, 131, generator=torch.Generator().manual_seed(2)) * 40.0
    for cap, mult in ((9.0, 0.3), (0.0, 1.7), (30.0, 1.0)):
        x = v.clone().cuda()
        K.softcap(x, cap, mult)
        want = f64(v) * mult
        H.assert_close(x.cpu().numpy(), cap * np.tanh(want / cap) if cap else want, 1e-6, f"cap {cap}")


@pytest.mark.parametrize("form", ["expand", "absorb"])
@pytest.mark.parametrize("heads,dim,vdim,rank,page", [(4, 32, 48, 64, 16), (3, 64, 8, 200, 8), (16, 128, 128, 512, 16), (6, 8, 72, 40, 32)])
def test_latent_attention_with_a_gate_per_element(form, heads, dim, vdim, rank, page):
    """The bfloat16 mixer in both forms of its portions: whole prompts of two requests, then portions beside single tokens,
    then single tokens, from one cache; large latents at position 0 and page borders."""
    from aien_sovereign_core_mv_b200 import kernels as K
    from aien_sovereign_core_mv_b200.parts.base import GroupView, RunBinding
    from test_gpu_parts import make_ctx as make_big_ctx
    width, eps = 96, 1e-5
    part, W = _bound_part("mixer", "latent_attention", 5, torch.bfloat16, hidden_size=width, num_heads=heads, head_dim=dim, rot_dim=0, value_dim=vdim,
                          kv_rank=rank, q_rank=0, position=SimpleNamespace(), scale=2.0 * dim ** -0.5, norm_eps=eps, out_gate=True)
    Wt = {"q": W["q_proj"], "dkv": W["dkv_proj"], "dkv.norm": W["dkv_norm"], "uk": W["uk_proj"], "uv": W["uv_proj"], "g": W["g_proj"], "o": W["o_proj"]}
    lens = [170, 23]
    g = torch.Generator().manual_seed(rank)
    hs = [torch.randn(n, width, generator=g).to(torch.bfloat16) for n in lens]
    want = [pf.latent_attention({"heads": heads, "dim": dim, "vdim": vdim, "scale": 2.0 * dim ** -0.5}, Wt, "", f64(h), eps) for h in hs]
    pages = [(n + page - 1) // page for n in lens]
    order = torch.randperm(sum(pages) + 3, generator=g).tolist()
    tabs = [order[:pages[0]], order[pages[0]:sum(pages)]]
    store = torch.full((1, (sum(pages) + 3) * page, rank), 50.0, dtype=torch.bfloat16).cuda()
    width_b = max(pages) + 2
    saved = K.LATENT_PORTIONS
    K.LATENT_PORTIONS = form
    try:
        for steps in ([[(0, 0, 170), (1, 0, 23)]], [[(0, 0, 100), (1, 0, 1)], [(0, 100, 68), (1, 1, 1)], [(1, 2, 20)], [(0, 168, 1), (1, 22, 1)], [(0, 169, 1)]],
                      [[(1, 0, 2), (0, 0, 1)], [(0, 1, 129), (1, 2, 1)], [(0, 130, 1), (1, 3, 20)], [(0, 131, 39)]]):
            for step in steps:
                pos, sot, slots, q_start, ctx_len = [], [], [], [0], []
                for i, (s, p0, n) in enumerate(step):
                    pos += list(range(p0, p0 + n)); sot += [i] * n
                    slots += [tabs[s][p // page] * page + p % page for p in range(p0, p0 + n)]
                    q_start.append(q_start[-1] + n); ctx_len.append(p0 + n)
                bt = torch.full((len(step), width_b), -1, dtype=torch.int32)
                for i, (s, _, _) in enumerate(step):
                    bt[i, :pages[s]] = torch.tensor(tabs[s])
                ctx = make_big_ctx(torch.bfloat16, pos, sot, q_start, ctx_len, [GroupView("full", page, 0, width_b, bt.cuda(), i32(slots), {"latent": store})], 1 << 27)
                if not ctx.decode_only:
                    single = [q_start[i] for i, (_, _, n) in enumerate(step) if n == 1]
                    ts = sum([[i] * ((n + 127) // 128) for i, (_, _, n) in enumerate(step) if n > 1], [])
                    tq = sum([list(range(0, n, 128)) for _, _, n in step if n > 1], [])
                    ctx.prefill_tiles, ctx.single_tokens = (i32(ts or [0]), i32(tq or [0]), len(ts)), (i32(single or [0]), len(single))
                h = torch.cat([hs[s][p0:p0 + n] for s, p0, n in step]).cuda()
                y = part.forward(ctx, h, RunBinding(0, 0, True))
                y = (y.float().sum(0) if y.dim() == 3 else y.float()).cpu().numpy()
                H.assert_close(y, np.concatenate([want[s][p0:p0 + n] for s, p0, n in step]), 4e-2, f"{form} step {step}")
    finally:
        K.LATENT_PORTIONS = saved


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
    cut = len(toks) - 60
    steps = [([(rid, toks[:cut], [0, cut - 1])], [])] + [([(rid, [toks[i]], [0])], []) for i in range(cut, len(toks))]
    check(H.run_steps(eng, steps), want, tol, f"{which} {dtype} decode")
    assert eng.cache_state()["check"] == ""


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_first_tokens_one_by_one(models, which, dtype, tol):
    d, reqs, want = models[which]
    eng = H.engine_for(d, dtype, PAGE[which], 512)
    rid = max(reqs, key=lambda r: len(reqs[r]))
    steps = [([(rid, [t], [0])], []) for t in reqs[rid][:60]]
    check(H.run_steps(eng, steps), want, tol, f"{which} {dtype} from the first token")


@pytest.mark.parametrize("latent", ["expand", "absorb"])
@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_changing_portions(models, which, dtype, tol, latent):
    from aien_sovereign_core_mv_b200 import kernels as K
    d, reqs, want = models[which]
    saved = K.LATENT_PORTIONS
    K.LATENT_PORTIONS = latent
    try:
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
    finally:
        K.LATENT_PORTIONS = saved


@pytest.mark.parametrize("latent", ["expand", ""])
@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("which", list(CONFIGS))
def test_mixed_batches_on_few_pages(models, which, dtype, tol, latent):
    """Unequal requests side by side in a pool so small that pages are used again; every logit equals the request's alone."""
    from aien_sovereign_core_mv_b200 import kernels as K
    d, reqs, want = models[which]
    page = PAGE[which]
    reqs, want = dict(reqs), dict(want)
    reqs.update({rid + 10: toks[: max(1, len(toks) - 3)] for rid, toks in list(reqs.items())})
    want.update({rid: want[rid - 10] for rid in reqs if rid > 10})
    longest = max(len(t) for t in reqs.values())
    pool = (3 * ((longest + page - 1) // page + 1) + 2) * page
    saved = K.LATENT_PORTIONS
    K.LATENT_PORTIONS = latent
    try:
        eng = H.engine_for(d, dtype, page, pool, max_requests=3)
        check(H.run_steps(eng, _side_by_side(reqs, random.Random(5), 3)), want, tol, f"{which} {dtype} mixed")
        state = eng.cache_state()
        assert state["check"] == "" and state["requests"] == 0
    finally:
        K.LATENT_PORTIONS = saved


def test_long_decoding_bfloat16_graphs(models):
    """Some 180 decode-only steps (captured graphs), over window, chunk and page borders."""
    d, reqs, want = models["C"]
    eng = H.engine_for(d, "bfloat16", 16, 1024)
    a, b = reqs[3], reqs[2]
    steps = [([(3, a[:15], [14]), (2, b[:4], [3])], [])]
    for i in range(len(a) - 15):
        steps.append(([(3, [a[15 + i]], [0])] + ([(2, [b[4 + i]], [0])] if 4 + i < len(b) else []), []))
    check(H.run_steps(eng, steps), want, BF16_TOL, "C bfloat16 long decoding")
    assert len(eng._graphs) > 0


def test_the_plain_forms_can_be_pinned(models):
    """A bfloat16 engine on the plain kernels gives the same logits."""
    from aien_sovereign_core_mv_b200 import kernels as K
    d, reqs, want = models["C"]
    saved = K._FORCE_ATTN, K._LATENT_IMPL
    K._FORCE_ATTN, K._LATENT_IMPL = "generic", "plain"
    try:
        eng = H.engine_for(d, "bfloat16", 16, 512)
        steps = [([(3, reqs[3][:180], list(range(180)))], [])] + [([(3, [t], [0])], []) for t in reqs[3][180:]]
        check(H.run_steps(eng, steps), want, BF16_TOL, "C on plain kernels")
    finally:
        K._FORCE_ATTN, K._LATENT_IMPL = saved


def test_greedy_generation_through_the_entry_point(models):
    from aien_sovereign_core_mv_b200.engine.generate import generate
    from aien_sovereign_core_mv_b200.sampling import SamplingParams
    d, reqs, _ = models["A"]
    cfg, tensors = load_plain(d)
    prompts = [reqs[2], reqs[3], reqs[1]]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(8):
            seq.append(int(np.argmax(pf.forward(cfg, tensors, seq)[-1])))
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
        seq.append(int(np.argmax(pf.forward(cfg, tensors, seq)[-1])))
    exe = os.path.join(H.ROOT, "bin", "aien-b200")
    out = subprocess.run([exe, "generate", "--model-dir", d, "--dtype", "float32", "--prompt-ids", ",".join(map(str, reqs[1])),
                          "--max-tokens", "5", "--temperature", "0", "--stop-token-ids", "", "--json"], capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert json.loads(out.stdout.strip().splitlines()[-1])["tokens"] == [seq[len(reqs[1]):]]
    info = subprocess.run([exe, "info", "--model-dir", d], capture_output=True, text=True, timeout=600)
    assert info.returncode == 0, info.stderr[-2000:]
    rec = json.loads(info.stdout.strip().splitlines()[-1])
    assert rec["architecture"] == "Folavik" and rec["layers"] == 3 and {"full", "window", "chunk"} <= set(rec["cache_groups"])


def test_trace_replay_from_the_command(models, tmp_path):
    d, reqs, want = models["A"]
    toks = reqs[4]
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:40], "want": [0, 39]}, {"id": 7, "tokens": reqs[1], "want": [0]}], "end": [7]},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[40:42], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[42:], "want": [len(toks) - 43]}], "end": ["x"]}]
    out = H.run_trace(d, "float32", str(tmp_path / "out"), 192, steps)
    assert sorted(out) == [0, 2]
    H.assert_close(out[0], np.stack([want[4][0], want[4][39], want[1][0]]), FP32_TOL, "trace step 0")
    H.assert_close(out[2], want[4][-1:], FP32_TOL, "trace step 2")


# ------------------------------------------------------------------ configurations drawn at random
def _random_config(rng):
    width = rng.choice([64, 72, 90, 128])
    layers = []
    for _ in range(rng.randint(1, 5)):
        kind, heads = rng.random(), rng.choice([1, 2, 3, 6])
        kv = rng.choice([k for k in (1, 2, 3, 6) if heads % k == 0])
        dim, vdim = rng.choice([8, 10, 16, 24, 40, 64, 80]), rng.choice([7, 8, 16, 24, 48, 64, 96])
        dims = 2 * rng.randint(1, dim // 2)
        size, scale, base = rng.choice([1, 2, 5, 16, 31, 64, 97, 500]), rng.choice([0.1, dim ** -0.5, 0.5]), rng.choice([10.0, 500.0, 1e5])
        factor, original = rng.choice([1.0, 2.0, 7.5, 32.0]), rng.choice([16, 100, 2048])
        if kind < 0.35:
            layer = _lat(heads, dim, vdim, rng.choice([16, 36, 64, 104, 128, 250]), scale)
        elif kind < 0.65:
            low = rng.choice([0.5, 1.0, 2.0])
            layer = _att(heads, kv, dim, vdim, size, scale, dims, base, factor, low, low * rng.choice([2.0, 4.0]), original)
        else:
            slow = rng.choice([0.5, 1.0, 4.0])
            layer = _dif(heads, kv, dim, vdim, size, rng.choice([2.0, 10.0, 50.0]), rng.choice([0.0, 0.2, 0.8]), scale, dims, base, factor, original,
                         slow * rng.choice([1.0, 8.0, 32.0]), slow)
        layers.append(_ff(layer, rng.choice([0, 24, 33, 96])))
    return {"architecture": "Folavik", "vocab": rng.choice([101, 256, 333]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])},
            "logit_scale": rng.choice([0.25, 1.0, 1.7]), "logit_softcap": rng.choice([4.0, 15.0, 40.0]), "layers": layers}


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Whole prompts, portions of changing size and three requests side by side."""
    for dtype, tol in (("float32", 2 * FP32_TOL), ("bfloat16", 2 * BF16_TOL)):
        rng = random.Random(seed)
        cfg = _random_config(rng)
        d = write_model(os.path.join(str(tmp_path), dtype), cfg, 5000 + seed, rng.choice([1.0, 2.0]), half=dtype == "bfloat16")
        c, tensors = load_plain(d)
        draw = np.random.default_rng(seed)
        reqs = {i + 1: [int(x) for x in draw.integers(0, cfg["vocab"], n)] for i, n in enumerate([rng.randint(1, 30), rng.randint(60, 100), rng.randint(130, 160)])}
        want = {r: pf.forward(c, tensors, t) for r, t in reqs.items()}
        portions = []
        for rid, t in reqs.items():
            at = 0
            while at < len(t):
                n = min(rng.choice([1, 2, 3, 17, 40, 64]), len(t) - at)
                portions.append(([(rid, t[at:at + n], list(range(n)))], [rid] if at + n == len(t) else []))
                at += n
        page = rng.choice([8, 16, 32])
        for name, steps in (("whole", [([(r, t, list(range(len(t))))], [r]) for r, t in reqs.items()]), ("portions", portions),
                            ("side by side", _side_by_side(reqs, random.Random(seed), 3))):
            eng = H.engine_for(d, dtype, page, 640)
            check(H.run_steps(eng, steps), want, tol, f"seed {seed} {dtype} {name}")
            assert eng.cache_state()["check"] == "" and eng.cache_state()["requests"] == 0
