"""Bonusun on the GPU against the plain implementation (tests/plain_bonusun.py): every mechanism alone (its kernels, and
one-layer models that hold nothing else), then whole models through the engine's step function, its cache and states, and
the public entry points."""
import copy
import os

import pytest
import torch

import plain_bonusun as P
from bonusun_configs import (CONFIGS, RowCheck, assert_rows, att, config_of, dense, layer, make_weights, mem, model, moe, par,
                             plain_logits, random_tokens, rec, row_error, write_model)

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
DEV = "cuda:0"


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("bonusun")
    out = {(n, "float32"): write_model(n, str(root / n)) for n in CONFIGS}
    out.update({(n, "bfloat16"): write_model(n, str(root / (n + "_mild")), mild=True) for n in CONFIGS})
    return out


_engines = {}


def engine_for(model_dir, dtype, **kw):
    from dlgo_b200.engine.engine import Engine
    key = (model_dir, dtype, tuple(sorted(kw.items())))
    if key not in _engines:
        kw.setdefault("max_tokens", 4096)
        _engines[key] = Engine(model_dir, dtype=dtype, **kw)
    return _engines[key]


def engine_of(cfg, w, dtype, **kw):
    from dlgo_b200.engine.engine import Engine
    kw.setdefault("max_tokens", 2048)
    return Engine(spec=config_of(cfg).architecture_spec(), tensors=w, dtype=dtype, **kw)


def plain_of(cfg, w, tokens):
    return P.forward(cfg, {k: v.double() for k, v in w.items()}, tokens).float()


def run_whole(eng, tokens):
    s = eng.take_slot()
    try:
        return eng.step([s], [tokens], [list(range(len(tokens)))])
    finally:
        eng.free_slot(s)


def run_cut(eng, tokens, cuts):
    """Logits of every token when they arrive in the portions ``cuts``."""
    s = eng.take_slot()
    got, at = [], 0
    for c in cuts:
        got.append(eng.step([s], [tokens[at:at + c]], [list(range(c))]).clone())
        at += c
    assert at == len(tokens)
    eng.free_slot(s)
    return torch.cat(got)


def prefill_then_decode(eng, tokens, start):
    return run_cut(eng, tokens, [start] + [1] * (len(tokens) - start))


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def tiles_of(ns, size):
    out, off = [], 0
    for q, n in enumerate(ns):
        out += [[q, off + b, min(size, n - b)] for b in range(0, n, size)]
        off += n
    return i32(out), len(out)


def worst(got, want):
    want = want.double()
    return float((got.double().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-30))


# ------------------------------------------------------------------ mechanisms alone: the kernels
@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d, s", [(72, 2), (46, 1), (128, 4), (101, 3), (600, 8), (1024, 2), (2048, 3), (3000, 2), (4096, 1), (5000, 2)])
def test_layer_norm_over_streams(d, s, act_dtype):
    """Read, write and norm of the streams in one launch, for rows in registers and rows read again; a row's large mean
    does not cost its deviations."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(d)
    T, eps = 5, 1e-5
    X, y = torch.randn(T, s, d, generator=g) + 30.0, torch.randn(T, d, generator=g)
    w, b = 1 + 0.3 * torch.randn(d, generator=g), torch.randn(d, generator=g)
    read, write, mix = torch.randn(s, generator=g), torch.randn(s, generator=g), torch.randn(s, s, generator=g)
    new = torch.einsum("rq,trd->tqd", mix, X) + write[None, :, None] * y[:, None]
    tol = 1e-2 if act_dtype == torch.bfloat16 else 2e-4
    dev = [t.to(DEV) for t in (X, y, w, b, read, write, mix)]
    args = dict(norm_kind=K.NORM_LAYER, norm_w=dev[2], norm_b=dev[3], eps=eps, out_dtype=act_dtype)
    n = P.layer_norm(torch.einsum("r,trd->td", read.double(), X.double()), w.double(), b.double(), eps)
    assert worst(K.streams_step(dev[0], read=dev[4], **args), n) < tol
    rows = [4, 0, 4]
    n = P.layer_norm(X.double().sum(1)[rows], w.double(), b.double(), eps)
    assert worst(K.streams_step(dev[0], rows=i32(rows), **args), n) < tol
    n = P.layer_norm(X.double().sum(1), w.double(), torch.zeros(d).double(), eps)
    assert worst(K.streams_step(dev[0], **dict(args, norm_b=None)), n) < tol
    if K.streams_step_passes(K.NORM_LAYER, d):       # read on without being stored, rows in any order and twice
        out = K.streams_step(dev[0], y=dev[1], mix=dev[6], write=dev[5], clear_y=True, rows=i32(rows), keep=False, **args)
        assert worst(out, P.layer_norm(new.double().sum(1)[rows], w.double(), b.double(), eps)) < tol
        assert torch.equal(dev[0].cpu(), X) and torch.equal(dev[1].cpu(), y)
    out = K.streams_step(dev[0], y=dev[1], mix=dev[6], write=dev[5], clear_y=True, read=dev[4], **args)
    assert worst(out, P.layer_norm(torch.einsum("q,tqd->td", read.double(), new.double()), w.double(), b.double(), eps)) < tol
    assert worst(dev[0], new) < 1e-6 and not dev[1].any()


@pytest.mark.parametrize("d, s", [(72, 2), (600, 3), (1000, 1), (2048, 3), (3072, 4), (1536, 6)])
def test_layer_norm_over_streams_of_many_tokens(d, s):
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(d)
    T, eps = 700, 1e-5
    X, y = torch.randn(T, s, d, generator=g), torch.randn(T, d, generator=g)
    w, b = 1 + 0.3 * torch.randn(d, generator=g), torch.randn(d, generator=g)
    read, write, mix = torch.randn(s, generator=g), torch.randn(s, generator=g), torch.randn(s, s, generator=g)
    new = torch.einsum("rq,trd->tqd", mix, X) + write[None, :, None] * y[:, None]
    dev = [t.to(DEV) for t in (X, y, w, b, read, write, mix)]
    out = K.streams_step(dev[0], y=dev[1], mix=dev[6], write=dev[5], clear_y=True, read=dev[4], norm_kind=K.NORM_LAYER, norm_w=dev[2],
                         norm_b=dev[3], eps=eps, out_dtype=torch.float32)
    want = P.layer_norm(torch.einsum("q,tqd->td", read.double(), new.double()), w.double(), b.double(), eps)
    assert worst(out, want) < 1e-4 and worst(dev[0], new) < 1e-6 and not dev[1].any()


@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, dk, dv, hd, rot", [(6, 2, 24, 40, 40, 12), (3, 3, 64, 48, 64, 64), (2, 1, 7, 5, 8, 4), (4, 1, 96, 128, 128, 0)])
def test_head_norm_rotation_and_append(H, G, dk, dv, hd, rot, act_dtype):
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(dk)
    T, eps, PS = 7, 1e-5, 64
    n = (H + G) * dk + G * dv
    proj = torch.randn(T, n + 3, generator=g)
    wq, wk = 1 + 0.2 * torch.randn(dk, generator=g), 1 + 0.2 * torch.randn(dk, generator=g)
    pos, seq = [62, 63, 64, 0, 1, 70001, 70002], [0, 0, 0, 1, 1, 2, 2]
    cols = 70002 // PS + 1
    table = torch.full((3, cols), -1, dtype=torch.int32)
    table[0, 0], table[0, 1], table[1, 0], table[2, cols - 1] = 3, 1, 0, 2
    pages = [torch.full((4, G, PS, hd), float("nan"), dtype=act_dtype, device=DEV) for _ in range(2)]
    f = {"base": 1000.0, "dims": rot, "scaling": {"factor": 8.0}}
    freq = torch.tensor([1000.0 ** (-2.0 * i / rot) / 8.0 for i in range(rot // 2)], dtype=torch.float32, device=DEV) if rot else None
    dproj = proj.to(DEV)
    q = K.headnorm_rope_append(dproj, None, wq.to(DEV), wk.to(DEV), eps, freq, rot, i32(pos), i32(seq), i32([0, 1, 2]),
                               table.to(DEV), pages[0], pages[1], H, G, hd, False, clear=True, qk_dim=dk, v_dim=dv, v_scale=1.5)
    assert not dproj[:, :n].any() and torch.equal(dproj[:, n:].cpu(), proj[:, n:])
    q = q.cpu().double().view(T, H, hd)
    tol = dict(rtol=2e-2, atol=2e-2) if act_dtype == torch.bfloat16 else dict(rtol=1e-4, atol=4e-3 if rot else 1e-5)
    for t in range(T):
        r = proj[t].double()

        def turned(x, w):
            x = P.over_rms(x, eps) * w.double()
            return P.rotate_halves(x[None], f, first=pos[t])[0] if rot else x
        pg, at = int(table[seq[t], pos[t] // PS]), pos[t] % PS
        k, v = pages[0][pg, :, at].cpu().double(), pages[1][pg, :, at].cpu().double()
        assert torch.allclose(q[t, :, :dk], turned(r[:H * dk].view(H, dk), wq), **tol) and not q[t, :, dk:].any()
        assert torch.allclose(k[:, :dk], turned(r[H * dk:(H + G) * dk].view(G, dk), wk), **tol) and not k[:, dk:].any()
        assert torch.allclose(v[:, :dv], 1.5 * r[(H + G) * dk:n].view(G, dv), rtol=1e-2, atol=1e-6) and not v[:, dv:].any()


def attention_reference(q, rows, scale, window, sink, H, G):
    """q [H, d] at the last of ``rows`` (k [n, G, d], v [n, G, d])."""
    k, v = rows
    n = k.shape[0]
    lo = max(0, n - window) if window else 0
    out = torch.zeros(H, v.shape[-1], dtype=torch.float64)
    for h in range(H):
        s = k[lo:, h // (H // G)].double() @ q[h].double() * scale
        p = torch.softmax(torch.cat([s, sink[h].double()[None]]), 0)[:-1]
        out[h] = p @ v[lo:, h // (H // G)].double()
    return out


@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [0, 1, 33, 64, 100])
@pytest.mark.parametrize("H, G, hd", [(4, 2, 64), (6, 1, 128), (5, 5, 40), (2, 1, 16), (12, 1, 64)])
def test_sinks_in_every_attention_kernel(H, G, hd, window, act_dtype):
    """One new token per sequence through each kernel and each way its slices meet, sinks far below, near and far above
    the scores; then whole prompts."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(H * hd + window)
    PS, lens, scale = 64, [1, 2, 64, 65, 129, 400], hd ** -0.5
    T, N = len(lens), 16
    kp, vp = (torch.randn(N, G, PS, hd, generator=g).to(act_dtype) for _ in range(2))
    table = torch.full((T, 7), -1, dtype=torch.int32)
    at, order = 0, torch.randperm(N, generator=g).tolist()
    for i, n in enumerate(lens):
        for p in range(-(-n // PS)):
            table[i, p] = order[at % N]
            at += 1
    sink = torch.linspace(-30.0, 9.0, H)
    q = (2 * torch.randn(T, H * hd, generator=g)).to(act_dtype)
    want = torch.zeros(T, H * hd, dtype=torch.float64)
    for i, n in enumerate(lens):
        rows = [torch.cat([x[int(table[i, p])].transpose(0, 1) for p in range(-(-n // PS))])[:n] for x in (kp, vp)]
        want[i] = attention_reference(q[i].view(H, hd), rows, scale, window, sink, H, G).reshape(-1)
    dq, dk, dv, dt, ds = q.to(DEV), kp.to(DEV), vp.to(DEV), table.to(DEV), sink.to(DEV)
    slot, pos = i32(range(T)), i32([n - 1 for n in lens])
    outs = {}

    def out():
        return torch.full((T, H * hd), float("nan"), dtype=act_dtype, device=DEV)
    tile1 = i32([[i, i, 1] for i in range(T)])
    group = H // G
    for splits in (1, 3):
        scratch = torch.empty(K.attention_scratch_floats(T, H, hd, splits) + 1, device=DEV)
        gchunk = K.attention_tile_shape(hd, group, True)[1]
        outs[f"general {splits}"] = K.attention(dq, H * hd, T, dk, dv, dt, tile1, 1, slot, pos, out(), H, G, hd, scale, window,
                                                splits, gchunk, scratch, sink=ds)
    if K.attention_decode_takes(act_dtype, hd, PS):
        for splits, how in ((1, "one"), (3, "cluster"), (3, "counters"), (3, "second kernel"), (12, "counters")):
            scratch = torch.empty(K.attention_scratch_floats(T, H, hd, splits) + 1, device=DEV) if how in ("counters", "second kernel") else None
            counters = torch.zeros(T * G * ((group + 3) // 4), dtype=torch.int32, device=DEV) if how == "counters" else None
            outs[f"decode {splits} {how}"] = K.attention_decode(dq, H * hd, T, dk, dv, dt, slot, pos, out(), H, G, hd, scale, window,
                                                                splits, scratch, counters, sink=ds)
    if K.attention_decode_mma_takes(act_dtype, hd, PS, 1):
        for splits in (1, 4, 11):
            for split in (False, True):
                scratch = torch.empty(K.attention_scratch_floats(T, H, hd, splits) + 1, device=DEV)
                outs[f"mma {splits} {split}"] = K.attention_decode_mma(dq, H * hd, T, dk, dv, dt, slot, pos, out(), H, G, hd, scale,
                                                                       window, splits, 32, scratch, sink=ds, split=split)
    for name, o in outs.items():
        assert torch.isfinite(o).all(), name
        tol = 2e-5 if act_dtype == torch.float32 else (6e-3 if name.endswith("True") or "mma" not in name else 2e-2)
        assert worst(o, want) < tol, (name, worst(o, want))
    # prompts: the rows of one sequence are its queries
    n = 200
    qs = (2 * torch.randn(n, H * hd, generator=g)).to(act_dtype)
    rows = [torch.cat([x[int(table[5, p])].transpose(0, 1) for p in range(4)])[:n] for x in (kp, vp)]
    want = torch.stack([attention_reference(qs[i].view(H, hd), [r[:i + 1] for r in rows], scale, window, sink, H, G).reshape(-1)
                        for i in range(n)])
    pos = i32(range(n))
    qt, gchunk = K.attention_tile_shape(hd, group, False)
    tl, _ = tiles_of([n], qt)
    o = torch.empty((n, H * hd), dtype=act_dtype, device=DEV)
    K.attention(qs.to(DEV), H * hd, n, dk, dv, dt, tl, qt, i32([5]), pos, o, H, G, hd, scale, window, 1, gchunk, None, sink=ds)
    assert worst(o, want) < (2e-5 if act_dtype == torch.float32 else 6e-3)
    if K.attention_prefill_tc_takes(act_dtype, hd, PS):
        tl, _ = tiles_of([n], K.PREFILL_TC_TILE)
        for split, tol in ((True, 6e-3), (False, 2e-2)):
            o = torch.empty((n, H * hd), dtype=act_dtype, device=DEV)
            K.attention_prefill_tc(qs.to(DEV), H * hd, n, dk, dv, dt, tl, i32([5]), pos, o, H, G, hd, scale, window, sink=ds, split=split)
            assert worst(o, want) < tol, (split, worst(o, want))


@pytest.mark.parametrize("T", [3, 200])
def test_router_with_groups_scored_by_two(T):
    """Groups whose largest score is not their largest sum, choice scores that are negative, weights without correction."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(T)
    h, wr = torch.randn(T, 40, generator=g), 2 * torch.randn(13, 40, generator=g) / 40 ** 0.5
    corr = -1.2 + 0.5 * torch.randn(12, generator=g)
    for groups, keep, top, scale in ((4, 2, 3, 2.5), (1, 1, 4, 0.3), (6, 3, 5, 1.0), (3, 1, 4, 7.0), (12, 5, 5, 1.0), (2, 1, 6, 1.0)):
        r = {"experts": 12, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}
        idx, wt = P.route(h.double(), wr[:12].double(), corr.double(), r)
        for plan in (None, (12, K.MOE_FEW_ROWS)):
            gi, gw, gate, _ = K.moe_router(h.to(DEV), wr.to(DEV), corr.to(DEV), 12, True, top, groups, keep, sigmoid_scores=True,
                                           renormalize=True, weight_scale=scale, group_top=2, plan=plan)
            assert torch.equal(gi.cpu().long(), idx), (groups, keep, top)
            assert torch.allclose(gw.cpu().double(), wt, rtol=1e-5)
            assert torch.allclose(gate.cpu().double(), torch.sigmoid(h.double() @ wr[12].double()), rtol=1e-5)


def clamped(z_gate, z_up, limit, alpha=1.702, offset=1.0):
    g, u = torch.clamp(z_gate, max=limit), torch.clamp(z_up, -limit, limit)
    return g * torch.sigmoid(alpha * g) * (u + offset)


@pytest.mark.parametrize("limit, alpha, offset", [(1.0, 1.702, 1.0), (0.3, 1.0, 0.0), (7.0, 2.5, -1.0)])
def test_clamped_gated_products(limit, alpha, offset):
    """The pass of its own, the contraction's epilogue for few and many tokens, and the grouped contraction's."""
    from dlgo_b200.csrc import kernels as K
    from dlgo_b200.engine.runtime import Runtime
    from dlgo_b200.parts.feedforward import SwiGLU
    g = torch.Generator().manual_seed(3)
    glu = K.ClampedGlu(limit, alpha, offset)
    z = 2 * torch.randn(9, 96, generator=g)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        a = z.to(dt)
        assert worst(K.swiglu(a.to(DEV), glu=glu).float(), clamped(a[:, :48].double(), a[:, 48:].double(), limit, alpha, offset)) < tol
        b = a.double().view(9, 3, 2, 16)
        assert worst(K.swiglu(a.to(DEV), block=16, glu=glu).float(), clamped(b[:, :, 0], b[:, :, 1], limit, alpha, offset).reshape(9, 48)) < tol
    d, f = 128, 160
    wg, wu, wd = (torch.randn(*s, generator=g).to(torch.bfloat16) * 0.3 for s in ((f, d), (f, d), (d, f)))
    part = SwiGLU(d, f, names={"gate": "g", "up": "u", "down": "d"}, clamp=glu)
    part.load(lambda n: {"g": wg, "u": wu, "d": wd}[n].to(DEV), Runtime(DEV, "bfloat16"))
    assert part.fused
    for T in (1, 7, 30, 64, 65, 300):
        x = torch.randn(T, d, generator=g).to(torch.bfloat16)
        want = clamped(x.double() @ wg.double().T, x.double() @ wu.double().T, limit, alpha, offset)
        assert worst(part.hidden(x.to(DEV)).float(), want) < 1e-2, T
    E, T = 3, 150
    w = torch.stack([torch.stack([gg.view(f // 16, 16, d), uu.view(f // 16, 16, d)], 1).reshape(2 * f, d)
                     for gg, uu in ((wg, wu), (wu, wg), (wg * 2, wu))])
    idx = torch.randint(0, E, (T, 1), generator=g).to(torch.int32)
    x = torch.randn(T, d, generator=g).to(torch.bfloat16)
    plan = K.moe_plan(idx.to(DEV), E, K.MOE_TC_ROWS)
    h = torch.empty((T, f), dtype=torch.bfloat16, device=DEV)
    K.moe_gemm_tc(plan, K.moe_gather_rows(plan, x.to(DEV), 1), w.to(DEV), h, True, K.MOE_ACT_SWIGLU, glu=glu)
    pairs = ((wg, wu), (wu, wg), (wg * 2, wu))
    want = torch.stack([clamped(x[t].double() @ pairs[e][0].double().T, x[t].double() @ pairs[e][1].double().T, limit, alpha, offset)
                        for t, e in enumerate(idx[:, 0].tolist())])
    assert worst(h.float(), want) < 1e-2
    with pytest.raises(K.KernelError):
        K.swiglu(z.to(DEV), glu=K.ClampedGlu(0.0))


MEMORIES = [(4, 32, 12), (3, 24, 20), (1, 7, 5), (2, 128, 64), (3, 64, 72), (1, 1, 1), (2, 200, 24), (1, 300, 9), (5, 16, 600), (2, 96, 136)]


def memory_case(H, N, P_, lens, seed):
    """Inputs with calm and violent gates: heads whose maximum never leaves the decayed start, jumps, and (the last head)
    read-outs whose size is set by exp(-m)."""
    g = torch.Generator().manual_seed(seed)
    cap, total = 8.0, [sum(l) for l in lens]
    cols = H * (2 * N + P_) + 2 * H
    proj = [torch.randn(n, cols + -cols % 4, generator=g) for n in total]
    bi, bf = 2 * torch.randn(H, generator=g), 2 + 2 * torch.randn(H, generator=g)
    for p in proj:
        p[:, H * (2 * N + P_):] *= 4
        bi[-1] = -6.0
    return g, cap, proj, bi, bf


def memory_reference(p, H, N, P_, bi, bf, cap, qk_scale, dtype=None):
    T = p.shape[0]
    vkq = p[:, :H * (2 * N + P_)]
    vkq = (vkq.to(dtype) if dtype else vkq).double()
    v, k, q = vkq[:, :H * P_].view(T, H, P_), vkq[:, H * P_:H * (P_ + N)].view(T, H, N), vkq[:, H * (P_ + N):].view(T, H, N)
    z = p[:, H * (2 * N + P_):].double()
    i = cap * torch.tanh((z[:, :H] + bi.double()) / cap)
    f = -P.softplus(-cap * torch.tanh((z[:, H:2 * H] + bf.double()) / cap))
    return P.matrix_memory(q * qk_scale, k, v, i, f)


@pytest.mark.parametrize("form", ["token by token", "segments", "tensor cores"])
@pytest.mark.parametrize("H, N, P_", MEMORIES)
def test_matrix_memory_kernels(H, N, P_, form):
    """Two sequences over five steps (prompt portions of unequal length, one token each): gates and running maximum,
    recurrence, normalizer, read-out with norm and gate, and what the state row holds afterwards."""
    from dlgo_b200.csrc import kernels as K
    tc = form == "tensor cores"
    if tc and not K.ssd_chunks_takes(torch.bfloat16, N, P_):
        pytest.skip("sizes of the other kernels")
    lens = [[41, 2, 1, 1, 90], [300, 1, 3, 1, 1]]
    g, cap, proj, bi, bf = memory_case(H, N, P_, lens, H * N + P_)
    eps, out_scale, n_vkq, c = 1e-5, 1.3, H * (2 * N + P_), N ** -0.5
    if tc:
        proj = [torch.cat([p[:, :n_vkq].to(torch.bfloat16).float(), p[:, n_vkq:]], 1) for p in proj]
    gate, nw = [torch.randn(p.shape[0], H * P_, generator=g) for p in proj], 1 + 0.2 * torch.randn(H * P_, generator=g)
    refs = []
    for p, gt in zip(proj, gate):
        o, st = memory_reference(p, H, N, P_, bi, bf, cap, c)
        a = P.over_rms(o, eps).reshape(-1, H * P_) * nw.double() * torch.sigmoid(gt.double()) * out_scale
        refs.append((a, st))
    state = torch.full((3, K.mlstm_state_floats(H, N, P_)), float("nan"), device=DEV)
    slots = [2, 0]
    state[slots] = 0.0
    dbi, dbf, dnw = bi.to(DEV), bf.to(DEV), nw.to(DEV)
    done = [0, 0]
    for step in range(5):
        ns = [lens[q][step] for q in range(2)]
        rows = torch.cat([proj[q][done[q]:done[q] + ns[q]] for q in range(2)]).to(DEV)
        gt = torch.cat([gate[q][done[q]:done[q] + ns[q]] for q in range(2)]).to(DEV)
        zi, zf = rows[:, n_vkq:n_vkq + H], rows[:, n_vkq + H:n_vkq + 2 * H]
        decode = ns == [1, 1]
        if decode:
            o, nq, m = K.mlstm_step(rows, zi, zf, dbi, dbf, cap, i32(slots), state, H, N, P_)
        else:
            seqs, n = tiles_of(ns, 1 << 30)
            steps, m = K.mlstm_gates(zi, zf, dbi, dbf, cap, seqs, n, max(ns), i32(slots), state, H, N, P_, log_decay=tc)
            tl, n = tiles_of(ns, 1 << 30 if form == "token by token" else 64)
            direct = n == 2
            scratch = None if direct else torch.full((n * H * (N * P_ + 1 + N),), float("nan"), device=DEV)
            if tc:
                o, nq = K.ssd_chunks(rows[:, :n_vkq].to(torch.bfloat16).contiguous() if n_vkq % 8 == 0 else
                                     torch.nn.functional.pad(rows[:, :n_vkq].to(torch.bfloat16), (0, -n_vkq % 8)),
                                     0, H * P_, H * (P_ + N), steps, None, None, tl, n, direct, i32(slots), state, scratch, H, H, N, P_,
                                     norm_off=H * N * P_)
            else:
                o = K.ssd_segments(rows, steps, None, tl, n, direct, i32(slots), state, scratch, K.SsdShape(H, H, N, P_, 1))
                nq = K.mlstm_norm_scan(rows[:, H * P_:H * (P_ + N)], rows[:, H * (P_ + N):n_vkq], steps, seqs, 2, i32(slots), state, H, N, P_)
        a = K.mlstm_gate_norm(o, nq, m, c, gt, dnw, eps, out_scale, torch.float32, i32(slots), state, decode, H, N, P_).cpu()
        at = 0
        for q in range(2):
            want = refs[q][0][done[q]:done[q] + ns[q]]
            # (a read-out divided by its own root mean square: relative to the row's size)
            d = (a[at:at + ns[q]].double() - want).abs().max()
            assert float(d / want.abs().max()) < (2e-3 if tc else 1e-3), (step, q, float(d / want.abs().max()))
            at += ns[q]
            done[q] += ns[q]
    for q in range(2):
        row = state[slots[q]].cpu()
        S, n, m = refs[q][1]
        tol = 3e-4 if tc else 3e-5
        assert worst(row[:H * N * P_].view(H, N, P_), S) < tol
        assert worst(row[H * N * P_:H * N * (P_ + 1)].view(H, N), n) < tol
        assert torch.allclose(row[H * N * (P_ + 1):H * N * (P_ + 1) + H].double(), m, rtol=1e-4, atol=1e-4)
    assert torch.isnan(state[1]).all()


@pytest.mark.parametrize("T", [1, 7, 256, 257, 1024, 1025, 5000])
def test_running_maximum_of_long_sequences(T):
    """The parallel scan of m against its recurrence, from a state that is not zero, with stretches where m only decays
    and jumps; every cut of the sequence gives the same."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(T)
    H, cap = 3, 15.0
    z = 4 * torch.randn(T, 2 * H, generator=g)
    z[:, 0] -= 12.0
    z[T // 3:T // 2, :H] = -40.0
    z[:, H:] += 3.0
    bi, bf, m0 = torch.randn(H, generator=g), torch.randn(H, generator=g), torch.tensor([0.0, 5.0, -3.0])
    i = cap * torch.tanh((z[:, :H].double() + bi.double()) / cap)
    f = -P.softplus(-cap * torch.tanh((z[:, H:].double() + bf.double()) / cap))
    m, want = m0.double(), []
    for t in range(T):
        now = torch.maximum(f[t] + m, i[t])
        want.append((torch.exp(i[t] - now), f[t] + m - now, now))
        m = now
    want = [torch.stack(x) for x in zip(*want)]
    dz = z.to(DEV)
    off = H * 2 * 3                                # (behind S and n)
    for cuts in ([T], [T // 2, T - T // 2] if T > 1 else [T]):
        state = torch.zeros(2, K.mlstm_state_floats(H, 2, 2), device=DEV)
        state[1, off:off + H] = m0.to(DEV)
        at, got = 0, []
        for n in cuts:
            zz = dz[at:at + n]
            s, mm = K.mlstm_gates(zz[:, :H], zz[:, H:], bi.to(DEV), bf.to(DEV), cap, i32([[0, 0, n]]), 1, n, i32([1]), state, H, 2, 2, True)
            got.append((s.cpu(), mm.cpu()))
            at += n
        s, mm = (torch.cat(x) for x in zip(*got))
        assert torch.allclose(mm.double(), want[2], rtol=1e-5, atol=2e-4)
        assert torch.allclose(s[..., 0].double(), want[0], rtol=1e-3, atol=1e-6)
        assert torch.allclose(s[..., 1].double(), want[1], rtol=1e-3, atol=3e-5)
        assert torch.equal(state[1, off:off + H].cpu(), mm[-1])


UNITS = [(512, 2, 4), (400, 2, 4), (64, 4, 3), (60, 3, 4), (33, 1, 1), (50, 5, 6), (256, 2, 4), (7, 7, 2), (640, 1, 4), (24, 3, 9), (128, 4, 2)]


@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W, parts, taps", UNITS)
def test_recurrent_unit_kernels(W, parts, taps, act_dtype):
    """Three sequences over seven steps (portions of unequal length, shorter than the taps' reach, single tokens):
    convolution across steps, gates in parts, segments side by side, and what the state row holds afterwards."""
    from dlgo_b200.csrc import kernels as K
    from dlgo_b200.parts.linear_unit import RealGatedLinearUnit
    from dlgo_b200.engine.runtime import Runtime, build_context
    d = 24
    g = torch.Generator().manual_seed(W + taps)
    B = W // parts
    w = {"y_proj.weight": torch.randn(W, d, generator=g) / d ** 0.5, "y_proj.bias": 0.5 * torch.randn(W, generator=g),
         "x_proj.weight": torch.randn(W, d, generator=g) / d ** 0.5, "x_proj.bias": 0.5 * torch.randn(W, generator=g),
         "conv.weight": 0.6 * torch.randn(W, taps, generator=g), "conv.bias": 0.3 * torch.randn(W, generator=g),
         "r_gate.weight": 1.5 * torch.randn(parts, B, B, generator=g) / B ** 0.5, "r_gate.bias": torch.randn(parts, B, generator=g),
         "i_gate.weight": 1.5 * torch.randn(parts, B, B, generator=g) / B ** 0.5, "i_gate.bias": torch.randn(parts, B, generator=g),
         "decay": -4 + 3 * torch.randn(W, generator=g), "o_proj.weight": torch.randn(d, W, generator=g) / W ** 0.5}
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    rt = Runtime(DEV, "float32" if act_dtype == torch.float32 else "bfloat16")
    part = RealGatedLinearUnit(d, W, parts, taps)
    part.load(lambda n: w[n].to(DEV), rt)
    names = {"y": "y_proj.weight", "y.b": "y_proj.bias", "x": "x_proj.weight", "x.b": "x_proj.bias", "conv": "conv.weight",
             "conv.b": "conv.bias", "ra": "r_gate.weight", "ra.b": "r_gate.bias", "ri": "i_gate.weight", "ri.b": "i_gate.bias",
             "lam": "decay", "o": "o_proj.weight"}
    plain = {k: w[v].double() for k, v in names.items()}
    lens = [[70, 1, 2, 1, 1, 30, 5], [1, 2, 1, 1, 1, 200, 1], [9, 1, 64, 1, 1, 3, 90]]
    hs = [torch.randn(sum(l), d, generator=g).to(act_dtype) for l in lens]
    refs = [P.rglru(h.double(), plain, "", {"width": W, "blocks": parts, "conv": taps}, 1e-6) for h in hs]
    state = torch.full((5, part.state_need().shape[0]), float("nan"), device=DEV)
    slots = [4, 0, 2]
    state[slots] = 0.0
    done = [0] * 3
    tol = 2e-5 if act_dtype == torch.float32 else 3e-2
    for step in range(7):
        ns = [l[step] for l in lens]
        x = torch.cat([hs[q][done[q]:done[q] + ns[q]] for q in range(3)]).to(DEV)
        ctx = build_context(rt, [[0] * n for n in ns], slots, done, 1 << 20)
        y = torch.zeros(sum(ns), d, device=DEV)
        part.forward(x, y, ctx, None, state, {})
        y, at = y.cpu(), 0
        for q in range(3):
            want = refs[q][done[q]:done[q] + ns[q]]
            scale = float(refs[q].abs().max())
            assert float((y[at:at + ns[q]].double() - want).abs().max()) < tol * scale, (step, q)
            at += ns[q]
            done[q] += ns[q]
    for q in range(3):
        row = state[slots[q]].cpu()
        xs = hs[q].double() @ plain["x"].T + plain["x.b"]
        for back in range(taps):
            t = len(hs[q]) - 1 - back
            got = row[W + (t % taps) * W:W + (t % taps) * W + W].double()
            assert float((got - xs[t]).abs().max()) < (1e-4 if act_dtype == torch.float32 else 3e-2), back
    assert torch.isnan(state[[1, 3]]).all()


@pytest.mark.parametrize("segment", [3, 16, 64])
def test_segments_of_the_recurrent_unit_side_by_side(segment, monkeypatch):
    """Long sequences in short segments, a strong and a weak decay, against the recurrence."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(segment)
    W, parts, T = 200, 2, [300, 1, 77]
    s = K.RglruShape(W, parts, 4, 8.0)
    n = sum(T)
    z = torch.randn(n, parts, 2, W // parts, generator=g) * 2
    u, x, y = (torch.randn(n, W, generator=g) for _ in range(3))
    br, bi, by, bx = (torch.randn(W, generator=g) for _ in range(4))
    lam = torch.linspace(-9.0, 3.0, W)
    r = torch.sigmoid(z[:, :, 0].reshape(n, W).double() + br.double())
    i = torch.sigmoid(z[:, :, 1].reshape(n, W).double() + bi.double())
    state = torch.randn(3, s.state_floats(), generator=g)
    start = state.clone()
    dstate = state.to(DEV)
    tl, nt = tiles_of(T, segment)
    seq, pos = sum([[q] * k for q, k in enumerate(T)], []), sum([list(range(5, 5 + k)) for k in T], [])
    scratch = torch.full((nt * 3 * W,), float("nan"), device=DEV)
    dev = lambda t: t.to(DEV)
    out = K.rglru_scan(dev(z.reshape(n * parts, -1).contiguous()), dev(u), dev(br), dev(bi), dev(lam), dev(y), dev(by), dev(x), dev(bx),
                       tl, nt, nt == 3, i32(seq), i32(pos), i32([1, 2, 0]), dstate, scratch, s, torch.float32).cpu()
    at = 0
    for q, k in enumerate(T):
        sl, slot = slice(at, at + k), [1, 2, 0][q]
        S = P.gated_recurrence(u[sl].double(), r[sl], i[sl], lam.double(), start[slot, :W].double())
        want = S * P.gelu_tanh(y[sl].double() + by.double())
        assert float((out[sl].double() - want).abs().max()) < 2e-5 * float(want.abs().max()), q
        assert torch.allclose(dstate[slot, :W].cpu().double(), S[-1], rtol=1e-4, atol=1e-5)
        at += k


# --------------------------------------------------- mechanisms alone: one-layer models that hold nothing else
def one_layer(mixer, mlp=None, width=48, vocab=60, **kw):
    kw.setdefault("streams", 1)
    return model(vocab, width, [layer(copy.deepcopy(mixer), mlp)], eps=1e-6, **kw)


def check_model(cfg, w, dtype, what, n=150, start=70, seed=6):
    """Whole prompt, a prompt followed by token-by-token decoding, and portions, against the oracle."""
    tokens = random_tokens(n, cfg["vocab"], seed)
    ref = plain_of(cfg, w, tokens)
    eng = engine_of(cfg, w, dtype)
    assert_rows(run_whole(eng, tokens), ref, dtype, f"{what}: whole")
    assert_rows(prefill_then_decode(eng, tokens, start), ref, dtype, f"{what}: prefill then decode")
    assert_rows(prefill_then_decode(eng, tokens[:40], 1), ref[:40], dtype, f"{what}: decoded from the first token")
    assert_rows(run_cut(eng, tokens, [2, 3, 64, n - 71, 2]), ref, dtype, f"{what}: portions")
    return eng


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [att(6, 2, 24, 40, 0.3, 12, 5000.0, 4.0), att(1, 1, 10, 7, 0.4, 10, 100.0), att(4, 4, 64, 48, 0.125, 64, 1e5, window=64),
                               att(3, 1, 48, 64, 0.15, 16, 1e4, 8.0, window=65), att(2, 2, 96, 128, 0.1), att(5, 1, 8, 12, 0.5, window=1),
                               att(8, 2, 20, 20, 0.2, 20, 3e5, window=33)],
                         ids=lambda m: f"{m['heads']}x{m['dim']}x{m['vdim']}w{m.get('mask', {}).get('size', 0)}")
def test_attention_alone(m, dtype):
    cfg = one_layer(m)
    check_model(cfg, make_weights(cfg, m["dim"] + m["vdim"]), dtype, f"attention {m}", n=200, start=60)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [mem(3, 16, 20, 6.0), mem(1, 7, 5, 2.0), mem(2, 64, 64), mem(3, 32, 72, 4.0), mem(1, 128, 136), mem(2, 33, 12, 30.0),
                               mem(4, 48, 48, 1.0)], ids=lambda m: "x".join(str(v) for v in m.values()))
def test_memory_beside_attention(m, dtype):
    """The matrix memory beside an attention whose share is small."""
    cfg = one_layer(par(att(1, 1, 8, 8, 0.35), m, 0.1, 1.5))
    check_model(cfg, make_weights(cfg, m["dim"] + m["vdim"]), dtype, f"memory {m}", n=290, start=130)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [rec(60, 3, 4), rec(33, 1, 1), rec(256, 4, 3), rec(50, 5, 6), rec(96, 3, 2), rec(20, 20, 4)],
                         ids=lambda m: "x".join(str(v) for v in m.values()))
def test_recurrent_unit_alone(m, dtype):
    cfg = one_layer(m)
    check_model(cfg, make_weights(cfg, m["width"]), dtype, f"recurrent unit {m}", n=290, start=130)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [dense(56), dense(33), moe(40, 6, 3, 1.5, 1.5, (3, 2), (24, 0.5)), moe(24, 1, 1, 0.6), moe(16, 6, 1, 1.0, 2.0, (3, 1)),
                                 moe(64, 12, 4, 2.0, 1.0, (4, 2), (96, 1.0)), moe(20, 4, 2, 0.4, 3.0, (2, 1), (1, 9.0)), moe(32, 8, 8, 7.0, 1.0, None, (33, 2.0))],
                         ids=["dense56", "dense33", "moe6top3", "moe1", "moe6top1", "moe12top4", "moe4top2", "moe8all"])
def test_feed_forwards_behind_a_mixer(mlp, dtype):
    cfg = one_layer(rec(16, 2, 2), mlp, width=64, vocab=80, mult=1.2)
    w = make_weights(cfg, 17, mild=(dtype == "bfloat16"))
    check_model(cfg, w, dtype, "feed-forward", n=90, start=30)


@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_on_many_tokens(dtype):
    """Sizes that the tensor-core contractions of the experts take in bfloat16, on prompts of several tiles."""
    cfg = one_layer(rec(16, 2, 2), moe(64, 8, 2, 1.0, 1.7, (4, 3), (80, 0.7)), width=128, vocab=200)
    w = make_weights(cfg, 18, mild=(dtype == "bfloat16"))
    tokens = random_tokens(700, cfg["vocab"], 3)
    assert_rows(run_whole(engine_of(cfg, w, dtype), tokens), plain_of(cfg, w, tokens), dtype, "experts, 700 tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams, loop", [(1, None), (2, (0, 2, 3)), (3, (1, 2, 4)), (8, (0, 1, 2)), (5, (2, 2, 7))])
def test_streams_and_loops(streams, loop, dtype):
    """Connections and repeated spans around small layers; every pass has a cache and a state of its own."""
    cfg = model(70, 40, [layer(rec(24, 2, 3)), layer(att(2, 1, 16, 8, 0.3, 8, window=20), dense(24))], streams=streams, mult=0.7, loop=loop)
    check_model(cfg, make_weights(cfg, 40 + streams), dtype, f"{streams} streams, loop {loop}", n=120, start=50)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_off_every_grid(dtype):
    """A width, a vocabulary and sizes that are no multiple of 8: contractions on the fp32 pipes also in bfloat16, the
    plain forms of the row kernels."""
    cfg = model(61, 101, [layer(par(att(3, 1, 10, 14, 0.3, 6, 500.0), mem(3, 9, 11, 5.0), 0.9, 1.1), moe(30, 6, 2, 1.1, 1.3, (3, 2), (21, 0.6))),
                          layer(rec(51, 3, 5), dense(51))], streams=3, eps=1e-6)
    check_model(cfg, make_weights(cfg, 23, mild=(dtype == "bfloat16")), dtype, "sizes off every grid", n=130, start=55)


# -------------------------------------------------- what lies far back carries the answer: keys and states
def far_tokens(cfg, w, n, far, moves=0.15):
    """(a, b, f): with the query token b at position n - 1 and a at position far among fillers f, a's presence moves b's
    logits by more than ``moves`` of their size."""
    wd = {k: v.double() for k, v in w.items()}
    g = torch.Generator().manual_seed(1)
    for _ in range(400):
        a, b, f = torch.randint(0, cfg["vocab"], (3,), generator=g).tolist()
        if len({a, b, f}) < 3:
            continue
        base = P.forward(cfg, wd, [f] * (n - 1) + [b])[-1:]
        moved = P.forward(cfg, wd, [f] * far + [a] + [f] * (n - 2 - far) + [b])[-1:]
        if float(row_error(moved, base)) > moves:
            return a, b, f
    raise AssertionError("no such tokens")


def check_far(cfg, w, dtype, n, places, first=None):
    a, b, f = far_tokens(cfg, w, n, places[0] if first is None else first)
    eng = engine_of(cfg, w, dtype)
    for kpos in places:
        tokens = [f] * (n - 1) + [b]
        tokens[kpos] = a
        ref = plain_of(cfg, w, tokens)[-1:]
        for cuts in ([n], [130, n - 132, 1, 1], [64, 64, n - 129, 1], [n - 1, 1], [1, n - 1], [n - 20] + [1] * 20):
            s = eng.take_slot()
            at = 0
            for c in cuts[:-1]:
                eng.step([s], [tokens[at:at + c]], [[]])
                at += c
            assert_rows(eng.step([s], [tokens[at:]], [[cuts[-1] - 1]]), ref, dtype, f"far token at {kpos}, portions {cuts[:4]}")
            eng.free_slot(s)
    eng.cache.book.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [32, 64])
def test_a_far_key_among_hundreds(dim, dtype):
    """Causal attention sees every earlier position: one key far back carries the answer."""
    cfg = one_layer(att(2, 1, dim, 24, 1.0, 4, 10000.0))
    check_far(cfg, make_weights(cfg, 77, sharpen=4.0), dtype, 401, (10, 0, 63, 64, 127, 398))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window, dim", [(1, 24), (33, 24), (64, 64), (65, 24), (100, 64)])
def test_a_key_just_inside_and_just_outside_the_window(window, dim, dtype):
    """The last position of the window counts, the one before it does not: in prompts, portions and decoding, the window's
    edge inside a page and on its border."""
    cfg = one_layer(att(2, 1, dim, 24, 1.0, 4, 10000.0, window=window))
    w = make_weights(cfg, 70 + window, sharpen=4.0)
    n = 230
    edge = n - window                              # the first visible position of the last token
    a, b, f = (5, 6, 7) if window == 1 else far_tokens(cfg, w, n, edge)
    if window > 1:
        wd = {k: v.double() for k, v in w.items()}
        outside = [f] * (n - 1) + [b]
        inside = list(outside)
        inside[edge] = a
        assert float(row_error(P.forward(cfg, wd, inside)[-1:], P.forward(cfg, wd, outside)[-1:])) > 0.15
    eng = engine_of(cfg, w, dtype)
    for kpos in (edge - 1, min(edge, n - 2), min(edge + 1, n - 2)):
        tokens = [f] * (n - 1) + [b]
        tokens[kpos] = a
        ref = plain_of(cfg, w, tokens)[-1:]
        for cuts in ([n], [n - 1, 1], [100] + [1] * (n - 100), [64, 64, n - 130, 2], [n - window - 1, window + 1] if window < n - 1 else [n]):
            s, at = eng.take_slot(), 0
            for c in cuts[:-1]:
                eng.step([s], [tokens[at:at + c]], [[]])
                at += c
            assert_rows(eng.step([s], [tokens[at:]], [[cuts[-1] - 1]]), ref, dtype, f"key at {kpos} (window from {edge}), portions {cuts[:4]}")
            eng.free_slot(s)
    eng.cache.book.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_count_once_and_unscaled(dtype):
    """Sinks far above and far below the scores; the plain implementation without them is far away."""
    cfg = one_layer(att(4, 2, 24, 24, 0.3, window=40))
    w = make_weights(cfg, 80)
    w["l0.mix.sink"] = torch.tensor([4.0, -20.0, 2.0, 8.0]).to(torch.bfloat16)
    tokens = random_tokens(120, cfg["vocab"], 2)
    gone = dict(w)
    gone["l0.mix.sink"] = torch.full((4,), -1e4).to(torch.bfloat16)
    assert float(row_error(plain_of(cfg, gone, tokens), plain_of(cfg, w, tokens)).median()) > 0.05
    check_model(cfg, w, dtype, "sinks", n=120, start=3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["memory", "memory on tensor cores", "unit"])
def test_a_token_far_back_in_the_state(which, dtype):
    """A state with a long memory: a token hundreds of positions back moves the answer, however the tokens between
    were cut into steps and segments."""
    cfg = one_layer(rec(64, 4, 4) if which == "unit" else
                    par(att(1, 1, 8, 8, 0.3), mem(2, 64 if "tensor" in which else 20, 24, 12.0), 0.02, 1.5))
    w = make_weights(cfg, 78)
    if which == "unit":
        # (a gate that is nearly shut, keeping the state as it is, or open, replacing most of it)
        w["l0.mix.lam"] = torch.full_like(w["l0.mix.lam"], -2.0)
        w["l0.mix.ra"] *= 5
        w["l0.mix.ra.b"] = torch.full_like(w["l0.mix.ra.b"], -5.0)
    else:
        w["l0.mix.right.f.b"] = torch.full_like(w["l0.mix.right.f.b"], 9.0)
        w["l0.mix.right.f"] *= 0.2
        w["l0.mix.right.i"] *= 5
    check_far(cfg, w, dtype, 301, (5, 0, 127, 128, 200))


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_read_out_s_lower_bound(dtype):
    """Input gates so low that exp(-m) is the larger part of the denominator, which then sets the read-out's size before
    the norm: with a norm constant as large as the read-out it shows."""
    cfg = model(60, 48, [layer(par(att(1, 1, 8, 8, 0.3), mem(2, 16, 24, 12.0), 0.05, 2.0))], streams=1, eps=0.05)
    w = make_weights(cfg, 81)
    w["l0.mix.right.i.b"] = torch.full_like(w["l0.mix.right.i.b"], -2.0)
    tokens = random_tokens(100, 60, 5)
    up = dict(w)
    up["l0.mix.right.i.b"] = torch.full_like(w["l0.mix.right.i.b"], -1.0)
    assert float(row_error(plain_of(cfg, up, tokens), plain_of(cfg, w, tokens)).median()) > 0.02
    check_model(cfg, w, dtype, "lower bound", n=150, start=66)


@pytest.mark.parametrize("dtype", DTYPES)
def test_positions_count(dtype):
    """The rotation tells positions apart, and its scaling by how much: the same key nearer or farther changes the answer."""
    cfg = one_layer(att(2, 2, 32, 24, 1.0, 32, 100.0, 3.0))
    w = make_weights(cfg, 79, sharpen=3.0)
    tokens = random_tokens(180, cfg["vocab"], 4)
    other = tokens[:20] + tokens[21:90] + [tokens[20]] + tokens[90:]
    ref, ref2 = plain_of(cfg, w, tokens), plain_of(cfg, w, other)
    assert float(row_error(ref2[-60:], ref[-60:]).max()) > 0.02
    eng = engine_of(cfg, w, dtype)
    for t, r in ((tokens, ref), (other, ref2)):
        for cuts in ([180], [1, 179], [70, 110], [100] + [1] * 80):
            assert_rows(run_cut(eng, t, cuts), r, dtype, f"positions, portions {cuts[:3]}")


# ------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(dirs, name, dtype):
    eng = engine_for(dirs[name, dtype], dtype)
    V = CONFIGS[name]["vocab"]
    rows = RowCheck(dtype, f"{name}: whole prompts")
    for n in (1, 2, 3, 4, 5, 63, 64, 65, 127, 128, 129, 211, 300):
        tokens = random_tokens(n, V, 100 + n)
        rows.add(run_whole(eng, tokens), plain_logits(dirs[name, dtype], tokens), f"{name}: prompt of {n}")
    rows.done()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_then_token_by_token(dirs, name, graphs, dtype):
    """A short prompt, then more than two pages of decoding (with and without captured steps)."""
    eng = engine_for(dirs[name, dtype], dtype, cuda_graphs=graphs)
    tokens = random_tokens(190, CONFIGS[name]["vocab"], 7)
    ref = plain_logits(dirs[name, dtype], tokens)
    for start in (1, 5):
        assert_rows(prefill_then_decode(eng, tokens, start), ref, dtype, f"{name}: decoding from {start}")
    eng.cache.book.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions(dirs, name, dtype):
    eng = engine_for(dirs[name, dtype], dtype)
    tokens = random_tokens(300, CONFIGS[name]["vocab"], 8)
    ref = plain_logits(dirs[name, dtype], tokens)
    for cuts in ([2] * 150, [3, 61, 1, 63, 2, 170], [64, 64, 64, 108], [7, 293], [299, 1], [129, 2, 128, 41], [1, 1, 298]):
        assert_rows(run_cut(eng, tokens, cuts), ref, dtype, f"{name}: portions {cuts[:3]}...")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_batch_against_each_alone(dirs, name, dtype):
    eng = engine_for(dirs[name, dtype], dtype)
    V = CONFIGS[name]["vocab"]
    lens = [1, 140, 2, 266, 31]
    seqs = [random_tokens(n + 40, V, 50 + n) for n in lens]
    refs = [plain_logits(dirs[name, dtype], t) for t in seqs]
    slots = [eng.take_slot() for _ in seqs]
    got = eng.step(slots, [t[:n] for t, n in zip(seqs, lens)], [list(range(n)) for n in lens])
    off = 0
    rows = RowCheck(dtype, f"{name}: a mixed batch")
    for i, n in enumerate(lens):
        rows.add(got[off:off + n], refs[i][:n], f"{name}: sequence {i} of a mixed prompt batch")
        off += n
    rows.done()
    rows = RowCheck(dtype, f"{name}: decoded together")
    live = list(range(len(seqs)))
    for step in range(40):
        if step in (9, 17, 30):
            eng.free_slot(slots[live.pop(0)])
        out = eng.step([slots[i] for i in live], [[seqs[i][lens[i] + step]] for i in live])
        for j, i in enumerate(live):
            rows.add(out[j:j + 1], refs[i][lens[i] + step:lens[i] + step + 1],
                     f"{name}: sequence {i}, decoded step {step} in a batch of {len(live)}")
    rows.done()
    for i in live:
        eng.free_slot(slots[i])
    eng.cache.book.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_and_single_tokens_in_one_batch(dirs, dtype):
    """Sequences that bring a portion, two tokens and one token in the same step."""
    name = "P"
    eng = engine_for(dirs[name, dtype], dtype)
    V = CONFIGS[name]["vocab"]
    seqs = [random_tokens(160, V, 400 + i) for i in range(4)]
    refs = [plain_logits(dirs[name, dtype], t) for t in seqs]
    cuts = [[1, 70, 1, 2, 86], [150, 1, 1, 1, 7], [2, 2, 2, 2, 152], [60, 3, 1, 90, 6]]
    slots = [eng.take_slot() for _ in seqs]
    at = [0] * 4
    rows = RowCheck(dtype, "portions and single tokens in one batch")
    for step in range(5):
        ns = [c[step] for c in cuts]
        got = eng.step(slots, [seqs[i][at[i]:at[i] + ns[i]] for i in range(4)], [list(range(n)) for n in ns])
        off = 0
        for i in range(4):
            rows.add(got[off:off + ns[i]], refs[i][at[i]:at[i] + ns[i]], f"sequence {i}, step {step}")
            off += ns[i]
            at[i] += ns[i]
    rows.done()
    for s in slots:
        eng.free_slot(s)


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_slots_and_states_used_again(dirs, dtype):
    """A small cache whose pages go round several times, poisoned where nothing was written; a slot's states must be
    zero again when the slot is taken anew."""
    name = "P"
    eng = engine_for(dirs[name, dtype], dtype, max_tokens=512, max_slots=3)
    eng.cache.poison()
    V = CONFIGS[name]["vocab"]
    rows = RowCheck(dtype, "pages and slots used again")
    for r in range(5):
        lens = [150 + 7 * r, 90 - r, 60 + r]
        seqs = [random_tokens(n, V, 300 + 10 * r + i) for i, n in enumerate(lens)]
        slots = [eng.take_slot() for _ in seqs]
        got = eng.step(slots, seqs, [[0, 1, n - 2, n - 1] for n in lens])
        assert torch.isfinite(got).all()                          # nothing unwritten reached a result
        for i, n in enumerate(lens):
            ref = plain_logits(dirs[name, dtype], seqs[i])
            rows.add(got[4 * i:4 * i + 4], ref[[0, 1, n - 2, n - 1]], f"round {r}, sequence {i}")
        for s in (slots[1], slots[0], slots[2]):
            eng.free_slot(s)
    rows.done()
    eng.cache.book.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dirs, dtype):
    name = "Q"
    eng = engine_for(dirs[name, dtype], dtype)
    tokens = random_tokens(620, CONFIGS[name]["vocab"], 9)
    ref = plain_logits(dirs[name, dtype], tokens)
    s = eng.take_slot()
    eng.step([s], [tokens[:20]], [[]])
    rows = RowCheck(dtype, "long decoding")
    for p in range(20, len(tokens)):
        out = eng.step([s], [tokens[p:p + 1]])
        if p % 17 == 0 or p >= len(tokens) - 8:
            rows.add(out.clone(), ref[p:p + 1], f"decoded position {p}")
    rows.done()
    eng.free_slot(s)


def test_greedy_generation_through_the_entry_point(dirs):
    import dlgo_b200
    for name in ("P", "Q"):
        dtype = "float32"
        llm = dlgo_b200.load_llm(dirs[name, dtype], dtype=dtype, max_tokens=2048)
        cfg, w = P.read_model(dirs[name, dtype], torch.float64)
        prompts = [random_tokens(n, cfg["vocab"], 70 + n) for n in (1, 9, 70)]
        got = llm.generate(prompts, max_tokens=12, greedy=True, ignore_eos=True)
        for p, g in zip(prompts, got):
            want = P.greedy_generate(cfg, w, p, 12)
            if g != want:                      # only a near tie may differ
                k = next(i for i in range(12) if g[i] != want[i])
                lg = P.forward(cfg, w, p + want[:k])[-1]
                assert float(lg[want[k]] - lg[g[k]]) < 1e-4 * float(lg.abs().max()), (name, g, want)
        info = llm.model_info()
        assert info.architecture == "Bonusun" and info.layers == len(P.run_order(cfg)) and info.vocab_size == cfg["vocab"]
        out = llm.generate(prompts[:2], max_tokens=5, temperature=0.8, top_k=20, seed=3, ignore_eos=True)
        assert all(len(o) == 5 and all(0 <= t < cfg["vocab"] for t in o) for o in out)


def test_command_line(dirs):
    """Greedy generation from the command line gives the entry point's tokens."""
    import subprocess
    import sys
    import dlgo_b200
    d = dirs["P", "float32"]
    prompt = random_tokens(9, CONFIGS["P"]["vocab"], 5)
    r = subprocess.run([sys.executable, "-m", "dlgo_b200", "generate", d, "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "6",
                        "--greedy", "--dtype", "float32", "--ctx", "256"], capture_output=True, text=True, timeout=600,
                       cwd=os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    assert r.returncode == 0, r.stderr[-2000:]
    want = dlgo_b200.load_llm(d, dtype="float32", max_tokens=512).generate(prompt, max_tokens=6, greedy=True)
    assert [int(t) for t in r.stdout.split()] == want


def test_trace_replay_command(dirs, tmp_path):
    """bin/trace_run on a Bonusun folder: a mixed batch, then decoding, against the plain implementation."""
    from traces import run_program
    name, dtype = "P", "float32"
    V = CONFIGS[name]["vocab"]
    a, b = random_tokens(30, V, 1), random_tokens(75, V, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:28], "want": [0, 27]}, {"id": "b", "tokens": b[:70], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[28:29], "want": [0]}, {"id": "b", "tokens": b[70:71], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[29:30], "want": []}, {"id": "b", "tokens": b[71:72], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[72:73], "want": [0]}], "end": ["b"]}]
    outs = run_program(dirs[name, dtype], dtype, steps, str(tmp_path / "out"), 256, V)
    ra, rb = plain_logits(dirs[name, dtype], a), plain_logits(dirs[name, dtype], b)
    want = {0: torch.stack([ra[0], ra[27]]), 1: torch.stack([ra[28], rb[70]]), 2: rb[71:72], 3: rb[72:73]}
    for i, ref in want.items():
        assert_rows(outs[i], ref, "float32", f"step {i}")
