"""Zetavik on the GPU against the plain implementation (tests/plain_zetavik.py): every mechanism alone (its kernels, and
one-layer models that hold nothing else), then whole models through the engine's step function, its cache and states, and
the public entry points."""
import copy
import json
import os

import pytest
import torch

import plain_zetavik as P
from zetavik_configs import (CONFIGS, SEEDS, RowCheck, assert_rows, config_of, dense, lat, layer, lin, make_weights, model,
                             moe, plain_logits, random_tokens, row_error, ssm, write_model)

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
DEV = "cuda:0"


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("zetavik")
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


# ------------------------------------------------------------------ mechanisms alone: the kernels
SSD_SHAPES = [(4, 2, 32, 12, 4), (6, 3, 24, 10, 3), (1, 1, 5, 7, 1), (2, 1, 128, 64, 4), (3, 3, 64, 36, 2), (4, 1, 16, 8, 6),
              (2, 2, 200, 20, 4), (1, 1, 130, 131, 5), (2, 1, 300, 9, 2), (5, 5, 16, 600, 4), (8, 2, 256, 64, 4)]


@pytest.mark.parametrize("segment", [4, 64])
@pytest.mark.parametrize("H, G, N, P_, taps", SSD_SHAPES)
def test_state_space_kernels(H, G, N, P_, taps, segment):
    """Two sequences over five steps (prompt portions of unequal length, portions shorter than the taps' reach, one
    token each): convolution, steps, recurrence, gate and norm, and what the state row holds afterwards."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(H * N + P_)
    s = K.SsdShape(H, G, N, P_, taps)
    inner, C = s.inner, s.channels
    lens = [[41, 2, 1, 1, 9], [130, 1, 3, 1, 1]]
    total = [sum(l) for l in lens]
    proj = [torch.randn(n, s.columns + 3, generator=g) for n in total]
    wt, wb = 0.5 * torch.randn(C, taps, generator=g), 0.3 * torch.randn(C, generator=g)
    dtb, alog, D = torch.randn(H, generator=g) - 1, torch.rand(H, generator=g) * 4 - 3.5, torch.randn(H, generator=g)
    nw, eps = 1 + 0.2 * torch.randn(inner, generator=g), 1e-5
    groups = next(k for k in (3, 2, 1) if inner % k == 0)
    refs = []
    for p in proj:
        p = p.double()
        z, xbc, dt = p[:, :inner], p[:, inner:inner + C], p[:, inner + C:inner + C + H]
        xbc = P.silu(P.short_conv(xbc, wt.double(), wb.double()))
        T = p.shape[0]
        x, B, Cm = xbc[:, :inner].view(T, H, P_), xbc[:, inner:inner + G * N].view(T, G, N), xbc[:, inner + G * N:].view(T, G, N)
        step = torch.nn.functional.softplus(dt + dtb.double(), threshold=1e9)
        y, S = P.state_space_recurrence(x, B, Cm, step, torch.exp(alog.double()), D.double())
        y = y.reshape(T, inner)
        refs.append((y, S, P.gate_then_group_norm(y, z, nw.double(), groups, eps)))
    floats = s.state_floats()
    state = torch.full((3, floats), float("nan"), device=DEV)      # (rows of other slots must not be touched or read)
    slots = [2, 0]
    state[slots] = 0.0
    dev = [t.to(DEV) for t in (wt, wb, dtb, alog, D, nw)]
    done = [0, 0]
    for step in range(5):
        ns = [lens[q][step] for q in range(2)]
        rows = torch.cat([proj[q][done[q]:done[q] + ns[q]] for q in range(2)]).to(DEV)
        seq = i32([0] * ns[0] + [1] * ns[1])

        def tiles(size):
            out, off = [], 0
            for q in range(2):
                for b in range(0, ns[q], size):
                    out.append([q, off + b, min(size, ns[q] - b)])
                off += ns[q]
            return i32(out), len(out)
        if ns == [1, 1]:
            y = K.ssd_step(rows, dev[0], dev[1], dev[2], dev[3], dev[4], i32(slots), state, s)
        else:
            tl, n = tiles(16)
            xbc, steps = K.ssd_conv(rows, dev[0], dev[1], dev[2], dev[3], tl, n, seq, i32(slots), state, s)
            tl, n = tiles(segment)
            direct = n == 2
            scratch = None if direct else torch.full((K.ssd_scratch_floats(n, s),), float("nan"), device=DEV)
            y = K.ssd_segments(xbc, steps, dev[4], tl, n, direct, i32(slots), state, scratch, s)
        a = K.ssd_gate_norm(y, rows, dev[5], groups, eps, torch.float32, i32([[0, 0, ns[0]], [1, ns[0], ns[1]]]), 2, i32(slots),
                            state, s).cpu().double()
        y = y.cpu().double()
        at = 0
        for q in range(2):
            part = slice(done[q], done[q] + ns[q])
            scale = float(refs[q][0].abs().max())
            assert torch.allclose(y[at:at + ns[q]], refs[q][0][part], rtol=1e-4, atol=2e-5 * scale), (step, q)
            assert torch.allclose(a[at:at + ns[q]], refs[q][2][part], rtol=1e-3, atol=1e-4), (step, q)
            at += ns[q]
            done[q] += ns[q]
    for q in range(2):
        row = state[slots[q]].cpu()
        S = row[:H * N * P_].view(H, N, P_).double()
        assert torch.allclose(S, refs[q][1], rtol=1e-4, atol=2e-5 * float(refs[q][1].abs().max()))
        if taps > 1:
            assert torch.equal(row[H * N * P_:H * N * P_ + (taps - 1) * C].view(taps - 1, C), proj[q][-(taps - 1):, inner:inner + C])
    assert torch.isnan(state[1]).all()


@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, groups", [(96, 2), (35, 1), (4096, 1), (4096, 8), (12288, 1), (60, 5)])
def test_gate_then_group_norm(n, groups, act_dtype):
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(n + groups)
    s = K.SsdShape(1, 1, 4, n, 1)
    y, proj, w = torch.randn(7, n, generator=g), torch.randn(7, s.columns, generator=g), 1 + 0.3 * torch.randn(n, generator=g)
    state = torch.zeros(2, s.state_floats(), device=DEV)
    got = K.ssd_gate_norm(y.to(DEV), proj.to(DEV), w.to(DEV), groups, 0.03, act_dtype, i32([[0, 0, 4], [1, 4, 3]]), 2,
                          i32([1, 0]), state, s)
    want = P.gate_then_group_norm(y.double(), proj[:, :n].double(), w.double(), groups, 0.03)
    tol = 1e-2 if act_dtype == torch.bfloat16 else 1e-5
    assert torch.allclose(got.cpu().double(), want, rtol=tol, atol=tol) and not state.any()


@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, dk, r, R, Q", [(3, 24, 8, 40, 28), (1, 8, 4, 9, 33), (4, 32, 32, 96, 80), (2, 64, 64, 128, 1536)])
def test_latents_with_halves_that_turn(H, dk, r, R, Q, act_dtype):
    """Both latents normed, the shared key part turned and appended behind its latent; query heads turned, zeros behind."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(H + R)
    T, eps, base, PS = 9, 1e-5, 1000.0, 64
    proj = torch.randn(T, Q + R + r + H, generator=g)
    w, wq = 1 + 0.2 * torch.randn(R, generator=g), 1 + 0.2 * torch.randn(Q, generator=g)
    pos, seq = [100, 101, 102, 103, 0, 1, 2, 63, 64], [0, 0, 0, 0, 1, 1, 1, 1, 1]
    pages = torch.full((4, 1, PS, R + r), float("nan"), dtype=act_dtype, device=DEV)
    table = i32([[3, 1], [0, 2]])
    freq = torch.tensor([base ** (-2.0 * i / r) for i in range(r // 2)], dtype=torch.float32, device=DEV)
    rope = K.LatentRope(freq, 1.0, r, halves=True)
    cq = K.latent_norm_append(proj.to(DEV), Q, R, w.to(DEV), 0, Q, wq.to(DEV), eps, i32(pos), i32(seq), i32([0, 1]), table, pages,
                              rope=rope)
    tol = dict(rtol=2e-2, atol=2e-2) if act_dtype == torch.bfloat16 else dict(rtol=1e-5, atol=2e-5)
    assert torch.allclose(cq.cpu().double(), P.rms_norm(proj[:, :Q].double(), wq.double(), eps), **tol)
    q = torch.randn(T, H * (dk + r) + 4, generator=g)
    out = K.latent_queries(q.to(DEV), H, dk + r, dk + r + 8, rope, i32(pos), act_dtype).cpu().double().view(T, H, dk + r + 8)
    assert not out[..., dk + r:].any()
    for t in range(T):
        c = P.rms_norm(proj[t, Q:Q + R].double(), w.double(), eps)
        kr = P.rotate_halves(proj[t, Q + R:Q + R + r].view(1, 1, r).double(), base, first=pos[t])[0, 0]
        row = pages[int(table[seq[t]][pos[t] // PS]), 0, pos[t] % PS].cpu().double()
        assert torch.allclose(row, torch.cat([c, kr]), **tol), t
        one = q[t, :H * (dk + r)].view(1, H, dk + r).double()
        want = torch.cat([one[..., :dk], P.rotate_halves(one[..., dk:], base, first=pos[t])], -1)[0]
        assert torch.allclose(out[t, :, :dk + r], want, **tol), t


@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("H, dk, dv, rank, rope", [(16, 24, 20, 48, 8), (3, 16, 8, 136, 16), (40, 8, 16, 64, 4), (2, 12, 10, 21, 6)])
def test_latent_attention_turns_queries_and_gates_heads(H, dk, dv, rank, rope, halves, act_dtype):
    """The three forms for few tokens (tiles, slices, one block per head) with queries that still have to turn and a gate
    per head, against their formulas."""
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(H + rank)
    PS, lens = 64, [1, 33, 65, 130]
    T = len(lens)
    pages = (torch.randn(8, PS, rank, generator=g) * 0.7).to(act_dtype)
    table = torch.full((T, 3), -1, dtype=torch.int32)
    at, order = 0, torch.randperm(8, generator=g).tolist()
    for i, n in enumerate(lens):
        for p in range(-(-n // PS)):
            table[i, p] = order[at]
            at += 1
    wk = (torch.randn(H * dk, rank, generator=g) / rank ** 0.5).to(act_dtype)
    wv = (torch.randn(H * dv, rank, generator=g) / rank ** 0.5).to(act_dtype)
    q, gate = torch.randn(T, H * dk + 5, generator=g) * 2.0, 2 * torch.randn(T, H + 3, generator=g)
    freq = [300.0 ** (-2.0 * i / rope) for i in range(rope // 2)]
    rp = K.LatentRope(torch.tensor(freq, dtype=torch.float32, device=DEV), 1.0, rope, halves)
    want = torch.zeros(T, H * dv, dtype=torch.float64)
    for i, n in enumerate(lens):
        rows = torch.cat([pages[int(table[i, p])] for p in range(-(-n // PS))]).double()[:n]
        for h in range(H):
            qh = q[i, h * dk:(h + 1) * dk].double().view(1, 1, dk)
            part = qh[..., dk - rope:]
            if not halves:
                part = torch.cat([part[..., 0::2], part[..., 1::2]], -1)
            part = P.rotate_halves(part, 300.0, first=n - 1)
            if not halves:
                part = torch.stack([part[..., :rope // 2], part[..., rope // 2:]], -1).flatten(-2)
            qh = torch.cat([qh[..., :dk - rope], part], -1)[0, 0]
            pr = torch.softmax(rows @ (wk.double()[h * dk:(h + 1) * dk].T @ qh) * 0.3, 0)
            want[i, h * dv:(h + 1) * dv] = torch.sigmoid(gate[i, h].double()) * (wv.double()[h * dv:(h + 1) * dv] @ (pr @ rows))
    args = (q.to(DEV)[:, :H * dk], wk.to(DEV), wv.to(DEV), None, pages.to(DEV), table.to(DEV), i32(range(T)), i32(range(T)),
            i32([n - 1 for n in lens]), H, dk, dv, 0.3, 0)
    gt = gate.to(DEV)[:, :H]
    outs = {"one": K.latent_attention(*args, rope=rp, gate=gt)}
    for n_slices in (1, 5):
        scratch = lambda: (torch.empty(T * H * rank, device=DEV), torch.empty(T * H * n_slices * (rank + 2), device=DEV))
        if K.latent_attention_tiles_takes(act_dtype, H, rank):
            outs[f"tiles{n_slices}"] = K.latent_attention_tiles(*args, n_slices, *scratch(), rope=rp, gate=gt)
        if K.latent_attention_few_takes(act_dtype, rank):
            outs[f"few{n_slices}"] = K.latent_attention_few(*args, n_slices, *scratch(), rope=rp, gate=gt)
    tol = 3e-2 if act_dtype == torch.bfloat16 else 1e-4
    for name, out in outs.items():
        assert torch.allclose(out.float().cpu().double(), want, rtol=tol, atol=tol * float(want.abs().max())), name


@pytest.mark.parametrize("act_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, dv", [(3, 20), (4, 64), (1, 7)])
def test_heads_scaled_by_a_sigmoid(H, dv, act_dtype):
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(dv)
    a, z = torch.randn(11, H * dv, generator=g).to(act_dtype), 2 * torch.randn(11, H + 5, generator=g)
    for sigmoid in (True, False):
        f = torch.sigmoid(z[:, :H]) if sigmoid else z[:, :H]
        got = K.scale_heads(a.to(DEV).clone(), z.to(DEV)[:, :H], dv, sigmoid=sigmoid).cpu()
        want = (a.float().view(11, H, dv) * f[:, :, None]).reshape(11, H * dv)
        tol = 1e-2 if act_dtype == torch.bfloat16 else 1e-6
        assert torch.allclose(got.float(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("T", [3, 200])
def test_router_with_groups_and_a_factor(T):
    from dlgo_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(T)
    h, wr = torch.randn(T, 40, generator=g), 2 * torch.randn(12, 40, generator=g) / 40 ** 0.5
    for groups, keep, top, scale in ((4, 2, 3, 2.5), (1, 1, 4, 0.3), (12, 5, 5, 1.0), (3, 1, 4, 7.0)):
        r = {"experts": 12, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}
        idx, wt = P.route(h.double(), wr.double(), r)
        gi, gw, _, _ = K.moe_router(h.to(DEV), wr.to(DEV), None, 12, False, top, groups, keep, weight_scale=scale)
        assert torch.equal(gi.cpu().long(), idx)
        assert torch.allclose(gw.cpu().double(), wt, rtol=1e-5)


# --------------------------------------------------- mechanisms alone: one-layer models that hold nothing else
def one_layer(mixer, mlp=None, width=48, vocab=60, **kw):
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
@pytest.mark.parametrize("m", [ssm(4, 12, 24, 2, 4, 2), ssm(1, 1, 1, 1, 1, 1), ssm(6, 8, 40, 3, 3, 4), ssm(2, 64, 128, 1, 4, 2),
                               ssm(3, 5, 7, 3, 7, 5), ssm(8, 16, 64, 8, 2, 1), ssm(2, 24, 256, 2, 4, 3)],
                         ids=lambda m: "x".join(str(v) for v in m.values()))
def test_state_space_alone(m, dtype):
    cfg = one_layer(m)
    check_model(cfg, make_weights(cfg, m["state"] + m["vdim"]), dtype, f"state space {m}", n=290, start=130)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, dk, r, dv, Q, R", [(3, 24, 8, 20, 28, 40), (1, 8, 4, 40, 3, 9), (4, 32, 32, 64, 80, 96), (2, 64, 64, 128, 40, 128),
                                                (6, 64, 16, 72, 96, 112), (2, 16, 2, 24, 17, 18), (2, 40, 24, 64, 64, 56), (3, 96, 32, 128, 24, 64)])
def test_latent_attention_alone(H, dk, r, dv, Q, R, dtype):
    cfg = one_layer(lat(H, dk, r, dv, Q, R, 0.9 * (dk + r) ** -0.5, 3000.0))
    check_model(cfg, make_weights(cfg, dk + dv + R), dtype, f"latent attention {H}x({dk}+{r})x{dv} ranks {Q}, {R}", n=200, start=60)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, dk, dv", [(2, 32, 40), (1, 20, 12), (3, 64, 32), (1, 128, 200), (5, 7, 9)])
def test_lightning_alone(H, dk, dv, dtype):
    cfg = one_layer(lin(H, dk, dv, [0.999, 0.9, 0.5, 0.97, 1.0][:H]))
    check_model(cfg, make_weights(cfg, dk + dv), dtype, f"lightning {H}x{dk}x{dv}", n=290, start=130)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [dense(56), dense(33), moe(40, 6, 3, 1.5, (3, 2), 24), moe(24, 1, 1, 0.6), moe(16, 5, 1, 2.0, (5, 2)),
                                 moe(64, 12, 4, 1.0, (4, 2), 96), moe(20, 4, 2, 3.0, (2, 1), 1), moe(32, 8, 8, 1.0, None, 33)],
                         ids=["dense56", "dense33", "moe6top3", "moe1", "moe5top1", "moe12top4", "moe4top2", "moe8all"])
def test_feed_forwards_beside_a_mixer(mlp, dtype):
    """The feed-forward reads the norm the mixer reads, not the mixer's result."""
    cfg = one_layer(lin(1, 8, 8, [0.5]), mlp, width=64, vocab=80)
    w = make_weights(cfg, 17, mild=(dtype == "bfloat16"))
    check_model(cfg, w, dtype, "feed-forward", n=90, start=30)


@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_on_many_tokens(dtype):
    """Sizes that the tensor-core contractions of the experts take in bfloat16, on prompts of several tiles."""
    cfg = one_layer(lin(1, 8, 8, [0.5]), moe(64, 8, 2, 1.7, (4, 3), 80), width=128, vocab=200)
    w = make_weights(cfg, 18, mild=(dtype == "bfloat16"))
    tokens = random_tokens(700, cfg["vocab"], 3)
    assert_rows(run_whole(engine_of(cfg, w, dtype), tokens), plain_of(cfg, w, tokens), dtype, "experts, 700 tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_off_every_grid(dtype):
    """A width, a vocabulary and sizes that are no multiple of 8: contractions on the fp32 pipes also in bfloat16, the
    plain forms of the row kernels."""
    cfg = model(61, 101, [layer(ssm(3, 7, 11, 1, 3, 7), moe(30, 3, 2, 1.1, (3, 2), 21)), layer(lat(3, 10, 6, 14, 19, 22, 0.3, 500.0), dense(51)),
                          layer(lin(2, 9, 5, [0.9, 0.99]), None)], eps=1e-6)
    check_model(cfg, make_weights(cfg, 23, mild=(dtype == "bfloat16")), dtype, "sizes off every grid", n=130, start=55)


# -------------------------------------------------- what lies far back carries the answer: keys and states
def far_tokens(cfg, w, n, far, filler=None):
    """(a, b, f): with the query token b at position n - 1 and a at position far among fillers f, a's presence moves b's
    logits by more than a fifth of their size."""
    wd = {k: v.double() for k, v in w.items()}
    g = torch.Generator().manual_seed(1)
    for _ in range(300):
        a, b, f = torch.randint(0, cfg["vocab"], (3,), generator=g).tolist()
        f = f if filler is None else filler
        if len({a, b, f}) < 3:
            continue
        base = P.forward(cfg, wd, [f] * (n - 1) + [b])[-1:]
        moved = P.forward(cfg, wd, [f] * far + [a] + [f] * (n - 2 - far) + [b])[-1:]
        if float(row_error(moved, base)) > 0.2:
            return a, b, f
    raise AssertionError("no such tokens")


def check_far(cfg, w, dtype, n, places, filler=None):
    a, b, f = far_tokens(cfg, w, n, places[0], filler)
    eng = engine_of(cfg, w, dtype)
    for kpos in places:
        tokens = [f] * (n - 1) + [b]
        tokens[kpos] = a
        ref = plain_of(cfg, w, tokens)[-1:]
        for cuts in ([n], [130, n - 132, 1, 1], [64, 64, n - 129, 1], [n - 1, 1], [1, n - 1]):
            s = eng.take_slot()
            at = 0
            for c in cuts[:-1]:
                eng.step([s], [tokens[at:at + c]], [[]])
                at += c
            assert_rows(eng.step([s], [tokens[at:]], [[cuts[-1] - 1]]), ref, dtype, f"far token at {kpos}, portions {cuts}")
            eng.free_slot(s)
    eng.cache.book.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds(dtype):
    """Causal latent attention sees every earlier position: one key far back carries the answer."""
    cfg = one_layer(lat(2, 32, 4, 24, 40, 48, 1.0, 10000.0))
    check_far(cfg, make_weights(cfg, 77, sharpen=14.0), dtype, 401, (10, 0, 63, 64, 127, 398))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [ssm(4, 32, 32, 2, 4, 1), lin(2, 32, 32, [0.9995, 0.999])], ids=["state space", "lightning"])
def test_a_token_far_back_in_the_state(m, dtype):
    """A state with a long memory: a token hundreds of positions back moves the answer, however the tokens between
    were cut into steps and segments."""
    cfg = one_layer(m)
    w = make_weights(cfg, 78)
    filler = None
    if "dim" in m:
        # one token, the filler, whose keys are next to nothing: silu of large negative numbers
        filler = 7
        w["embed"][:, 0] = -1.0
        w["embed"][filler, 0] = 6.0
        w["l0.mix.k"][:, 0] = -2.0
    if "state" in m:
        w["l0.mix.A_log"] = torch.full_like(w["l0.mix.A_log"], -9.0)
        w["l0.mix.dt_bias"] = torch.full_like(w["l0.mix.dt_bias"], -4.0)
        # fillers add little, one token adds much: its step is scaled up through dt's rows
        w["l0.mix.in"][-4:] *= 4
    check_far(cfg, w, dtype, 301, (5, 0, 127, 128, 200), filler)


@pytest.mark.parametrize("dtype", DTYPES)
def test_positions_count(dtype):
    """The rotated part tells positions apart: the same key nearer or farther changes the answer, at every cut."""
    cfg = one_layer(lat(2, 8, 32, 24, 40, 48, 1.0, 100.0))
    w = make_weights(cfg, 79, sharpen=8.0)
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
    for name in ("P", "R"):
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
        assert info.architecture == "Zetavik" and info.layers == len(cfg["layers"]) and info.vocab_size == cfg["vocab"]
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
    """bin/trace_run on a Zetavik folder: a mixed batch, then decoding, against the plain implementation."""
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


# ------------------------------------------------- the recurrence's products on the tensor cores (bfloat16 prompts)
@pytest.mark.parametrize("segment", [64, 256])
@pytest.mark.parametrize("fixed", [False, True], ids=["step per token", "fixed decay"])
@pytest.mark.parametrize("H, G, N, P_", [(4, 2, 32, 48), (2, 1, 128, 64), (3, 3, 64, 72), (1, 1, 8, 8), (6, 2, 24, 136), (2, 2, 104, 16)])
def test_recurrence_on_tensor_cores(H, G, N, P_, fixed, segment):
    """Three sequences over two steps (a prompt, then a portion that continues it): outputs and the states left behind,
    against the recurrence on the same bfloat16 inputs, at the precision of two bfloat16 terms."""
    from dlgo_b200.csrc import kernels as K
    assert K.ssd_chunks_takes(torch.bfloat16, N, P_) and not K.ssd_chunks_takes(torch.float32, N, P_)
    if fixed:
        G = H
    g = torch.Generator().manual_seed(H * N + P_)
    lens = [[300, 65], [1, 64], [130, 3]]
    pad, width = 8, H * P_ + 2 * G * N + 16
    x0, b0, c0 = pad, pad + H * P_, pad + H * P_ + G * N
    rows = [torch.randn(sum(l), width, generator=g).to(torch.bfloat16) for l in lens]
    D = None if fixed else torch.randn(H, generator=g)
    decay = torch.tensor([0.999, 0.5, 0.97, 1.0, 0.9, 0.01][:H])
    steps = [torch.stack([torch.rand(sum(l), H, generator=g) + 0.01, -torch.rand(sum(l), H, generator=g) ** 8 * 30], -1) for l in lens]
    refs = []
    for q in range(3):
        r, T = rows[q].double(), rows[q].shape[0]
        x, B, C = r[:, x0:b0].view(T, H, P_), r[:, b0:c0].view(T, G, N), r[:, c0:c0 + G * N].view(T, G, N)
        if fixed:
            S, y = torch.zeros(H, N, P_, dtype=torch.float64), torch.zeros(T, H, P_, dtype=torch.float64)
            y = P.decayed_linear_attention(C, B, x, decay.double())
            for t in range(T):
                S = decay.double()[:, None, None] * S + B[t][:, :, None] * x[t][:, None, :]
        else:
            S, y = torch.zeros(H, N, P_, dtype=torch.float64), torch.zeros(T, H, P_, dtype=torch.float64)
            d, f = steps[q][..., 0].double(), torch.exp(steps[q][..., 1].double())
            per = H // G
            for t in range(T):
                Bt, Ct = B[t].repeat_interleave(per, 0), C[t].repeat_interleave(per, 0)
                S = f[t][:, None, None] * S + (d[t][:, None] * Bt)[:, :, None] * x[t][:, None, :]
                y[t] = torch.einsum("hnp,hn->hp", S, Ct) + D.double()[:, None] * x[t]
        refs.append((y.reshape(T, H * P_), S))
    state = torch.full((4, H * N * P_ + 4), float("nan"), device=DEV)
    slots = [3, 0, 2]
    state[slots] = 0.0
    done = [0, 0, 0]
    for step in range(2):
        ns = [l[step] for l in lens]
        cat = torch.cat([rows[q][done[q]:done[q] + ns[q]] for q in range(3)]).to(DEV)
        st = torch.cat([steps[q][done[q]:done[q] + ns[q]] for q in range(3)]).to(DEV).contiguous()
        tiles, off = [], 0
        for q in range(3):
            tiles += [[q, off + b, min(segment, ns[q] - b)] for b in range(0, ns[q], segment)]
            off += ns[q]
        direct = len(tiles) == 3
        scratch = None if direct else torch.full((len(tiles) * H * (N * P_ + 1),), float("nan"), device=DEV)
        y = K.ssd_chunks(cat, x0, b0, c0, None if fixed else st, torch.log(decay).to(DEV) if fixed else None,
                         None if fixed else D.to(DEV), i32(tiles), len(tiles), direct, i32(slots), state, scratch, H, G, N, P_)
        y, at = y.cpu().double(), 0
        for q in range(3):
            want = refs[q][0][done[q]:done[q] + ns[q]]
            err = (y[at:at + ns[q]] - want).abs().max() / want.abs().max()
            assert float(err) < 1e-4, (step, q, float(err))
            at += ns[q]
            done[q] += ns[q]
    for q in range(3):
        got = state[slots[q]][:H * N * P_].view(H, N, P_).cpu().double()
        assert float((got - refs[q][1]).abs().max() / refs[q][1].abs().max()) < 1e-4
    assert torch.isnan(state[1]).all()
