"""The layer-stack kernels one mechanism at a time against tests/roluzen_oracle.py and tovalix_oracle.py: odd and even sizes, 32-bit and bf16, the
simple and the tensor-core forms, and inputs in which one key stands out at a window's, a page's or the kept tokens' edge."""
import math

import pytest
import torch

from tests import roluzen_oracle as O
from tests import tovalix_oracle as TO
from tests import zigipel_oracle as ZG
from tests import zikezen_oracle as ZO

pytestmark = pytest.mark.gpu
DT = [torch.float32, torch.bfloat16]


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).norm() / b.norm()).item()


def rand(*shape, dtype=torch.float32, std=1.0, seed=None):
    g = torch.Generator("cuda").manual_seed(seed if seed is not None else 7 + sum(shape))
    return (torch.randn(*shape, device="cuda", generator=g) * std).to(dtype)


def batch(parts):
    """[(slot, first position, length)] -> RaggedBatch"""
    from tunix_b200.ops.ragged import RaggedBatch
    return RaggedBatch.build([(s, p, [0] * n) for s, p, n in parts], "cuda")


# ------------------------------------------------------------------------------------------------ streams
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("S,D", [(1, 40), (2, 36), (3, 37), (4, 1024), (5, 130), (8, 64)])
def test_stream_step(S, D, dtype):
    from tunix_b200.ops import stack_kernels as SK
    n, eps, tol = 9, 1e-3, 1e-6 if dtype == torch.float32 else 5e-3
    w = {k: rand(*s, dtype=dtype, seed=i) for i, (k, s) in enumerate({"in": (S,), "out": (S,), "mix": (S, S)}.items())}
    wd = {k: v.double().cpu() for k, v in w.items()}
    embed, nw, wy, wy2 = (rand(*s, dtype=dtype, seed=20 + i) for i, s in enumerate([(50, D), (D,), (D,), (D,)]))
    y, y2 = rand(n, D, dtype=dtype, seed=30), rand(n, D, dtype=dtype, seed=31)
    toks = torch.tensor([3, 0, 49, 7, 7, 1, 2, 48, 5], device="cuda")
    d = lambda t: t.double().cpu()  # noqa: E731
    x = torch.empty(n, S, D, device="cuda")
    h = SK.stream_step(x, eps, tokens=toks, embed=embed, w_in=w["in"], norm_w=nw)
    ref = d(embed)[toks.cpu()][:, None].repeat(1, S, 1)
    assert rel(x, ref) == 0 and rel(h, O.rms(O.hyper_in(wd, "", ref), eps) * d(nw)) < tol
    total = torch.empty(n, D, device="cuda")
    h = SK.stream_step(x, eps, y=y, mix=w["mix"], w_out=w["out"], w_in=w["in"], norm_w=nw, sum_out=total)
    ref = O.hyper_out(wd, "", ref, d(y))
    assert rel(x, ref) < 1e-6 and rel(total, ref.sum(1)) < 1e-6 and rel(h, O.rms(O.hyper_in(wd, "", ref), eps) * d(nw)) < tol
    h = SK.stream_step(x, eps, y=y, y2=y2, wy=wy, wy2=wy2, mix=w["mix"], w_out=w["out"], norm_w=nw)      # no w_in: the plain sum
    ref = O.hyper_out(wd, "", ref, 0.5 * (O.rms(d(y), eps) * d(wy) + O.rms(d(y2), eps) * d(wy2)))
    assert rel(x, ref) < 1e-6 and rel(h, O.rms(ref.sum(1), eps) * d(nw)) < tol


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("F", [8, 31, 500])
def test_glu(F, dtype):
    from tunix_b200.ops import kernels as K
    from tunix_b200.ops import stack_kernels as SK
    gu = rand(17, 2 * F, dtype=dtype, std=3)
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    assert rel(SK.glu(gu, K.GLU_SILU), O.silu(gu[:, :F].double()) * gu[:, F:].double()) < tol
    wide = torch.full((17, F + 5), 7.0, dtype=dtype, device="cuda")
    got = SK.glu(gu, K.GLU_GELU, wide[:, 2:F + 2])
    assert rel(got, ZG.gelu_tanh(gu[:, :F].double()) * gu[:, F:].double()) < tol and wide[:, :2].eq(7).all() and wide[:, F + 2:].eq(7).all()


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("C1,heads,vdim", [(64, 2, 40), (6, 3, 7), (256, 1, 72)])
def test_gate_outputs(C1, heads, vdim, dtype):
    from tunix_b200.ops import stack_kernels as SK
    n, C2, eps = 11, heads * vdim, 1e-2
    attn, o, proj, w = rand(n, C1, dtype=dtype), rand(n, heads, vdim, std=0.05), rand(n, 5 + C1 + C2 + 3, dtype=dtype, std=2), rand(C2, dtype=dtype)
    a1, a2 = SK.gate_outputs(attn, o, proj, 5, 5 + C1, w, eps, heads, vdim)
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    assert rel(a1, attn.double() * torch.sigmoid(proj[:, 5:5 + C1].double())) < tol
    ref = O.rms(o.double(), eps).reshape(n, C2) * w.double() * torch.sigmoid(proj[:, 5 + C1:5 + C1 + C2].double())
    assert rel(a2, ref) < tol


@pytest.mark.parametrize("K,N", [(40, 4), (1024, 6), (4096, 16), (256, 70)])
def test_few_outputs(K, N):
    from tunix_b200.ops import stack_kernels as SK
    for n in (5, 16, 35):
        x, w = rand(n, K, dtype=torch.bfloat16), rand(N, K, dtype=torch.bfloat16, seed=1)
        assert rel(SK.few_outputs(x, w), x.double() @ w.double().T) < 1e-5


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("D,groups", [(48, 3), (36, 1), (37, 1), (1024, 4), (60, 15), (66, 6)])
def test_stream_step_norm_groups_embedding_norm_and_normed_updates(D, groups, dtype):
    from tunix_b200.ops import stack_kernels as SK
    n, eps, tol = 5, 1e-2, 1e-6 if dtype == torch.float32 else 5e-3
    one = torch.ones(1, device="cuda", dtype=dtype)
    embed, nw, ew, wy, y = (rand(*s, dtype=dtype, std=t, seed=i) for i, (s, t) in enumerate([((20, D), 0.1), ((D,), 1), ((D,), 1), ((D,), 1), ((n, D), 0.1)]))
    embed[:, : D // groups] *= 9                            # groups of unequal size
    toks = torch.tensor([3, 0, 19, 7, 7], device="cuda")
    d = lambda t: t.double().cpu()  # noqa: E731
    x = torch.empty(n, 1, D, device="cuda")
    h = SK.stream_step(x, eps, tokens=toks, embed=embed, embed_w=ew, groups=groups, w_in=one, norm_w=nw)
    ref = TO.group_norm(d(embed)[toks.cpu()], d(ew), groups, eps)
    assert rel(x[:, 0], ref) < 1e-6 and rel(h, TO.group_norm(ref, d(nw), groups, eps)) < tol
    h = SK.stream_step(x, eps, y=y, wy=wy, mix=one, w_out=one, w_in=one, norm_w=nw, groups=groups)    # the update has a plain norm
    ref = ref + TO.rms(d(y), eps) * d(wy)
    assert rel(x[:, 0], ref) < 1e-6 and rel(h, TO.group_norm(ref, d(nw), groups, eps)) < tol
    h = SK.stream_step(x, eps, y=y, mix=one, w_out=one, raw=True, groups=groups)
    ref = ref + d(y)
    assert rel(x[:, 0], ref) < 1e-6 and rel(h, ref) < tol


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("rows,F", [(3, 8), (5, 31), (64, 500)])
@pytest.mark.parametrize("p,q", [(0.5, -1.25), (-3.0, 4.0), (6.0, 0.0)])
def test_xielu(rows, F, p, q, dtype):
    from tunix_b200.ops import stack_kernels as SK
    z = rand(rows, F, dtype=dtype, std=3)
    z.view(-1)[:4] = torch.tensor([0.0, -1e-3, -60.0, 1e-3], device="cuda")
    act = torch.tensor([p, q], device="cuda", dtype=dtype)
    want = TO.xielu(z.double().cpu(), torch.tensor(p).double(), torch.tensor(q).double())
    got = SK.xielu_(z.clone(), act)
    assert rel(got, want) < (1e-6 if dtype == torch.float32 else 5e-3)
    assert torch.allclose(got.view(-1)[:4].double().cpu(), want.view(-1)[:4], rtol=1e-6 if dtype == torch.float32 else 5e-3, atol=1e-7)


@pytest.mark.parametrize("M,N,K", [(5, 64, 128), (64, 16640, 256), (130, 200, 64)])
def test_packed_product_with_xielu(M, N, K):
    from tunix_b200.ops import kernels as K_
    x, w = rand(M, K, dtype=torch.bfloat16), rand(N, K, dtype=torch.bfloat16, std=0.2, seed=1)
    act = torch.tensor([0.5, 1.25], device="cuda", dtype=torch.bfloat16)
    want = TO.xielu((x.double() @ w.double().T).cpu(), *act.double().cpu())
    assert rel(K_.gemm_packed(x, K_.PackedWeight(w), xielu=act), want) < 5e-3


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("K,N", [(40, 3), (64, 16), (256, 70)])
def test_few_outputs_with_their_activations(K, N, dtype):
    """tanh, and gelu times the token's own columns of a table; the narrow product and the two-step form."""
    from tunix_b200.ops import stack_kernels as SK
    x, w, rows = rand(5, K, dtype=dtype), rand(N, K, dtype=dtype, std=0.3, seed=1), rand(11, N + 9, dtype=dtype, seed=2)
    toks = torch.tensor([10, 0, 3, 3, 7], device="cuda")
    z = x.double().cpu() @ w.double().cpu().T
    e = rows.double().cpu()[toks.cpu(), 4:4 + N]
    kw = dict(tokens=toks, rows=rows, col=4)
    for act, want, args in ((SK.ACT_TANH, torch.tanh(z), {}), (SK.ACT_GELU_ROW, TO.gelu_tanh(z) * e, kw)):
        t = 2e-6 if dtype == torch.float32 else 5e-3
        assert rel(SK.small_act(z.float().cuda(), dtype, act, **args), want) < t
        if dtype == torch.bfloat16:
            assert rel(SK.few_outputs(x, w, act, **args), want) < t


# ------------------------------------------------------------------------------------------------ gated recurrence
def rglru_reference(m, proj, s0, past):
    """One sequence's portion: proj [T, 2 W] (y | x), state s0 [W], the inputs before it [P, W] (oldest first)."""
    d = lambda t: t.detach().double().cpu()  # noqa: E731
    W, nb = m.spec.width, m.spec.blocks
    P = past.shape[0]
    x = torch.cat([d(past), d(proj[:, W:])])
    u = O.causal_conv(x, d(m.conv_weight), d(m.conv_bias))[P:]
    if m.ra_weight.dtype == torch.bfloat16:
        u = u.to(torch.bfloat16).double()                  # the convolution's output is an activation
    ub = u.view(u.shape[0], nb, -1)
    gate = lambda w, b: torch.sigmoid(torch.einsum("boi,tbi->tbo", d(w), ub) + d(b)).reshape(-1, W)  # noqa: E731
    a = torch.exp(-8 * gate(m.ra_weight, m.ra_bias) * torch.nn.functional.softplus(d(m.lam)))
    i = gate(m.ri_weight, m.ri_bias)
    s, out = d(s0), []
    for t in range(u.shape[0]):
        s = a[t] * s + torch.sqrt(1 - a[t] ** 2) * i[t] * u[t]
        out.append(s)
    return torch.stack(out) * O.gelu_tanh(d(proj[:, :W])), s


@pytest.mark.parametrize("dtype,plain", [(torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("W,blocks,K", [(96, 3, 4), (64, 1, 1), (36, 9, 2), (512, 4, 3), (80, 2, 9), (256, 1, 4)])
def test_gated_recurrence(W, blocks, K, dtype, plain):
    """Three sequences of unequal portions, decoded steps after them, then a slot that starts over."""
    from tunix_b200.models.mixers import RGLRUMixer, RGLRUSpec
    from tunix_b200.ops import stack_kernels as SK
    m = RGLRUMixer(RGLRUSpec(W, blocks, K), 8, 1e-6, dtype, "cuda")
    for i, p in enumerate(m.parameters()):
        p.data.copy_(rand(*p.shape, dtype=dtype, std=0.4, seed=i))
    m.lam.data.copy_(rand(W, dtype=dtype, std=3) - 3)
    state = {"s": rand(4, W, seed=50), "ring": rand(4, K, W, seed=51)}         # left by earlier owners
    past = {s: torch.zeros(0, W, device="cuda") for s in range(4)}
    s_ref = {s: torch.zeros(W) for s in range(4)}
    tol = 2e-6 if dtype == torch.float32 else 4e-3
    seed = 60
    for parts in ([(2, 0, 130), (0, 0, 64), (3, 0, 1)], [(0, 64, 2), (3, 1, 65), (2, 130, 63)], [(0, 66, 1), (2, 193, 1), (3, 66, 1)],
                  [(2, 194, 1), (0, 67, 1), (3, 67, 1)], [(1, 0, 1), (0, 0, 3)]):
        for s, p, _ in parts:
            if p == 0:
                past[s], s_ref[s] = torch.zeros(0, W, device="cuda"), torch.zeros(W)
        n = sum(k for _, _, k in parts)
        seed += 1
        proj = rand(n, 2 * W, dtype=dtype, seed=seed)
        out = SK.rglru(proj, W, 0, m, batch(parts), state, plain)
        at = 0
        for s, p, k in parts:
            part = proj[at:at + k]
            want, s_ref[s] = rglru_reference(m, part, s_ref[s], past[s][-(K - 1):] if K > 1 else past[s][:0])
            assert rel(out[at:at + k], want) < tol, (parts, s)
            assert rel(state["s"][s], s_ref[s]) < (2e-6 if dtype == torch.float32 else 2e-3)
            past[s] = torch.cat([past[s], part[:, W:].float()])
            at += k


# ------------------------------------------------------------------------------------------------ matrix memory
def mlstm_reference(q, k, v, ig, fg, S, n, m):
    out = []
    dk = q.shape[-1]
    for t in range(q.shape[0]):
        new = torch.maximum(fg[t] + m, ig[t])
        a, b = torch.exp(fg[t] + m - new), torch.exp(ig[t] - new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None]
        n = a[:, None] * n + b[:, None] * k[t]
        m = new
        qt = q[t] * dk ** -0.5
        out.append(torch.einsum("hkv,hk->hv", S, qt) / (torch.maximum((n * qt).sum(-1).abs(), torch.exp(-m)) + 1e-6)[:, None])
    return torch.stack(out), S, n, m


@pytest.mark.parametrize("dtype,plain", [(torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("H,dk,dv,cap", [(2, 24, 40, 15.0), (1, 64, 64, 5.0), (3, 8, 8, 9.0), (2, 12, 33, 15.0), (1, 136, 72, 15.0),
                                         (2, 256, 32, 20.0)])
def test_matrix_memory(H, dk, dv, cap, dtype, plain):
    """Portions around the chunk length, decoded steps, a slot that starts over; gates from closed to wide open, so that both
    branches of the denominator and of the running maximum occur."""
    from tunix_b200.models.mixers import MatrixMemorySpec
    from tunix_b200.ops import stack_kernels as SK
    shapes = MatrixMemorySpec(H, dk, dv, cap).state_shapes()
    state = {k: rand(4, *s, seed=70 + i) for i, (k, s) in enumerate(shapes.items())}
    ib, fb = rand(H, dtype=dtype, std=1.0, seed=80), rand(H, dtype=dtype, std=2.0, seed=81) + 3
    d = lambda t: t.double().cpu()  # noqa: E731
    zero = lambda: (torch.zeros(H, dk, dv).double(), torch.zeros(H, dk).double(), torch.zeros(H).double())  # noqa: E731
    refs, seed = {s: zero() for s in range(4)}, 90
    tol = 3e-4 if dtype == torch.float32 or plain else 2e-2     # a denominator near zero magnifies rounding
    for parts in ([(3, 0, 64), (1, 0, 131), (0, 0, 1)], [(1, 131, 2), (0, 1, 63), (3, 64, 65)], [(3, 129, 1), (1, 133, 1), (0, 64, 1)],
                  [(2, 0, 1), (1, 134, 1), (0, 65, 1)], [(2, 1, 2), (1, 0, 5)]):
        for s, p, _ in parts:
            if p == 0:
                refs[s] = zero()
        n = sum(k for _, _, k in parts)
        seed += 1
        off = 8
        proj = rand(n, off + H * (2 * dk + dv), dtype=dtype, seed=seed)
        gates = rand(n, 2 * H, std=4.0, seed=seed + 100)
        ko, vo = off + H * dk, off + 2 * H * dk
        out = SK.mlstm(proj, off, ko, vo, gates.clone(), ib, fb, cap, batch(parts), H, dk, dv, state, plain)
        at = 0
        for s, p, k in parts:
            sl = slice(at, at + k)
            q, kk, v = d(proj[sl, off:ko]).view(k, H, dk), d(proj[sl, ko:vo]).view(k, H, dk), d(proj[sl, vo:]).view(k, H, dv)
            ig = cap * torch.tanh((d(gates[sl, :H]) + d(ib)) / cap)
            fg = torch.nn.functional.logsigmoid(cap * torch.tanh((d(gates[sl, H:]) + d(fb)) / cap))
            want, *refs[s] = mlstm_reference(q, kk, v, ig, fg, *refs[s])
            assert rel(out[sl], want) < tol, (parts, s)
            S, nn, m = refs[s]
            assert rel(state["S"][s], S) < 2e-5
            for x in range(shapes["n"][1]):
                assert rel(state["n"][s][:, x], nn) < 2e-5
                assert (state["m"][s][:, x].double().cpu() - m).abs().max() < 1e-4
            at += k


# ------------------------------------------------------------------------------------------------ learned positions, loops
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("S,D", [(1, 48), (1, 37), (3, 64), (1, 1024)])
def test_stream_step_scaled_embedding_positions_and_repetition(S, D, dtype):
    """The embedding output at the start, and once more on top of a closed sublayer, whose sum is reported without it."""
    from tunix_b200.ops import stack_kernels as SK
    eps, tol, scale = 1e-3, 1e-6 if dtype == torch.float32 else 5e-3, 2.5
    rb = batch([(1, 7, 3), (0, 0, 2), (2, 40, 1), (3, 5, 1)])
    rb.pos0[3] = -1
    n, at = 7, [7, 8, 9, 0, 1, 40, 0]
    rb.tokens.copy_(torch.tensor([3, 0, 49, 7, 7, 1, 2]))
    embed, pos, nw, wy, y = (rand(*s, dtype=dtype, seed=50 + i) for i, s in enumerate([(50, D), (41, D), (D,), (D,), (n, D)]))
    one, mix = torch.ones(S, device="cuda", dtype=dtype), torch.eye(S, device="cuda", dtype=dtype)
    d = lambda t: t.double().cpu()  # noqa: E731
    cfg, w = {"embedding": {"scale": scale}}, {"embed": d(embed), "pos": d(pos)}
    rows = torch.cat([ZO.embedding(cfg, w, rb.tokens[t:t + 1].cpu(), p) for t, p in enumerate(at)])
    kw = dict(tokens=rb.tokens, embed=embed, embed_scale=scale, pos=pos, rb=rb)
    x = torch.empty(n, S, D, device="cuda")
    h = SK.stream_step(x, eps, w_in=one, norm_w=nw, **kw)
    assert rel(x, rows[:, None].repeat(1, S, 1)) < 1e-6 and rel(h, ZO.rms(S * rows, eps) * d(nw)) < tol
    total = torch.empty(n, D, device="cuda")
    h = SK.stream_step(x, eps, y=y, wy=wy, mix=mix, w_out=one, w_in=one, norm_w=nw, sum_out=total, **kw)
    closed = rows + ZO.rms(d(y), eps) * d(wy)
    assert rel(total, S * closed) < 1e-6 and rel(x, (closed + rows)[:, None].repeat(1, S, 1)) < 1e-6
    assert rel(h, ZO.rms(S * (closed + rows), eps) * d(nw)) < tol


# ------------------------------------------------------------------------------------------------ experts
def expert_case(D, F, E, top, n, dtype, seed=0):
    h, gu, down = rand(n, D, dtype=dtype, seed=seed), rand(E, 2 * F, D, dtype=dtype, std=D ** -0.5, seed=seed + 1), \
        rand(E, D, F, dtype=dtype, std=F ** -0.5, seed=seed + 2)
    return h, gu, down, rand(n, E, seed=seed + 3, std=1.5), rand(E, dtype=dtype, seed=seed + 4, std=0.3)


def expert_reference(h, gu, down, logits, correction, top):
    h, gu, down, z = (t.double().cpu() for t in (h, gu, down, logits))
    E, F2, _ = gu.shape
    # the oracle's router reads the logits as they are
    r = ZO.route(z, torch.eye(E).double(), 0.0 if correction is None else correction.double().cpu(), top)
    out = torch.zeros_like(h)
    for e in range(E):
        t = r[:, e] > 0
        w = {"gate": gu[e, :F2 // 2], "up": gu[e, F2 // 2:], "down": down[e]}
        out[t] += r[t, e:e + 1] * ZO.glu(w, "", h[t])
    return out, r


EXPERTS = [(64, 64, 8, 2), (128, 40, 33, 4), (48, 24, 5, 5), (36, 13, 7, 3), (256, 128, 64, 8), (72, 200, 130, 6), (40, 8, 3, 1), (64, 64, 1, 1)]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("D,F,E,top", EXPERTS)
def test_experts(D, F, E, top, dtype):
    """Few and many tokens (lists of few rows per expert, row segments for the grouped product, choice by choice), experts that
    nobody takes, a correction that changes the choice and not the weights."""
    from tunix_b200.ops import stack_kernels as SK
    for n in (1, 5, 64, 128, 129, 300):
        h, gu, down, z, corr = expert_case(D, F, E, top, n, dtype, seed=n)
        for c in (corr, None):
            want, _ = expert_reference(h, gu, down, z, c, top)
            assert rel(SK.moe(h, z, c, gu, down, top, batch([(0, 0, n)])), want) < (2e-6 if dtype == torch.float32 else 1.2e-2), (n, c is None)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("n", [40, 400])
def test_one_expert_takes_every_token(n, dtype):
    """Segments of very unequal length, and scores that the choice must not follow."""
    from tunix_b200.ops import stack_kernels as SK
    D, F, E = 64, 32, 12
    h, gu, down, z, corr = expert_case(D, F, E, 2, n, dtype, seed=3)
    corr[:], z[:, 7] = 0.0, -9.0
    corr[7], corr[2] = 5.0, 3.0                                          # chosen by everyone for the correction's sake
    want, r = expert_reference(h, gu, down, z, corr, 2)
    assert ((r > 0).sum(0).tolist()) == [n if e in (2, 7) else 0 for e in range(E)] and r[:, 7].max() < 1e-2
    assert rel(SK.moe(h, z, corr, gu, down, 2, batch([(0, 0, n)])), want) < (2e-6 if dtype == torch.float32 else 1.2e-2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("D,F", [(64, 32), (36, 13)])
def test_idle_slots_choose_no_expert(D, F, dtype):
    from tunix_b200.ops import stack_kernels as SK
    h, gu, down, z, corr = expert_case(D, F, 6, 2, 5, dtype, seed=4)
    rb = batch([(s, 3, 1) for s in range(5)])
    rb.pos0[[1, 4]] = -1
    h[[1, 4]], z[[1, 4]] = float("nan"), float("nan")                    # whatever an idle row holds
    got = SK.moe(h, z, corr, gu, down, 2, rb)
    live = [0, 2, 3]
    want, _ = expert_reference(h[live], gu, down, z[live], corr, 2)
    assert rel(got[live], want) < (2e-6 if dtype == torch.float32 else 1.2e-2) and got[[1, 4]].eq(0).all()


def test_rows_of_experts_do_not_depend_on_the_company():
    """A token alone, in a decode batch and inside a long portion: the same result to rounding."""
    from tunix_b200.ops import stack_kernels as SK
    h, gu, down, z, corr = expert_case(128, 64, 16, 4, 300, torch.bfloat16, seed=8)
    full = SK.moe(h, z, corr, gu, down, 4, batch([(0, 0, 300)]))
    for at, n in ((0, 1), (17, 40), (299, 1), (100, 128)):
        part = SK.moe(h[at:at + n], z[at:at + n].contiguous(), corr, gu, down, 4, batch([(0, at, n)]))
        assert rel(part, full[at:at + n]) < 8e-3


# ------------------------------------------------------------------------------------------------ token pairs, shifted rows, gated products
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("D", [40, 37, 1024])
def test_stream_step_token_pairs_and_rows_beside_it(D, dtype):
    """The pair table's rows across portions, first tokens and idle slots; the embedding output in columns of a wider row; the tokens
    that the next portions start from."""
    from tunix_b200.ops import stack_kernels as SK
    eps, tol = 1e-3, 1e-6 if dtype == torch.float32 else 5e-3
    rb = batch([(1, 7, 3), (0, 0, 2), (2, 40, 1), (3, 5, 1), (4, 0, 1)])
    rb.pos0[3] = -1
    n, toks = 8, [3, 0, 49, 7, 7, 1, 2, 30]
    rb.tokens.copy_(torch.tensor(toks))
    rule = (13, 17, 5)
    last = torch.tensor([11, 22, 33, 44, 55, 66], device="cuda")
    embed, pairs, nw, y = (rand(*s, dtype=dtype, seed=80 + i) for i, s in enumerate([(50, D), (14, D), (D,), (n, D)]))
    one = torch.ones(1, device="cuda", dtype=dtype)
    d = lambda t: t.double().cpu()  # noqa: E731
    cfg = {"embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), rule))}}
    w = {"embed": d(embed), "bigram": d(pairs)}
    seq = lambda before, own: ZG.embedding(cfg, w, torch.tensor(before + own))[len(before):]  # noqa: E731
    want = torch.cat([seq([22], toks[:3]), seq([], toks[3:5]), seq([33], toks[5:6]), seq([], toks[6:7]), seq([], toks[7:])])
    x, row = torch.empty(n, 1, D, device="cuda"), torch.full((n, 2 * D + 3), 9.0, dtype=dtype, device="cuda")
    h = SK.stream_step(x, eps, w_in=one, norm_w=nw, tokens=rb.tokens, embed=embed, pairs=(pairs, rule, last), start_out=row[:, D:2 * D], rb=rb)
    assert rel(x[:, 0], want) < 1e-6 and rel(h, ZG.rms(want, eps) * d(nw)) < tol and rel(row[:, D:2 * D], want) < tol
    got = SK.stream_step(x, eps, y=y, mix=one, w_out=one, raw=True, out=row[:, :D], keep=last, rb=rb)
    assert got.data_ptr() == row.data_ptr() and rel(row[:, :D], want + d(y)) < tol and row[:, 2 * D:].eq(9).all()
    assert rel(row[:, D:2 * D], want) < tol and last.tolist() == [7, 49, 1, 44, 30, 66]
    h = SK.stream_step(x, eps, w_in=one, norm_w=nw)                     # nothing to close: the rows as they are
    assert rel(h, ZG.rms(want + d(y), eps) * d(nw)) < tol


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("D", [40, 37, 1000])
def test_token_shift_of_one_mix(D, dtype):
    """Portions and single tokens: the same mixes beside the rows themselves, the same carried rows."""
    from tunix_b200.ops import stack_kernels as SK
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    mu, nw = rand(1, D, dtype=dtype, seed=1), torch.ones(D, device="cuda", dtype=dtype)
    one, eps = torch.ones(1, device="cuda", dtype=dtype), 1e-3
    seq = rand(41, D, dtype=dtype, seed=2)
    h_all = (ZG.rms(seq.double().cpu(), eps)).to(dtype).double()
    want = ZG.token_shift(h_all, mu[0].double().cpu())
    carry = torch.full((3, D), 5.0, device="cuda")
    at = 0
    for k in (1, 19, 1, 2, 1, 17):
        h = h_all[at:at + k].to(dtype).cuda()
        if k == 1:
            rb = batch([(2, at, 1)])
            x = torch.empty(1, 1, D, device="cuda")
            h2, mixed = SK.stream_step(x, eps, tokens=torch.zeros(1, dtype=torch.long, device="cuda"), embed=seq[at:at + 1], w_in=one, norm_w=nw,
                                       shift=(mu, carry), both=True, rb=rb)
            assert rel(h2, h) < tol
        else:
            rb = batch([(2, at, k)])
            mixed = SK.token_shift(h, mu, carry, rb)
            SK.keep_last(h, carry, rb)
        assert mixed.shape == (1, k, D) and rel(mixed[0], want[at:at + k]) < 2 * tol
        at += k
        assert rel(carry[2], h_all[at - 1]) < tol and carry[:2].eq(5).all()
    rb = batch([(0, 4, 2), (1, 0, 1)])
    rb.pos0[1] = -1
    SK.keep_last(seq[:3].contiguous(), carry, rb)                       # an idle slot keeps what it has
    assert torch.equal(carry[0].to(dtype), seq[1]) and carry[1].eq(5).all()


@pytest.mark.parametrize("M,N,K", [(5, 64, 128), (64, 16640, 256), (130, 224, 64)])
def test_packed_gated_product_with_bias(M, N, K):
    from tunix_b200.ops import kernels as K_
    x, w, b = rand(M, K, dtype=torch.bfloat16), rand(N, K, dtype=torch.bfloat16, std=0.2, seed=1), rand(N, dtype=torch.bfloat16, seed=2)
    z = (x.double() @ w.double().T + b.double()).cpu()
    want = ZG.gelu_tanh(z[:, :N // 2]) * z[:, N // 2:]
    pw = K_.PackedWeight(w, glu=True)
    rows = torch.full((M, N // 2 + 16), 9.0, dtype=torch.bfloat16, device="cuda")
    got = K_.gemm_packed(x, pw, glu=K_.GLU_GELU, bias=b, out=rows[:, 8:8 + N // 2])
    assert rel(got, want) < 5e-3 and rows[:, :8].eq(9).all() and rows[:, 8 + N // 2:].eq(9).all()
    assert rel(K_.glu_fwd(z[:, :N // 2].bfloat16().cuda(), z[:, N // 2:].bfloat16().cuda(), K_.GLU_GELU, rows[:, 8:8 + N // 2]), want) < 1e-2
