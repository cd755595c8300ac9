"""Matrix memories with a decay per head and channel (csrc/linear_attention.cu) and what feeds them: token shift and output norm
against tests/tovalix_oracle.py and zikezen_oracle.py, in their three kernels (token by token, tensor-core blocks, decode step), with decays from
none to total, keys that stand out far away, and slots that start over."""
import pytest
import torch

from tests import tovalix_oracle as O
from tests import zikezen_oracle as ZO
from tests.test_stack_kernels_gpu import batch, rand, rel

pytestmark = pytest.mark.gpu
FORMS = [(torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)]
MODES = ["bonus", "lower", "root"]
# heads, key size, value size
SIZES = [(2, 64, 64), (3, 16, 24), (1, 128, 128), (2, 104, 136), (2, 10, 6), (1, 40, 200), (2, 136, 16), (4, 8, 8)]


def d(t):
    return t.detach().double().cpu()


class Memory:
    """One head group's parameters and a reference state per slot."""

    def __init__(self, mode, H, dk, dv, dtype, slots=4, gated=True, per_head=True, strength=(-7.0, 1.5), seed=0, tau=1.5):
        self.tau = tau
        self.mode, self.H, self.dk, self.dv, self.dtype, self.per_head = mode, H, dk, dv, dtype, per_head
        u = torch.rand(H * dk, generator=torch.Generator().manual_seed(seed))
        lo, hi = strength
        if mode == "root":
            self.c0, self.c1 = (-tau * (lo + (hi - lo) * u)).to(dtype).cuda(), None
        elif mode == "bonus":
            self.c0, self.c1 = (lo + (hi - lo) * u).to(dtype).cuda(), rand(H * dk, dtype=dtype, seed=seed + 1)
        else:
            self.c0, self.c1 = (-(lo + (hi - lo) * u)).to(dtype).cuda(), (u.flip(0) * 0.98).to(dtype).cuda()
            self.c1[::3] = 0
        self.keyed = mode != "lower"
        self.nw = rand(H * dv if per_head else dv, dtype=dtype, seed=seed + 2)
        self.gated = gated
        self.S = rand(slots, H, dk, dv, seed=seed + 3, std=5)          # left by earlier owners
        self.ref = {s: torch.zeros(H, dk, dv).double() for s in range(slots)}

    def inputs(self, n, seed):
        w = self.H * (2 * self.dk + 2 * self.dv) + 8
        x = rand(n, w, dtype=self.dtype, seed=seed)
        H, dk, dv = self.H, self.dk, self.dv
        q, k = x[:, 8:8 + H * dk], x[:, 8 + H * dk:8 + 2 * H * dk]
        v, g = x[:, 8 + 2 * H * dk:8 + 2 * H * dk + H * dv], x[:, 8 + 2 * H * dk + H * dv:]
        return q, k, v, g, rand(n, H * dk, seed=seed + 1000)

    def run(self, x, rb, eps=1e-3, plain=False, **kw):
        from tunix_b200.ops import stack_kernels as SK
        q, k, v, g, z = x
        mode = {"bonus": SK.GATES_BONUS, "lower": SK.GATES_LOWER, "root": SK.GATES_ROOT}[self.mode]
        if self.mode == "root":
            kw = dict(q_scale=0.3, tau=self.tau, **kw)
        return SK.gated_linear(mode, q, k if self.keyed else None, v, z, self.c0, self.c1, rb, self.H, self.dk, self.dv, self.S,
                               self.nw, eps, gate=g if self.gated else None, per_head=self.per_head, plain=plain, **kw)

    def decays(self, z):
        if self.mode == "root":
            return ZO.decays(z + d(self.c0), self.tau).view(-1, self.H, self.dk)
        c0, c1 = d(self.c0), d(self.c1)
        f = torch.exp(-torch.exp(z + c0)) if self.mode == "bonus" else c1 + (1 - c1) * torch.sigmoid(z + c0)
        return f.view(-1, self.H, self.dk)

    def reference(self, x, s, sl, eps=1e-3):
        q, k, v, g, z = (d(t[sl]) for t in x)
        H, dk, dv = self.H, self.dk, self.dv
        q, k, v, f = q.reshape(-1, H, dk), k.reshape(-1, H, dk), v.reshape(-1, H, dv), self.decays(z)
        u, S, out = None if self.c1 is None else d(self.c1).view(H, dk, 1), self.ref[s], []
        if self.mode == "root":
            q = q * 0.3
        if self.mode == "lower":
            q, k = O.silu(q), 1 - f
        for t in range(q.shape[0]):
            kv = k[t][:, :, None] * v[t][:, None, :]
            new = f[t][:, :, None] * S + kv
            out.append(torch.einsum("hkv,hk->hv", S + u * kv if self.mode == "bonus" else new, q[t]))
            S = new
        self.ref[s] = S
        o = O.rms(torch.stack(out), eps)
        nw = d(self.nw).view(H, dv) if self.per_head else d(self.nw)
        o = (o * nw).reshape(-1, H * dv)
        return o * O.silu(g) if self.gated else o


def tol(dtype):
    return 3e-5 if dtype == torch.float32 else 1.5e-2


PARTS = ([(2, 0, 130), (0, 0, 64), (3, 0, 1)], [(0, 64, 2), (3, 1, 65), (2, 130, 31)], [(0, 66, 1), (2, 161, 1), (3, 66, 1)],
         [(2, 162, 1), (0, 67, 1), (3, 67, 1)], [(1, 0, 17), (0, 0, 3), (2, 163, 16)], [(1, 17, 1), (0, 3, 1)])


@pytest.mark.parametrize("dtype,plain", FORMS)
@pytest.mark.parametrize("H,dk,dv", SIZES)
@pytest.mark.parametrize("mode", MODES)
def test_portions_and_steps(mode, H, dk, dv, dtype, plain):
    """Unequal portions around the block and tile lengths, down to two tokens, decoded steps after them, slots that start over."""
    m = Memory(mode, H, dk, dv, dtype, gated=mode == "bonus", per_head=mode == "bonus")
    for i, parts in enumerate(PARTS):
        for s, p, _ in parts:
            if p == 0:
                m.ref[s].zero_()
        x = m.inputs(sum(n for _, _, n in parts), 100 + i)
        out, at = m.run(x, batch(parts), plain=plain), 0
        for s, _, n in parts:
            want = m.reference(x, s, slice(at, at + n))
            assert rel(out[at:at + n], want) < tol(dtype), (parts, s)
            assert rel(m.S[s], m.ref[s]) < (5e-6 if dtype == torch.float32 else 5e-5), (parts, s)
            at += n


@pytest.mark.parametrize("gated,per_head", [(False, False), (True, False), (False, True)])
@pytest.mark.parametrize("dtype,plain", FORMS)
def test_output_norm_and_gate(dtype, plain, gated, per_head):
    """Whole heads and slices of heads, in portions and steps; an idle slot gives zeros and leaves its state alone."""
    for H, dk, dv in ((2, 16, 24), (1, 16, 136)):
        m = Memory("lower", H, dk, dv, dtype, gated=gated, per_head=per_head)
        for at, n in ((0, 40), (40, 1)):
            x = m.inputs(n, 300 + n)
            assert rel(m.run(x, batch([(1, at, n)]), plain=plain), m.reference(x, 1, slice(None))) < tol(dtype)
        rb = batch([(1, 41, 1), (0, 0, 1)])
        rb.pos0[1] = -1
        x, before = m.inputs(2, 310), m.S[0].clone()
        out = m.run(x, rb, plain=plain)
        assert rel(out[:1], m.reference(x, 1, slice(0, 1))) < tol(dtype)
        assert torch.equal(m.S[0], before) and out[1].abs().max() == 0


@pytest.mark.parametrize("strength", [(1.0, 3.0), (-12.0, -9.0), (3.0, 5.0)])
@pytest.mark.parametrize("dtype,plain", FORMS)
@pytest.mark.parametrize("dk", [48, 112])
@pytest.mark.parametrize("mode", MODES)
def test_extreme_decays(mode, dk, dtype, plain, strength):
    """Decays that empty the state within a block (the blocks' factors would overflow) and decays that hardly move it."""
    m = Memory(mode, 2, dk, 32, dtype, strength=strength, gated=False, per_head=False)
    for i, (at, n) in enumerate(((0, 200), (200, 3), (203, 1))):
        x = m.inputs(n, 400 + i)
        out = m.run(x, batch([(0, at, n)]), plain=plain)
        assert torch.isfinite(out).all() and torch.isfinite(m.S[0]).all()
        assert rel(out, m.reference(x, 0, slice(None))) < tol(dtype)
        assert rel(m.S[0], m.ref[0]) < (2e-5 if dtype == torch.float32 else 1e-4)


@pytest.mark.parametrize("dtype,plain", FORMS)
@pytest.mark.parametrize("channel", [0, 63, 70])
def test_total_decay_of_one_channel(channel, dtype, plain):
    """One token empties one channel in the middle of a block: the others go on, what follows is kept."""
    for mode in MODES:
        m = Memory(mode, 1, 72, 16, dtype, strength=(-6.0, -3.0), gated=False, per_head=False)
        if m.c1 is not None:
            m.c1[:] = 0.0
        for t in (5, 7, 8, 15):
            m.ref[0].zero_()
            x = m.inputs(40, 500 + t)
            x[4][:] = 0.0
            x[4][16 + t, channel] = 12.0 if mode == "bonus" else -130.0
            out = m.run(x, batch([(0, 0, 40)]), plain=plain)
            assert rel(out, m.reference(x, 0, slice(None))) < tol(dtype), (mode, t)
            assert rel(m.S[0], m.ref[0]) < 1e-4, (mode, t)


@pytest.mark.parametrize("dtype,plain", FORMS)
@pytest.mark.parametrize("cuts", [[700], [1] * 3 + [500] + [1] * 197, [64, 2, 300, 33, 301]])
def test_a_key_far_away(dtype, plain, cuts):
    """Slow decays and one loud token: a query hundreds of tokens later, and on every side of a portion's edge, reads its value."""
    n, far = sum(cuts), 1
    for mode in MODES:
        m = Memory(mode, 2, 32, 16, dtype, strength=(-14.0, -12.0), gated=False, per_head=False)
        if m.c1 is not None:
            m.c1[:] = 0.0
        q, k, v, g, z = m.inputs(n, 600)
        z[:] = 0.0
        if m.keyed:
            k *= 0.01
            k[far] = 30.0
        else:
            z[far] = -40.0                                  # this token replaces the whole state by its own value
            m.c0[:] = 12.0
        q[:] = 1.0
        x, at, got = (q, k, v, g, z), 0, []
        for c in cuts:
            got.append(m.run(tuple(t[at:at + c] for t in x), batch([(3, at, c)]), plain=plain))
            at += c
        got = torch.cat(got)
        assert rel(got, m.reference(x, 3, slice(None))) < tol(dtype)
        want = O.rms(d(v[far]).view(2, 16), 1e-3) * d(m.nw)
        for t in (far + 1, 63, 64, 65, 300, 503, 504, n - 1):
            assert rel(got[t], want.reshape(-1)) < 0.2, (mode, t)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,n_mix", [(40, 5), (37, 3), (256, 8), (64, 1)])
def test_token_shift(D, n_mix, dtype):
    """Portions, the first token of a sequence, the carry of a slot; the recurrence behind it replaces the carry."""
    from tunix_b200.ops import stack_kernels as SK
    mu = rand(n_mix, D, dtype=dtype, seed=1)
    parts = [(2, 0, 35), (0, 9, 2), (1, 4, 1), (3, 0, 1), (4, 7, 20)]
    carry = rand(5, D, dtype=dtype, seed=2).float()
    h = rand(59, D, dtype=dtype, seed=3)
    got, at = SK.token_shift(h, mu, carry, batch(parts)), 0
    for s, p, n in parts:
        part = d(h[at:at + n])
        first = d(carry[s]) if p > 0 else torch.zeros(D).double()
        before = torch.cat([first[None], part[:-1]])
        want = part + (before - part) * d(mu)[:, None]
        assert rel(got[:, at:at + n], want) < (1e-6 if dtype == torch.float32 else 5e-3), s
        at += n
    old = carry.clone()
    for plain in (True, False):
        carry.copy_(old)
        m = Memory("bonus", 2, 8, 8, dtype, slots=5)
        m.run(m.inputs(59, 4), batch(parts), carry=carry, h=h, plain=plain)
        for (s, _, _), last in zip(parts, (34, 36, 37, 38, 58)):
            assert torch.equal(carry[s], h[last].float())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,groups", [(40, 1), (48, 3), (37, 1), (512, 4)])
def test_token_shift_of_single_tokens(D, groups, dtype):
    """In a decode step the launch that norms the residual makes the mixes and replaces the carry; idle slots keep theirs."""
    from tunix_b200.ops import stack_kernels as SK
    one = torch.ones(1, device="cuda", dtype=dtype)
    x, y, w, mu = rand(4, 1, D), rand(4, D, dtype=dtype, seed=1), rand(D, dtype=dtype, seed=2), rand(5, D, dtype=dtype, seed=3)
    carry = rand(6, D, dtype=dtype, seed=4).float()
    old = carry.clone()
    rb = batch([(5, 3, 1), (0, 0, 1), (2, 64, 1), (1, 0, 1)])
    rb.pos0[3] = -1
    ref = d(x[:, 0]) + d(y)
    got = SK.stream_step(x, 1e-3, y=y, mix=one, w_out=one, w_in=one, norm_w=w, groups=groups, shift=(mu, carry), rb=rb)
    h = O.group_norm(ref, d(w), groups, 1e-3)
    before = torch.stack([d(old[5]), torch.zeros(D).double(), d(old[2])])
    t = 1e-6 if dtype == torch.float32 else 1e-2
    assert got.shape == (5, 4, D) and rel(got[:, :3], h[:3] + (before - h[:3]) * d(mu)[:, None]) < t
    assert rel(carry[[5, 0, 2]], h[:3]) < t and torch.equal(carry[[1, 3, 4]], old[[1, 3, 4]])


@pytest.mark.parametrize("dtype,plain", FORMS)
@pytest.mark.parametrize("tau", [1.0, 16.0, 40.0])
@pytest.mark.parametrize("cuts", [[900], [1] * 2 + [600] + [1] * 298])
def test_roots_of_sigmoids_over_many_tokens(tau, cuts, dtype, plain):
    """Decays from nearly one to small, as the root's degree sets them, over portions and hundreds of decoded tokens."""
    m = Memory("root", 2, 40, 24, dtype, tau=tau, gated=False, per_head=False)
    m.c0 = (torch.linspace(-9.0, 9.0, 80)).to(dtype).cuda()
    x, at, got = m.inputs(sum(cuts), 700), 0, []
    for c in cuts:
        got.append(m.run(tuple(t[at:at + c] for t in x), batch([(3, at, c)]), plain=plain))
        at += c
    assert rel(torch.cat(got), m.reference(x, 3, slice(None))) < tol(dtype)
    assert rel(m.S[3], m.ref[3]) < (2e-5 if dtype == torch.float32 else 1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank", [8, 16, 5, 72])
def test_gates_from_a_bottleneck_in_a_decode_step(rank, dtype):
    """The gates' product inside the step kernel against the same gates given to it."""
    from tunix_b200.ops import stack_kernels as SK
    for H, dk, dv in ((2, 64, 64), (3, 7, 9), (1, 40, 136)):
        a, b = Memory("root", H, dk, dv, dtype, seed=3), Memory("root", H, dk, dv, dtype, seed=3)
        rb = batch([(2, 5, 1), (0, 0, 1), (1, 64, 1)])
        rb.pos0[2] = -1
        q, k, v, g, _ = a.inputs(3, 800)
        for lead in (8, 3):                                # columns of a wider row, with and without 16-byte alignment
            x, w2 = rand(3, lead + rank, dtype=dtype, seed=9)[:, lead:], rand(H * dk, rank, dtype=dtype, seed=10, std=0.5)
            z = (d(x) @ d(w2).T).float().cuda()
            want = a.run((q, k, v, g, z), rb)
            got = SK.gated_linear(SK.GATES_ROOT, q, k, v, None, b.c0, None, rb, H, dk, dv, b.S, b.nw, 1e-3, gate=g, per_head=True,
                                  low_rank=(x, w2), q_scale=0.3, tau=b.tau)
            assert rel(got[:2], want[:2]) < (1e-5 if dtype == torch.float32 else 5e-3) and rel(b.S[[0, 2]], a.S[[0, 2]]) < 1e-5
            assert got[2].abs().max() == 0 and torch.equal(b.S[1], a.S[1])


@pytest.mark.parametrize("dtype,plain", FORMS)
@pytest.mark.parametrize("H,dk,dv", [(2, 16, 24), (1, 16, 136), (3, 10, 6), (2, 64, 64)])
def test_output_into_columns_of_a_row(H, dk, dv, dtype, plain):
    for lead, factor in ((8, 0.5), (3, 1.75), (16, -2.0)):
        for n in (70, 1):
            a, b = (Memory("root", H, dk, dv, dtype, seed=5) for _ in range(2))
            x, rb = a.inputs(n, 900), batch([(1, 0, n)])
            want = a.run(x, rb, plain=plain)
            rows = torch.full((n, lead + H * dv + 5), 7.0, dtype=dtype, device="cuda")
            out = b.run(x, rb, plain=plain, out=rows[:, lead:lead + H * dv], out_scale=factor)
            assert rel(out, want.double() * factor) < (1e-6 if dtype == torch.float32 else 5e-3)
            assert rows[:, :lead].eq(7).all() and rows[:, lead + H * dv:].eq(7).all()
