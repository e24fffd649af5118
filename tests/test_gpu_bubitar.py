"""Bubitar models on the GPU: every kernel against a plain fp64 statement of its operation, the model in bf16 and in 32-bit
against the plain model, decoding steps, portions, batches, graph-replayed generation."""

import pytest
import torch

import bubitar_oracle as oracle
from bubitar_cases import CONFIGS
from hybrid_cases import build, rel, run_portions, tokens

pytestmark = pytest.mark.gpu

DT = [torch.float32, torch.bfloat16]


def agrees(got, want, dtype):
    """32-bit: every position. bf16, at widths of 36 to 96: rounding alone leaves a median of 1 to 2 percent, and single
    positions beyond 20 where a norm divides a nearly cancelled sum (a PyTorch run in bf16 has the same ones)."""
    if dtype == torch.float32:
        return rel(got, want) < 5e-5
    got, want = got.double().cpu(), want.double()
    d, w = (t - t.mean(-1, keepdim=True) for t in (got - want, want))
    e = d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
    return float(e.median()) < 3e-2 and float(e.quantile(0.9)) < 7e-2 and float(e.max()) < 0.5


def dev(t, dtype=None):
    return t.to("cuda") if dtype is None else t.to(device="cuda", dtype=dtype)


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g)


def rounded(t, dtype):
    return t.to(dtype).double()


def close(got, want, dtype, scale=1.0):
    got, want = got.double().cpu(), want.double()
    tol = (2e-5 if dtype == torch.float32 else 1.2e-2) * scale
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))
    assert err < tol, err


def pad8(n):
    return -(-n // 8) * 8


# ---- rows --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("rows,width", [(1, 37), (5, 96), (7, 768), (33, 2048), (9, 3072), (3, 8192), (2, 12000)])
def test_sum_and_norm(dtype, rows, width):
    from triune_b200.ops import hybrid as hops

    r = gen(width)
    x, y, b, w1, w2 = r(rows, width) * 2, r(rows, width) + 0.7, r(width), r(width), r(width)
    for post, pre, bias in (("rms", "rms", b), ("layer", "rms", None), ("rms", "layer", b), ("rms", "rows", None), ("rms", None, b)):
        yb = rounded(y, dtype) + (0 if bias is None else bias.double())
        norm = lambda v, w, k, e: oracle.rms_norm(v - v.mean(-1, keepdim=True) if k == "layer" else v, w.double(), e)
        want = x.double() + norm(yb, w1, post, 1e-3)
        xd = dev(x).clone()
        h = hops.add_norm(xd, dev(y, dtype), None if bias is None else dev(bias), (dev(w1), 1e-3, post),
                          (dev(w2), 1e-5, pre) if pre in ("rms", "layer") else pre, dtype)
        close(xd, want, torch.float32)
        if pre is None:
            assert h is None
        else:
            close(h, want if pre == "rows" else norm(want, w2, pre, 1e-5), dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("rows,width,F", [(9, 40, 24), (70, 64, 96), (600, 1024, 256), (3, 30, 17)])
def test_clamped_feed_forward(dtype, rows, width, F):
    """With biases; the scale of the inputs puts values beyond both limits. The large case runs on CTA pairs."""
    from triune_b200.ops import hybrid as hops

    r = gen(F)
    h, gu, b = r(rows, width), r(2 * F, width) * 3 * width ** -0.5, r(2 * F)
    pre = rounded(h, dtype) @ rounded(gu, dtype).T + b.double()
    g, u = torch.clamp(pre[:, :F], max=1.25), torch.clamp(pre[:, F:], -1.25, 1.25)
    assert (pre[:, :F] > 1.25).any() and (pre[:, F:] < -1.25).any()
    want = g * oracle.sigmoid(1.702 * g) * (u + 1)
    close(hops.gated_mlp_hidden(dev(h, dtype), dev(gu, dtype), "clamped", dev(b), 1.25, 1.702), want, dtype, 2)
    close(hops.gated_mlp_hidden(dev(h, dtype), dev(gu, dtype), "silu", dev(b)), oracle.silu(pre[:, :F]) * pre[:, F:], dtype, 2)


@pytest.mark.parametrize("dtype", DT)
def test_token_side_rows(dtype):
    from triune_b200.ops import hybrid as hops

    r = gen(4)
    gate, table, ids = r(50, 6) * 2, r(20, 18), torch.randint(0, 20, (50,))
    want = oracle.gelu_tanh(rounded(gate, dtype)) * rounded(table, dtype)[ids][:, 6:12]
    close(hops.token_side_hidden(dev(gate, dtype), dev(table, dtype), dev(ids), 6), want, dtype)


@pytest.mark.parametrize("dims,scaling", [(16, None), (64, {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 1.0})])
def test_rotation_rows_near_and_far(dims, scaling):
    from triune_b200.models.rotary import rotary_frequencies
    from triune_b200.ops import hybrid as hops

    f, amp = rotary_frequencies(dims, 1e4, scaling)
    for pos in (0, 5, 3000, 1000000):
        want = (torch.arange(pos, pos + 9, dtype=torch.float64)[:, None] * f)
        want = torch.cat((want.cos(), want.sin()), 1) * amp
        for p in (pos, torch.tensor([pos], device="cuda")):
            assert (hops.rotation_rows(dev(f), amp, p, 9).double().cpu() - want).abs().max() < 1e-6


# ---- retention ---------------------------------------------------------------------------------------------------
def retention_case(seed, B, T, H, D, E, rot, dtype):
    r = gen(seed)
    q, k, v = r(B, T, H, D), r(B, T, H, D), r(B, T, H, E)
    decay = torch.tensor([[0.125, 0.9, 0.95, 0.9975, 1.0][i % 5] for i in range(H)], dtype=torch.float64)
    spec = {"dims": rot, "base": 1e3}
    turn = lambda x: oracle.rotate_halves(rounded(x, dtype), torch.arange(T), spec)
    want = [oracle.retention_scan(turn(q[b]), turn(k[b]) * D ** -0.5, rounded(v[b], dtype), decay) for b in range(B)]
    freqs = torch.tensor(oracle.rotation_table(spec)[0], dtype=torch.float64)
    return q, k, v, decay, freqs, torch.stack([y for y, _ in want]), torch.stack([S for _, S in want])


def run_retention(q, k, v, decay, freqs, dtype, cut):
    from triune_b200.ops import hybrid as hops

    B, T, H, D = q.shape
    E = v.shape[-1]
    qd, kd, vd = (dev(t, dtype) for t in (q, k, v))
    st, at, outs = torch.zeros(B, H, D, E, device="cuda"), 0, []
    for n in cut:
        s = slice(at, at + n)
        out = torch.empty(B * n, pad8(H * E), device="cuda", dtype=dtype)
        hops.retention(qd[:, s].reshape(B * n, -1), kd[:, s].reshape(B * n, -1), vd[:, s].reshape(B * n, -1),
                       hops.rotation_rows(dev(freqs), 1.0, at, n), dev(decay), st, out, B, n)
        outs.append(out[:, : H * E].reshape(B, n, H, E))
        at += n
    hops.check_status(torch.device("cuda", 0))
    return torch.cat(outs, 1), st


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("B,H,D,E,rot", [(1, 5, 24, 16, 24), (2, 3, 64, 64, 32), (1, 2, 128, 96, 128), (1, 2, 48, 200, 16), (1, 1, 200, 33, 50),
                                         (3, 2, 9, 6, 4), (1, 2, 128, 256, 128), (1, 6, 32, 72, 0)])
def test_retention_whole_and_in_portions(dtype, B, H, D, E, rot):
    T = 300
    q, k, v, decay, freqs, want, S = retention_case(H * D + E, B, T, H, D, E, rot, dtype)
    for cut in ([300], [64, 128, 108], [1, 2, 63, 234], [130, 2, 2, 166], [129, 171]):
        got, st = run_retention(q, k, v, decay, freqs, dtype, cut)
        for h in range(H):
            close(got[:, :, h], want[:, :, h], dtype)
            # the state is 32-bit whatever the model's dtype
            assert float((st[:, h].double().cpu() - S[:, h]).abs().max() / S[:, h].abs().max()) < 2e-5, (cut, h)


def test_retention_remembers_far_tokens():
    """A token whose key answers the last query shows through slow decays at any distance and across every chunk's edge,
    and a state from before the prompt does."""
    T, H, D, E = 700, 2, 64, 64
    for far in (0, 63, 64, 127, 128, 255, 256, 600):
        q, k, v, _, freqs, _, _ = retention_case(3, 1, T, H, D, E, 0, torch.bfloat16)
        decay = torch.tensor([0.999, 1.0], dtype=torch.float64)
        k, v = k * 0.01, v * 0.01
        k[0, far], v[0, far] = 8 * q[0, -1], 5.0
        y, _ = oracle.retention_scan(rounded(q[0], torch.bfloat16), rounded(k[0], torch.bfloat16) * D ** -0.5, rounded(v[0], torch.bfloat16), decay)
        got, _ = run_retention(q, k, v, decay, freqs, torch.bfloat16, [700])
        close(got[0, -1], y[-1], torch.bfloat16)
        got, _ = run_retention(q, k, v, decay, freqs, torch.bfloat16, [far + 1, T - far - 1])
        close(got[0, -1], y[-1], torch.bfloat16)


def test_long_retention_prompts_against_the_token_recurrence():
    """Prompt kernels (chunks, ragged ends) on the same values in fp32, from a state that is not zero."""
    from triune_b200.ops import hybrid as hops

    for B, H, D, E, rot in ((1, 2, 128, 128, 128), (2, 3, 96, 72, 32), (1, 4, 64, 256, 64), (3, 2, 32, 40, 16), (1, 2, 128, 512, 64)):
        for T in (1500, 1024, 129, 65):
            r = gen(T + D)
            bf = lambda t: t.to("cuda", torch.bfloat16)
            q, k, v, S0 = bf(r(B * T, H * D)), bf(r(B * T, H * D)), bf(r(B * T, H * E)), dev(r(B, H, D, E))
            decay = torch.linspace(0.2, 1.0, H, dtype=torch.float64, device="cuda")
            i = torch.arange(rot // 2, dtype=torch.float64, device="cuda")
            table = hops.rotation_rows(1e4 ** (-2 * i / rot), 1.0, 77, T)
            outs = []
            for dtype in (torch.float32, torch.bfloat16):
                st, out = S0.clone(), torch.empty(B * T, H * E, device="cuda", dtype=dtype)
                hops.retention(q.to(dtype), k.to(dtype), v.to(dtype), table, decay, st, out, B, T)
                outs.append((out.view(B, T, H, E).double(), st.double()))
            hops.check_status(torch.device("cuda", 0))
            (want, sw), (got, sg) = outs
            for h in range(H):
                assert float((got - want)[:, :, h].abs().max() / want[:, :, h].abs().max()) < 1e-2, (T, D, E, h)
                assert float((sg - sw)[:, h].abs().max() / sw[:, h].abs().max()) < 1e-4, (T, D, E, h)


# ---- latent attention --------------------------------------------------------------------------------------------
class LatentCase:
    """Projected rows, expansion weights and the plain result; ``far``: the last query of the last head answers one key."""

    def __init__(self, seed, B, T, H, D, R, E, rank, dtype, far=None, gate=True, sink=True, own=True):
        r = gen(seed)
        self.B, self.T, self.dims, self.dtype, self.rank = B, T, (D, R, E), dtype, rank
        self.Dp, self.Rp, self.Ep, self.rank_p = pad8(D), pad8(R), pad8(E), pad8(rank)
        self.rot = {"dims": R, "base": 500.0, "scaling": {"factor": 4.0, "original": 50, "fast": 6.0, "slow": 1.0}}
        f, self.amp = oracle.rotation_table(self.rot)
        self.freqs = torch.tensor(f, dtype=torch.float64)
        q, qr, z, zr, g = r(B, T, H, D), r(B, T, H, R), r(B, T, rank), r(B, T, R), r(B, T, H)
        if far is not None:
            a = oracle.rotate_halves(qr[:, -1:, -1:].reshape(B, 1, R), torch.tensor([T - 1 - far]), {**self.rot})[:, 0]
            zr[:, far] = 5 * a
        self.uk, self.uv = r(H, D, rank) * rank ** -0.5, r(H, E, rank) * rank ** -0.5
        self.norm, self.eps = r(rank).abs() + 0.5, 1e-4
        self.sink = r(H) if sink else None
        self.scale = (D + R) ** -0.5
        self.col_q, self.col_c = 8, 8 + H * (self.Dp + self.Rp)
        self.col_g = self.col_c + self.rank_p + self.Rp
        proj = torch.zeros(B, T, self.col_g + pad8(H))
        heads = proj[..., self.col_q : self.col_c].view(B, T, H, self.Dp + self.Rp)
        heads[..., :D], heads[..., self.Dp : self.Dp + R] = q, qr
        proj[..., self.col_c : self.col_c + rank] = z
        proj[..., self.col_c + self.rank_p : self.col_c + self.rank_p + R] = zr
        proj[..., self.col_g : self.col_g + H] = g
        self.proj, self.has_gate, self.own = proj, gate, own
        x = lambda t: rounded(t, dtype)
        pos = torch.arange(T)
        self.want = torch.stack([oracle.latent_core(
            x(q[b]), oracle.rotate_halves(x(qr[b]), pos, self.rot), oracle.rms_norm(x(z[b]), self.norm.double(), self.eps),
            oracle.rotate_halves(x(zr[b])[:, None], pos, self.rot)[:, 0], x(self.uk), x(self.uv),
            oracle.sigmoid(x(g[b])) if gate else None, None if self.sink is None else self.sink.double(), self.scale) for b in range(B)])
        up = torch.zeros(H, self.Dp + self.Ep, self.rank_p)
        up[:, :D, :rank], up[:, self.Dp : self.Dp + E, :rank] = self.uk, self.uv
        self.up = dev(up, dtype)

    def run(self, cut, step_from=None):
        from triune_b200.ops import hybrid as hops

        D, R, E = self.dims
        B, T, H = self.B, self.T, self.up.shape[0]
        cache = torch.zeros(B, 1, 64 * (T // 64 + 2), self.rank_p + self.Rp, device="cuda", dtype=self.dtype)
        own = (self.col_c, dev(self.norm), self.eps)
        col_g = self.col_g if self.has_gate else None
        sink = None if self.sink is None else dev(self.sink)
        at, outs = 0, []
        for n in cut:
            part = self.proj[:, at : at + n].reshape(B * n, -1)
            if n == 1 and step_from is not None and at >= step_from:
                out = torch.empty(B, H * E, device="cuda")
                qa = torch.empty(B, H, self.rank_p + self.Rp, device="cuda")
                res = torch.empty(B, H, hops.latent_step_splits(B, H), hops.step_part_stride(self.rank_p), device="cuda")
                where = at if at % 2 else torch.tensor([at], device="cuda")
                hops.latent_step(dev(part.to(self.dtype).float()), self.col_q, col_g, own, cache, self.up, dev(self.freqs), self.amp, sink, qa,
                                 res, out, self.rank, D, R, E, self.scale, 0.5, where)
            else:
                out = torch.empty(B * n, pad8(H * E), device="cuda", dtype=self.dtype)
                hops.latent_attention(dev(part, self.dtype), self.col_q, col_g, own, cache, self.up,
                                      hops.rotation_rows(dev(self.freqs), self.amp, at, n), sink, out, B, n, self.rank, D, R, E, self.scale,
                                      0.5, at)
            outs.append(out[:, : H * E].reshape(B, n, H, E).double().cpu())
            at += n
        hops.check_status(torch.device("cuda", 0))
        return torch.cat(outs, 1) * 2


LATENT_SIZES = [(4, 16, 8, 24, 32), (3, 10, 6, 14, 20), (2, 128, 64, 128, 256), (2, 96, 32, 64, 128), (2, 64, 64, 72, 64), (1, 128, 64, 40, 136),
                (2, 136, 16, 144, 48), (18, 8, 8, 8, 16), (1, 16, 8, 300, 24)]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,D,R,E,rank", LATENT_SIZES)
def test_latent_prompts_in_portions(dtype, H, D, R, E, rank):
    c = LatentCase(1, 2, 301, H, D, R, E, rank, dtype)
    for cut in ([301], [130, 2, 64, 105], [1, 129, 171], [256, 45]):
        close(c.run(cut), c.want, dtype, 2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,D,R,E,rank", LATENT_SIZES + [(16, 32, 16, 32, 512), (5, 24, 8, 16, 200), (2, 16, 8, 16, 640)])
def test_latent_steps(dtype, H, D, R, E, rank):
    """Steps behind a prompt against the plain result, and alone from the first token."""
    for B, T, start in ((1, 330, 318), (2, 30, 0)):
        c = LatentCase(2, B, T, H, D, R, E, rank, dtype)
        got = c.run([start] * (start > 0) + [1] * (T - start), step_from=0)
        close(got[:, start:], c.want[:, start:], dtype, 2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("gate,sink", [(False, True), (True, False)])
def test_latent_without_gate_or_sink(dtype, gate, sink):
    c = LatentCase(3, 1, 80, 3, 16, 8, 24, 32, dtype, gate=gate, sink=sink)
    close(c.run([70] + [1] * 10, step_from=0), c.want, dtype, 2)


@pytest.mark.parametrize("dtype", DT)
def test_latent_far_keys(dtype):
    """One key stands out for the last query of the last head, at the borders of tiles, splits and portions; the last token
    comes in a prompt and in a step."""
    T = 403
    for far in (0, 1, 63, 64, 127, 128, 255, 256, 383, 384, 401):
        c = LatentCase(4, 1, T, 2, 32, 16, 16, 48, dtype, far=far)
        plain = LatentCase(4, 1, T, 2, 32, 16, 16, 48, dtype)
        assert (c.want[0, -1, -1] - plain.want[0, -1, -1]).abs().max() > 0.2 * c.want.abs().max()
        for cut in ([T], [T - 1, 1], [far + 1, T - far - 1]):
            close(c.run(cut, step_from=0)[0, -1], c.want[0, -1], dtype, 2)


def test_groups_of_heads_bound_the_expansion(monkeypatch):
    from triune_b200.ops import hybrid as hops

    c = LatentCase(5, 2, 70, 5, 24, 8, 16, 40, torch.bfloat16)
    whole = c.run([64, 6])
    monkeypatch.setattr(hops, "LATENT_BYTES", 2 * 2 * 64 * 40 * 2)  # two heads at a time
    assert torch.equal(c.run([64, 6]), whole)


# ---- steps -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("B", [1, 2, 3, 8])
@pytest.mark.parametrize("n,N", [(48, 40), (37, 33), (1024, 260)])
def test_projection_of_a_sum(dtype, B, n, N):
    """norm(x + norm(y + bias)) in the prologue, the sum kept; biases, the clamped activation and the token side behind."""
    from triune_b200.ops import hybrid as hops

    r = gen(B + n)
    x, y, b, w1, w2 = r(B, n), r(B, n) + 0.5, r(n), r(n), r(n)
    W, b2, table, ids = r(2 * N, n) * 2 * n ** -0.5, r(2 * N), r(11, 3 * N), torch.randint(0, 11, (B,))
    Wb = rounded(W, dtype)
    total = x.double() + oracle.rms_norm(y.double() + b.double(), w1.double(), 1e-3)
    h = oracle.rms_norm(total, w2.double(), 1e-5)

    def seg(pre, keep):
        return hops.seg_added(dev(x), dev(y), dev(b), (dev(w1), 1e-3, "rms"), (dev(w2), 1e-5, "rms") if pre else None, keep)

    keep, out = torch.empty(B, n, device="cuda"), torch.empty(B, N, device="cuda")
    close(hops.gemv([seg(True, keep)], dev(W[:N], dtype), out, bias=dev(b2[:N])), h @ Wb[:N].T + b2[:N].double(), torch.float32)
    close(keep, total, torch.float32)
    g, u = (h @ Wb[:N].T + b2[:N].double()).clamp(max=0.9), (h @ Wb[N:].T + b2[N:].double()).clamp(-0.9, 0.9)
    close(hops.gemv([seg(True, None)], dev(W, dtype), out, "glu", "clamped", dev(b2), 0.9, 1.702), g * oracle.sigmoid(1.702 * g) * (u + 1),
          torch.float32)
    close(hops.gemv([seg(False, None)], dev(W[:N], dtype), out, "side", "gelu_tanh", side=(dev(table, dtype), dev(ids), N)),
          oracle.gelu_tanh(total @ Wb[:N].T) * rounded(table, dtype)[ids][:, N : 2 * N], torch.float32)


@pytest.mark.parametrize("H,D,E,rot", [(3, 24, 16, 24), (2, 128, 256, 64), (5, 9, 33, 0), (1, 200, 40, 100)])
def test_retention_steps(H, D, E, rot):
    from triune_b200.ops import hybrid as hops

    B, T = 2, 40
    q, k, v, decay, freqs, want, S = retention_case(6, B, T, H, D, E, rot, torch.float32)
    st, outs = torch.zeros(B, H, D, E, device="cuda"), []
    for t in range(T):
        proj = dev(torch.cat((torch.zeros(B, 3), q[:, t].reshape(B, -1), k[:, t].reshape(B, -1), v[:, t].reshape(B, -1)), 1))
        out = torch.empty(B, H * E, device="cuda")
        hops.mixer_step(proj, {"state": st, "out": out, "kind": hops.KINDS["retention"], "col_q": 3, "col_k": 3 + H * D, "col_v": 3 + 2 * H * D,
                               "decay": dev(decay), "freqs": dev(freqs), "amplitude": 1.0}, None, t)
        outs.append(out.view(B, H, E).clone())
    close(torch.stack(outs, 1), want, torch.float32)
    close(st, S, torch.float32)


def test_gated_norm_without_a_weight():
    from triune_b200.ops import hybrid as hops

    r = gen(9)
    for inner, groups in ((48, 3), (35, 5), (1024, 4)):
        y, z, W = r(3, inner), r(3, inner), r(20, inner)
        want = oracle.unit_rms(y.double().view(3, groups, -1), 1e-3).reshape(3, inner) * oracle.silu(z.double()) * 0.7
        out = torch.empty(3, inner, device="cuda")
        hops.gated_norm(dev(y), dev(z), None, out, inner, groups, 1e-3, False, 0.7)
        close(out, want, torch.float32)
        acc = torch.empty(3, 20, device="cuda")
        close(hops.gemv([hops.seg_gated(dev(y), dev(z), None, groups, 1e-3, False, 0.7)], dev(W), acc), want @ W.double().T, torch.float32)


# ---- the model ---------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=sorted(CONFIGS))
def case(request):
    cfg = CONFIGS[request.param]
    W = oracle.make_weights(cfg, seed=3)
    toks = tokens(cfg, 150)
    return cfg, W, toks, oracle.forward(cfg, W, toks)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("portions", [[], [1] * 150, [2] * 75, [2, 3, 65, 7, 2, 11], [140, 1, 1, 2, 1], [64, 64]])
def test_model_prompts_decoding_and_portions(case, dtype, portions):
    cfg, W, toks, want = case
    assert agrees(run_portions(build(cfg, W, "cuda", dtype), toks, portions), want, dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("B", [3, 9])
def test_model_batches(case, dtype, B):
    """Rows of a batch against each alone; nine rows are more than the step kernels take."""
    cfg, W, _, _ = case
    m = build(cfg, W, "cuda", dtype)
    seqs = [tokens(cfg, 40, seed=s) for s in range(B)]
    lg, cache = m(torch.tensor([s[:36] for s in seqs], device="cuda"), cache=m.init_cache(B))
    parts = [lg]
    for t in range(36, 40):
        lg, cache = m(torch.tensor([s[t : t + 1] for s in seqs], device="cuda"), cache=cache)
        parts.append(lg)
    got = torch.cat(parts, 1)
    for i in (0, B - 1):
        assert agrees(got[i], oracle.forward(cfg, W, seqs[i]), dtype)


def test_layers_of_the_residual_stream(case):
    cfg, W, toks, _ = case
    _, layers = oracle.forward(cfg, W, toks[:40], want_layers=True)
    m = build(cfg, W, "cuda", torch.float32)
    seen, step = {}, {}
    m(torch.tensor([toks[:40]], device="cuda"), on_layer=lambda i, x: seen.update({i: x.double().cpu()}))
    _, cache = m(torch.tensor([toks[:39]], device="cuda"), cache=m.init_cache(1))
    m(torch.tensor([toks[39:40]], device="cuda"), cache=cache, on_layer=lambda i, x: step.update({i: x.double().cpu()}))
    for i, l in enumerate(layers):
        assert (seen[i] - l).abs().max() < 2e-4 * l.abs().max()
        assert (step[i][0] - l[39]).abs().max() < 2e-4 * l[39].abs().max()


def test_new_sequences_do_not_see_old_ones(case):
    cfg, W, toks, want = case
    m = build(cfg, W, "cuda", torch.float32)
    for n in (90, 3):
        run_portions(m, tokens(cfg, n, seed=n), [n - 2])   # leaves freed caches behind for the allocator to reuse
        assert agrees(run_portions(m, toks[:60], [50]), want[:60], torch.float32)


def test_long_decoding():
    cfg = CONFIGS["single"]
    W = oracle.make_weights(cfg, seed=8)
    toks = tokens(cfg, 700)
    want = oracle.forward(cfg, W, toks)
    for dtype in DT:
        assert agrees(run_portions(build(cfg, W, "cuda", dtype), toks, [20] + [1] * 680), want, dtype)


@pytest.mark.parametrize("name", ["shared", "odd", "wide"])
def test_greedy_generation_eager_and_graph(name):
    from triune_b200.inference import GraphedGreedyDecoder, generate_tokens

    cfg = CONFIGS[name]
    W = oracle.make_weights(cfg, seed=11)
    toks = tokens(cfg, 70)
    out = list(toks)
    for _ in range(12):
        out.append(int(oracle.forward(cfg, W, out)[-1].argmax()))
    m = build(cfg, W, "cuda", torch.float32)
    ids = torch.tensor([toks], device="cuda")
    got, _, _ = generate_tokens(m, ids, 12, temperature=0.0, repetition_penalty=1.0, count_penalty=0.0, prefill_chunk=33)
    assert got == out[70:]
    dec = GraphedGreedyDecoder(m)
    assert dec.generate(ids, 12)[0].tolist() == out
    assert dec.generate(ids[:, :40], 220)[0, :41].tolist() == toks[:40] + [int(oracle.forward(cfg, W, toks[:40])[-1].argmax())]
    assert dec.generate(ids, 12)[0].tolist() == out          # after the cache grew and was captured again
    b = build(cfg, W, "cuda", torch.bfloat16)
    two = GraphedGreedyDecoder(b, batch_size=2).generate(ids.expand(2, -1).contiguous(), 8)
    assert torch.equal(two[0], two[1])
    nine = GraphedGreedyDecoder(m, batch_size=9).generate(ids.expand(9, -1).contiguous(), 6)  # prompt kernels at a device position
    assert all(row.tolist() == out[:76] for row in nine)


def test_sessions_resume_and_fork():
    """Parked and resumed states continue as if nothing had happened, layers that share latents included."""
    from triune_b200.inference import advance
    from triune_b200.serve.srsm import _pack, _unpack

    cfg = CONFIGS["shared"]
    W = oracle.make_weights(cfg, seed=6)
    toks = tokens(cfg, 60)
    want = oracle.forward(cfg, W, toks)
    m = build(cfg, W, "cuda", torch.float32)
    _, cache = advance(m, torch.tensor([toks[:50]], device="cuda"), m.init_cache(1))
    flat, layout = _pack(cache)
    parked = flat.cpu()
    run_portions(m, tokens(cfg, 80, seed=2), [40])
    for _ in range(2):
        cache, got = _unpack(parked.to("cuda"), layout), []
        for t in range(50, 60):
            lg, cache = advance(m, torch.tensor([toks[t : t + 1]], device="cuda"), cache)
            got.append(lg[0].double().cpu())
        assert agrees(torch.cat(got), want[50:], torch.float32)
