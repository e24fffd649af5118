"""Heterogeneous-layer models on the GPU: every kernel against a plain fp64 statement of its operation, the model in bf16
and in 32-bit against the plain model, decoding steps, portions, batches, graph-replayed generation."""

import pytest
import torch

import hybrid_oracle as oracle
from hybrid_cases import CONFIGS, build, rel, run_portions, tokens

pytestmark = pytest.mark.gpu

DT = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-5, torch.bfloat16: 6e-2}  # bf16 at widths of 36 to 96: rounding alone reaches 5e-2


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


# ---- mechanisms --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("rows,width", [(1, 37), (5, 96), (33, 2048), (3, 16384)])
def test_norm_rows(dtype, rows, width):
    from triune_b200.ops import hybrid as hops

    r = gen(0)
    x, w = r(rows, width) * 3 + 1.5, r(width)
    close(hops.norm_rows(dev(x), dev(w), 1e-3, "layer", dtype), oracle.layer_norm(x.double(), w.double(), 1e-3), dtype)
    close(hops.norm_rows(dev(x), dev(w), 1e-3, "rms", dtype), oracle.unit_rms(x.double(), 1e-3) * w.double(), dtype)


@pytest.mark.parametrize("dtype", DT)
def test_gated_activation_and_gated_norm(dtype):
    from triune_b200.ops import hybrid as hops

    r = gen(1)
    h, gu = r(9, 40), r(2 * 24, 40) * 0.3
    hb, gb = rounded(h, dtype), rounded(gu, dtype)
    pre = hb @ gb.T
    for act, fn in (("relu", lambda z: z.clamp(min=0)), ("silu", oracle.silu)):
        close(hops.gated_mlp_hidden(dev(h, dtype), dev(gu, dtype), act), fn(pre[:, :24]) * pre[:, 24:], dtype, 2)
    y, z, w = r(7, 48), r(7, 50), r(48)
    yb, zb = rounded(y, dtype), rounded(z, dtype)[:, :48]
    out = torch.empty(7, 60, device="cuda", dtype=dtype)
    hops.gated_norm(dev(y, dtype), dev(z, dtype), dev(w), out, 48, 3, 1e-3, True, 0.7)
    want = oracle.unit_rms((yb * oracle.silu(zb)).view(7, 3, 16), 1e-3).reshape(7, 48) * w.double() * 0.7
    close(out[:, :48], want, dtype)
    hops.gated_norm(dev(y, dtype), dev(z, dtype), dev(w[:16].contiguous()), out, 48, 3, 1e-3, False, 1.0)
    want = (oracle.unit_rms(yb.view(7, 3, 16), 1e-3) * w[:16].double()).reshape(7, 48) * oracle.silu(zb)
    close(out[:, :48], want, dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_convolution_portions(dtype, taps):
    from triune_b200.ops import hybrid as hops

    r = gen(taps)
    T, C = 150, 70
    u, w, b = r(T, C), r(C, taps), r(C)
    want = oracle.causal_conv(rounded(u, dtype), w.double(), b.double())
    ud = dev(u, dtype)
    for cut in ([150], [2] * 75, [33, 2, 64, 1, 50], [1, 2, 3, 144]):
        ring, at, out = torch.full((1, taps, C), 9.0, device="cuda"), 0, []
        for n in cut:
            y, ring = hops.causal_conv(ud[at : at + n], dev(w), dev(b), ring, 1, n, at)
            out.append(y[:, :C])
            at += n
        close(torch.cat(out), want, dtype)


def recurrence_inputs(seed, T, H, K, D, E):
    r = gen(seed)
    return r(T, K, D), r(T, K, D), r(T, H, E), r(T, H), r(T, H), r(H), r(H) - 1, r(H)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", ["mamba2", "delta"])
@pytest.mark.parametrize("H,K,D,E", [(4, 2, 24, 20), (3, 3, 64, 64), (2, 1, 128, 96), (2, 2, 48, 48), (1, 1, 200, 33), (4, 1, 9, 6)])
def test_recurrence_whole_and_in_portions(dtype, kind, H, K, D, E):
    from triune_b200.ops import hybrid as hops

    T = 203
    q, k, v, a, b, A, bias, Dd = recurrence_inputs(H * D + E, T, H, K, D, E)
    qb, kb, vb, ab, bb = (rounded(t, dtype) for t in (q, k, v, a, b))
    dt = oracle.softplus(ab + bias.double())
    if kind == "mamba2":
        want, S = oracle.mamba2_scan(vb, kb, qb, dt, A.double(), Dd.double())
    else:
        unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
        want, S = oracle.delta_scan(unit(qb) * D ** -0.5, unit(kb), vb, torch.exp(-torch.exp(A.double()) * dt), oracle.sigmoid(bb))
    qd, kd, vd, ad, bd = (dev(t.reshape(T, -1), dtype) for t in (q, k, v, a, b))
    for cut in ([203], [64, 64, 75], [1, 2, 63, 137], [130, 2, 2, 69]):
        st, at = torch.zeros(1, H, D, E, device="cuda"), 0
        out = torch.empty(T, H * E, device="cuda", dtype=dtype)
        for n in cut:
            s = slice(at, at + n)
            hops.recurrent(qd[s], kd[s], vd[s], ad[s], bd[s] if kind == "delta" else None, dev(A), dev(bias),
                           dev(Dd) if kind == "mamba2" else None, st, out[s], 1, n, kind, K)
            at += n
        close(out.view(T, H, E), want, dtype)
        # the state is 32-bit whatever the model's dtype
        assert float((st[0].double().cpu() - S).abs().max() / S.abs().max()) < 1e-4


@pytest.mark.parametrize("kind", ["mamba2", "delta"])
@pytest.mark.parametrize("B,H,K,D,E", [(1, 2, 1, 128, 64), (2, 3, 3, 96, 72), (1, 4, 2, 64, 48), (3, 2, 2, 72, 40), (1, 40, 1, 128, 128), (1, 6, 2, 20, 10)])
def test_long_prompts_in_segments(kind, B, H, K, D, E):
    """The chunk-parallel prompt kernels (segments, chunks, ragged ends) against the token recurrence on the same values in
    fp32, from a state that is not zero; slow and fast decays side by side."""
    from triune_b200.ops import hybrid as hops

    for T in (1500, 1024, 129, 65):
        r = gen(T + D)
        bf = lambda t: t.to("cuda", torch.bfloat16)
        q, k, v, a, b = bf(r(B * T, K * D)), bf(r(B * T, K * D)), bf(r(B * T, H * E)), bf(r(B * T, H)), bf(r(B * T, H))
        A, bias, Dd, S0 = dev(torch.linspace(-6, 2.5, H)), dev(r(H) - 1), dev(r(H)), dev(r(B, H, D, E))
        outs = []
        for dtype in (torch.float32, torch.bfloat16):
            c = lambda t: t.to(dtype)
            st, out = S0.clone(), torch.empty(B * T, H * E, device="cuda", dtype=dtype)
            hops.recurrent(c(q), c(k), c(v), c(a), c(b) if kind == "delta" else None, A, bias, Dd if kind == "mamba2" else None, st, out, B,
                           T, kind, K)
            outs.append((out.view(B, T, H, E).double(), st.double()))
        hops.check_status(torch.device("cuda", 0))
        (want, sw), (got, sg) = outs
        for h in range(H):
            assert float((got - want)[:, :, h].abs().max() / want[:, :, h].abs().max()) < 1e-2, (T, h)
            assert float((sg - sw)[:, h].abs().max() / sw[:, h].abs().max()) < 1e-4, (T, h)


def attention_case(seed, T, H, G, D, E, rot, dtype, far=None):
    r = gen(seed)
    pr = r(T, H * D + G * D + G * E)
    if far is not None:  # the last query of the last head answers one early key
        q = pr[T - 1, (H - 1) * D : H * D].clone()
        pr[far, H * D + (G - 1) * D : H * D + G * D] = q
    qw, kw, sink = r(D).abs() + 0.5, r(D).abs() + 0.5, r(H)
    p = rounded(pr, dtype)
    q, k, v = p.split([H * D, G * D, G * E], -1)
    n = lambda x, h, w: oracle.rotate_interleaved(oracle.unit_rms(x.reshape(T, h, D), 1e-4) * w.double(), torch.arange(T), rot, 1e4)
    want = lambda scale: oracle.sink_attention(n(q, H, qw), n(k, G, kw), v.reshape(T, G, E), scale, sink.double())
    i = torch.arange(rot // 2, dtype=torch.float64)
    return pr, qw, kw, sink, dev(1e4 ** (-2 * i / max(rot, 1))), want


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,G,D,E,rot", [(4, 2, 16, 24, 8), (3, 1, 20, 10, 20), (8, 2, 128, 64, 64), (2, 2, 64, 128, 0), (6, 3, 64, 40, 48),
                                         (4, 4, 80, 48, 16), (2, 1, 128, 128, 128)])
def test_attention_prompt_portions_and_far_keys(dtype, H, G, D, E, rot):
    from triune_b200.ops import hybrid as hops

    T = 331
    for far in (None, 0, 63, 64, 127, 128, 200):
        pr, qw, kw, sink, fr, want = attention_case(7, T, H, G, D, E, rot, dtype, far)
        scale = D ** -0.5 if far is None else 6.0 / D
        ref = want(scale)
        prd = dev(pr, dtype)
        for cut in ([331], [130, 2, 64, 135], [1, 129, 201]) if far is None else ([331],):
            kc = torch.zeros(1, G, 384, -(-D // 8) * 8, device="cuda", dtype=dtype)
            vc = torch.zeros(1, G, 384, -(-E // 8) * 8, device="cuda", dtype=dtype)
            out, at = torch.empty(T, -(-H * E // 8) * 8, device="cuda", dtype=dtype), 0
            for n in cut:
                s = slice(at, at + n)
                hops.attention(prd[s], [0, H * D, (H + G) * D], dev(qw), dev(kw), 1e-4, fr, dev(sink), kc, vc, out[s], 1, n, H, D, E,
                               scale, 0.5, at)
                at += n
            got = out[:, : H * E].reshape(T, H, E)
            close(got, ref * 0.5, dtype, 2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("B", [1, 2, 3, 8])
def test_gemv_segments_and_epilogues(dtype, B):
    from triune_b200.ops import hybrid as hops

    r = gen(B)
    for n1, n2, N in ((48, 64, 40), (37, 30, 33), (512, 768, 260)):
        x, y1, y2, gate, w1, w2 = r(B, n1), r(B, n2), r(B, n2), r(B, n2 + 3), r(n1), r(n2)
        W = r(2 * N, n1) * n1 ** -0.5
        Wb = rounded(W, dtype)
        out = torch.empty(B, N, device="cuda")
        seg = lambda: hops.seg_norm(dev(x), dev(w1), 1e-3, "layer")
        h = oracle.layer_norm(x.double(), w1.double(), 1e-3)
        close(hops.gemv([seg()], dev(W[:N], dtype), out), h @ Wb[:N].T, torch.float32)
        close(hops.gemv([seg()], dev(W, dtype), out, "glu", "relu"), (h @ Wb[:N].T).clamp(min=0) * (h @ Wb[N:].T), torch.float32)
        W2 = r(N, n1 + n2) * n1 ** -0.5
        base = dev(r(B, N))
        groups = 2 if n2 % 2 == 0 else 1
        want = base.double().cpu() + torch.cat((0.3 * x.double(), 0.9 * oracle.unit_rms((y2.double() * oracle.silu(gate[:, :n2].double())).view(
            B, groups, -1), 1e-3).reshape(B, n2) * w2.double()), 1) @ rounded(W2, dtype).T
        hops.gemv([hops.seg_plain(dev(x), 0.3), hops.seg_gated(dev(y2), dev(gate), dev(w2), groups, 1e-3, True, 0.9)], dev(W2, dtype), base, "add")
        close(base, want, torch.float32)


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
    assert rel(run_portions(build(cfg, W, "cuda", dtype), toks, portions), want) < TOL[dtype]


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
        assert rel(got[i], oracle.forward(cfg, W, seqs[i])) < TOL[dtype]


def test_new_sequences_do_not_see_old_ones(case):
    cfg, W, toks, want = case
    m = build(cfg, W, "cuda", torch.float32)
    for n in (90, 3):
        run_portions(m, tokens(cfg, n, seed=n), [n - 2])   # leaves freed caches behind for the allocator to reuse
        assert rel(run_portions(m, toks[:60], [50]), want[:60]) < TOL[torch.float32]


def test_long_decoding():
    cfg = CONFIGS["plain"]
    W = oracle.make_weights(cfg, seed=8)
    toks = tokens(cfg, 700)
    want = oracle.forward(cfg, W, toks)
    for dtype in DT:
        assert rel(run_portions(build(cfg, W, "cuda", dtype), toks, [20] + [1] * 680), want) < TOL[dtype]


@pytest.mark.parametrize("name", ["grouped", "odd", "wide"])
def test_greedy_generation_eager_and_graph(name):
    from triune_b200.inference import GraphedGreedyDecoder, generate_tokens

    cfg = CONFIGS[name]
    W = oracle.make_weights(cfg, seed=11)
    toks = tokens(cfg, 70)
    out = list(toks)
    for _ in range(16):
        out.append(int(oracle.forward(cfg, W, out)[-1].argmax()))
    m = build(cfg, W, "cuda", torch.float32)
    ids = torch.tensor([toks], device="cuda")
    got, _, _ = generate_tokens(m, ids, 16, temperature=0.0, repetition_penalty=1.0, count_penalty=0.0, prefill_chunk=33)
    assert got == out[70:]
    dec = GraphedGreedyDecoder(m)
    assert dec.generate(ids, 16)[0].tolist() == out
    assert dec.generate(ids[:, :40], 200)[0, :41].tolist() == toks[:40] + [int(oracle.forward(cfg, W, toks[:40])[-1].argmax())]
    assert dec.generate(ids, 16)[0].tolist() == out          # after the cache grew and was captured again
    b = build(cfg, W, "cuda", torch.bfloat16)
    two = GraphedGreedyDecoder(b, batch_size=2).generate(ids.expand(2, -1).contiguous(), 8)
    assert torch.equal(two[0], two[1])
