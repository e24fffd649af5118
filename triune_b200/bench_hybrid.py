"""Serving benchmark of heterogeneous-layer models (layers at the sizes of a real model, random weights) beside another
family at equal size, whole models and kernel by kernel: Famalorn beside the dense family, Bubitar beside Famalorn.

    python bench.py --workload hybrid [--hybrid-design bubitar|famalorn] [--hybrid-size 1b|3b] [--hybrid-seq 8192]
                    [--hybrid-parts model,kernels]

Every kernel line carries its roofline time (the slower of its bytes over the measured copy bandwidth and its tensor-core
operations over the measured bf16 rate) and ``x_roofline`` = time / roofline; the like kernels of the other family are
measured by the same rule in the same run. CUDA events around a replayed graph of the call, warm-up, L2 flushed between
iterations. Model lines: prefill is one forward over the prompt into the cache, decoding is the graph-replayed greedy loop
after that prompt."""

from __future__ import annotations

import json
import time
from typing import Callable, Dict, List

import torch

from .bench_kernels import flush_l2, peaks, timeit


def famalorn_config(size: str) -> Dict:
    w, ah, kv, mh, dh, ff, reps = {"1b": (2048, 16, 4, 32, 16, 5632, 2), "3b": (3072, 24, 8, 48, 24, 8192, 3)}[size]
    attn = {"heads": ah, "kv_heads": kv, "dim": 128, "vdim": 128, "rot": {"base": 1e6, "dims": 64}, "scale": 128 ** -0.5}
    mamba = {"heads": mh, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1}
    layers = [
        {"type": "parallel", "mixer": {"left": attn, "right": mamba, "left_scale": 0.5, "right_scale": 0.5}, "mlp": {"kind": "dense", "ff": ff}},
        {"type": "delta", "mixer": {"heads": dh, "kv_heads": dh, "dim": 128, "vdim": 128, "conv": 4}, "mlp": None},
        {"type": "mamba2", "mixer": {**mamba, "heads": 2 * mh}, "mlp": None},
    ]
    return {"architecture": "Famalorn", "layers": layers * reps, "norm": {"eps": 1e-5}, "vocab": 32000, "width": w}


def bubitar_config(size: str) -> Dict:
    """Retention with values twice as wide as keys, latent attention of which every second layer reads earlier latents."""
    w, h, ff, reps = {"1b": (2048, 16, 5632, 1), "3b": (3072, 24, 8192, 2)}[size]
    decay = [1 - 2.0 ** -(5 + 4 * i / (h - 1)) for i in range(h)]
    mlp = {"kind": "dense", "ff": ff, "limit": 7.0}
    ret = {"type": "retention", "mlp": mlp, "mixer": {"heads": h, "dim": 128, "vdim": 256, "decay": decay, "rot": {"dims": 128, "base": 1e4}}}
    rot = {"dims": 64, "base": 1e4, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    lat = {"heads": h, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5, "rot": rot}
    own, shared = ({"type": "latent_attention", "mlp": mlp, "mixer": m} for m in (lat, {**lat, "kv_from": 2}))
    return {"architecture": "Bubitar", "layers": [ret, ret, own] + [ret, ret, shared] * reps, "norm": {"eps": 1e-5}, "vocab": 32000,
            "width": w, "token_side": {"dim": 256}}


def dense_config(size: str, mixer: str):
    from .config import ModelConfig

    c = famalorn_config(size)
    a = c["layers"][0]["mixer"]["left"]
    return ModelConfig(family="universal", vocab_size=32000, hidden_dim=c["width"], num_layers=len(c["layers"]), num_heads=a["heads"],
                       head_dim=128, num_kv_heads=a["kv_heads"] if mixer == "sdpa" else None, mixer=mixer, ffn="swiglu",
                       dense_hidden=c["layers"][0]["mlp"]["ff"], tie_embeddings=False).validate()


def emit(**kw) -> None:
    print(json.dumps({k: (round(v, 4) if isinstance(v, float) else v) for k, v in kw.items()}), flush=True)


def replayed(fn: Callable) -> Callable:
    """``fn`` as a replayed CUDA graph, so that a short kernel's time is not the host's."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        fn()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        fn()
    return g.replay


class Table:
    """Kernel lines with their roofline ratios."""

    def __init__(self, iters: int):
        p = peaks()
        self.bw, self.tf, self.iters = p["hbm_gbs"] * 1e9, p["tflops"] * 1e12, iters

    def __call__(self, model: str, kernel: str, fn: Callable, nbytes: float, flops: float = 0.0) -> float:
        ms = timeit(replayed(fn), self.iters)
        roof = max(nbytes / self.bw, flops / self.tf) * 1e3
        emit(workload="hybrid", model=model, kernel=kernel, us=ms * 1e3, roofline_us=roof * 1e3, x_roofline=ms / roof,
             gbs=nbytes / ms / 1e6, tflops=flops / ms / 1e9)
        return ms


def build_design(name: str, size: str, dev):
    from .models import Bubitar, Famalorn
    from .utils import place_model

    with torch.device(dev):
        m = {"famalorn": lambda: Famalorn(config=famalorn_config(size)), "bubitar": lambda: Bubitar(config=bubitar_config(size))}[name]()
    return place_model(m.init_weights(), dev, torch.bfloat16).eval()


def portion(T: int, pos, dev):
    from .models.hybrid_mixers import Portion

    return Portion(1, T, pos, torch.bfloat16, torch.randint(0, 32000, (T,), device=dev), [])


def build_dense(size: str, mixer: str, dev):
    from .models.factory import build_model
    from .utils import place_model

    torch.manual_seed(0)
    with torch.device(dev):
        m = build_model(dense_config(size, mixer))
    return place_model(m, dev, torch.bfloat16).eval()


# ---------------------------------------------------------------------------------------------------- kernels
def famalorn_kernels(size: str, T: int, iters: int) -> None:
    """The layer's kernels at prompt length T, then one decoding step at that context."""
    from .ops import hybrid as hops

    dev, name, t = torch.device("cuda"), f"famalorn-{size}", Table(iters)
    m = build_design("famalorn", size, dev)
    W = m.hidden_dim
    x = torch.randn(T, W, device=dev)
    with torch.no_grad():
        for layer, label in zip(m.layers[:3], ("parallel", "delta", "mamba2")):
            mix = layer.mixer
            st = mix.new_state(1, dev, torch.bfloat16)
            st.reserve(T + 64)
            h = layer.norm1(x, torch.bfloat16)
            proj = hops.linear(h, mix.in_weight)
            y = torch.empty(T, mix.out_weight.shape[1], device=dev, dtype=torch.bfloat16)
            N, K = mix.in_weight.shape[0], mix.out_weight.shape[1]
            if label == "parallel":
                t(name, "layer norm", lambda: layer.norm1(x, torch.bfloat16), T * W * 6)
            t(name, f"{label}: input GEMM", lambda: hops.linear(h, mix.in_weight), 2 * (T * W + N * W + T * N), 2 * T * N * W)
            for i, c in enumerate(mix.cores):
                col, out, at = mix.cols[i], y[:, mix.outs[i] :], c.inputs.at
                if hasattr(c, "kind") and c.kind:
                    C, H, dk, dv = c.conv_at.total, c.heads, c.dk, c.dv
                    u, _ = hops.causal_conv(proj[:, col + at["u"] :], c.conv_w, getattr(c, "conv_b", None), st[f"{i}.conv"], 1, T, 0)
                    t(name, f"{label}: {c.kind} convolution", lambda: hops.causal_conv(
                        proj[:, col + at["u"] :], c.conv_w, getattr(c, "conv_b", None), st[f"{i}.conv"], 1, T, 0), 4 * T * C)
                    yy = torch.empty(T, c.out_width, device=dev, dtype=torch.bfloat16)
                    ca = c.conv_at.at
                    # chunk form, 64 tokens: scores and state products per head; the delta rule solves a triangle more
                    L = 64
                    fl = T * H * 2.0 * (L * dv + 2 * dk * dv) + T * c.key_groups * 2.0 * L * dk
                    if c.kind == "delta":
                        fl += T * H * 2.0 * (2 * L * dv + dk * dv) + T * c.key_groups * 2.0 * L * dk
                    t(name, f"{label}: {c.kind} recurrence", lambda: hops.recurrent(
                        u[:, ca["q"] :], u[:, ca["k"] :], u[:, ca["v"] :], proj[:, col + at["a"] :],
                        proj[:, col + at["b"] :] if "b" in at else None, c.A_log, c.dt_bias, getattr(c, "D", None), st[f"{i}.S"],
                        yy, 1, T, c.kind, c.key_groups), 2 * T * (C + H * dv), fl)
                    t(name, f"{label}: {c.kind} gated norm", lambda: hops.gated_norm(
                        yy, proj[:, col + at[c.gate_name] :], c.norm, out, c.out_width, c.norm_groups, c.eps, c.gate_first, c.out_scale),
                      6 * T * c.out_width)
                else:
                    fl = 2.0 * T * T / 2 * c.heads * (c.dim + c.vdim)
                    by = 2 * T * (2 * c.heads * c.dim + 2 * c.kv_heads * (c.dim + c.vdim) + c.heads * c.vdim)
                    t(name, f"{label}: attention (prep + softmax)", lambda: c(proj, col, st, f"{i}.", portion(T, 0, dev), out), by, fl)
            t(name, f"{label}: output GEMM into the residual", lambda: hops.linear_accumulate(x, y, mix.out_weight),
              2 * (T * K + W * K) + 8 * T * W, 2.0 * T * K * W)
            if layer.ffn is not None:
                F = layer.ffn.hidden
                t(name, "gated FFN hidden", lambda: hops.gated_mlp_hidden(h, layer.ffn.gate_up, layer.ffn.act),
                  2 * (T * W + 2 * F * W + T * F), 4.0 * T * F * W)
        x1 = torch.randn(1, W, device=dev)
        pos = torch.full((1,), T, dtype=torch.long, device=dev)
        for layer, label in zip(m.layers[:3], ("parallel", "delta", "mamba2")):
            mix = layer.mixer
            st = mix.new_state(1, dev, torch.bfloat16)
            st.reserve(T + 64)
            proj = torch.randn(1, mix.in_width, device=dev)
            t(name, f"step {label}: norm + input projection", lambda: hops.gemv([layer.norm1.segment(x1)], mix.in_weight[: mix.in_width], proj),
              mix.in_width * W * 2)
            recs, atts, segs, by = [], [], [], 0
            for i, c in enumerate(mix.cores):
                a, s = c.step(proj, mix.cols[i], st, f"{i}.", portion(1, pos, dev))
                segs.append(s)
                if hasattr(c, "kind") and c.kind:
                    recs.append(a)
                    by += 8 * c.heads * c.dk * c.dv
                else:
                    atts.append(a)
                    by += 2 * T * c.kv_heads * (c.dim + c.vdim)
            t(name, f"step {label}: mixer", lambda: hops.mixer_step(proj, recs[0] if recs else None, atts[0] if atts else None, pos), by)
            t(name, f"step {label}: gated norm + output projection", lambda: hops.gemv(segs, mix.out_weight, x1, "add"), mix.out_weight.numel() * 2)
            if layer.ffn is not None:
                hh = torch.empty(1, layer.ffn.hidden, device=dev)
                t(name, "step norm + gated FFN hidden", lambda: hops.gemv([layer.norm2.segment(x1)], layer.ffn.gate_up, hh, "glu"),
                  layer.ffn.gate_up.numel() * 2)


def bubitar_kernels(size: str, T: int, iters: int) -> None:
    """The layer's kernels at prompt length T, then one decoding step at that context."""
    from .models.hybrid import Residual
    from .ops import hybrid as hops

    dev, name, t, bf = torch.device("cuda"), f"bubitar-{size}", Table(iters), torch.bfloat16
    m = build_design("bubitar", size, dev)
    W, x = m.hidden_dim, torch.randn(T, m.hidden_dim, device=dev)
    p = portion(T, 0, dev)
    table = m.side_embed
    with torch.no_grad():
        p.states = [l.mixer.new_state(1, dev, bf) for l in m.layers]
        for st in p.states:
            st.reserve(T + 64)
        ys = torch.randn(T, W, device=dev).to(bf)
        for i, label in ((0, "retention"), (2, "latent"), (5, "shared latent")):
            layer, st = m.layers[i], p.states[i]
            mix, c = layer.mixer, layer.mixer.cores[0]
            h = layer.norm1(x, bf)
            proj = hops.linear(h, mix.in_weight)
            y = torch.empty(T, mix.out_weight.shape[1], device=dev, dtype=bf)
            N, K, at = mix.in_weight.shape[0], mix.out_weight.shape[1], c.inputs.at
            if i == 0:
                t(name, "shortest launch (one embedding row)", lambda: hops.embed_rows(p.ids[:1], m.embed), 6 * W)
                t(name, "norm behind + sum + next norm", lambda: hops.add_norm(x, ys, None, layer.norm1b.args, layer.norm2.args, bf), 12 * T * W)
            t(name, f"{label}: input GEMM", lambda: hops.linear(h, mix.in_weight), 2 * (T * W + N * W + T * N), 2 * T * N * W)
            if i == 0:
                H, D, E = c.heads, c.dim, c.vdim
                rows = hops.rotation_rows(c.freqs, 1.0, 0, T)
                t(name, "rotation rows (once per prompt)", lambda: hops.rotation_rows(c.freqs, 1.0, 0, T), 4 * T * D)
                q, k, v, g = (proj[:, at[n] :] for n in ("q", "k", "v", "g"))
                o = torch.empty(T, H * E, device=dev, dtype=bf)
                L = 64
                t(name, "retention: recurrence", lambda: hops.retention(q, k, v, rows, c.decay, st["0.S"], o, 1, T), 2 * T * H * (2 * D + 2 * E),
                  2.0 * T * H * (L * E + L * D + 2 * D * E))
                t(name, "retention: gated norm", lambda: hops.gated_norm(o, g, None, y, c.out_width, H, c.eps, False, 1.0), 6 * T * c.out_width)
            else:
                H, Q = c.heads, c.dim + c.rot
                fl = 2.0 * T * T / 2 * H * (Q + c.vdim) + 2.0 * T * c.rank * H * (c.dim + c.vdim)
                by = 2 * T * (H * Q + 2 * H * (c.dim + c.vdim) + H * c.vdim + 2 * (c.rank + c.rot)) + 2 * c.up.numel()
                t(name, f"{label}: attention (prep + expansion + softmax)", lambda: c(proj, 0, st, "0.", p, y), by, fl)
                lat = p.states[2]["0.c"][:, 0, :T, : c.rank_p]
                t(name, f"{label}: expansion GEMM", lambda: hops.linear(lat, c.up.view(-1, c.rank_p)),
                  2 * (T * c.rank + c.up.numel() + T * H * (c.dim + c.vdim)), 2.0 * T * c.rank * H * (c.dim + c.vdim))
            t(name, f"{label}: output GEMM", lambda: hops.linear(y, mix.out_weight), 2 * (T * K + W * K + T * W), 2.0 * T * K * W)
            if i == 0:
                F = layer.ffn.hidden
                t(name, "clamped FFN hidden", lambda: layer.ffn(h), 2 * (T * W + 2 * F * W + T * F), 4.0 * T * F * W)
                hid = layer.ffn(h)
                t(name, "FFN output GEMM", lambda: hops.linear(hid, layer.ffn.down), 2 * (T * F + W * F + T * W), 2.0 * T * F * W)
                S = layer.side.dim
                t(name, "token side: gate GEMM", lambda: hops.linear(h, layer.side.gate), 2 * (T * W + S * W + T * S), 2.0 * T * S * W)
                gate = hops.linear(h, layer.side.gate)
                t(name, "token side: gate rows", lambda: hops.token_side_hidden(gate, table, p.ids, 0), 6 * T * S)
                t(name, "token side: output GEMM", lambda: hops.linear(gate, layer.side.proj), 2 * (T * S + S * W + T * W), 2.0 * T * S * W)
        x1, y1 = torch.randn(1, W, device=dev), torch.randn(1, W, device=dev)
        p1 = portion(1, torch.full((1,), T, dtype=torch.long, device=dev), dev)
        p1.states = p.states

        def stream(norm):
            s = Residual(x1)
            s.add(y1, None, norm)
            return s

        for i, label in ((0, "retention"), (2, "latent"), (5, "shared latent")):
            layer, st = m.layers[i], p.states[i]
            mix, c = layer.mixer, layer.mixer.cores[0]
            proj = torch.randn(1, mix.in_width, device=dev)
            t(name, f"step {label}: sum + norms + input projection", lambda: hops.gemv([stream(layer.norm1b).segment(layer.norm1)],
                                                                                      mix.in_weight[: mix.in_width], proj), mix.in_width * W * 2)
            args, seg = c.step(proj, 0, st, "0.", p1)
            if i == 0:
                t(name, "step retention: mixer", lambda: hops.mixer_step(proj, args, None, p1.pos), 8 * c.heads * c.dim * c.vdim)
            else:
                t(name, f"step {label}: mixer (query + attention + value)", lambda: c.step(proj, 0, st, "0.", p1),
                  2 * T * (c.rank + c.rot) + 2 * c.up.numel())
            t(name, f"step {label}: output projection", lambda: hops.gemv([seg], mix.out_weight, y1), mix.out_weight.numel() * 2)
        layer = m.layers[0]
        hh = layer.ffn.step(layer.norm2.segment(x1), 1)
        t(name, "step sum + norms + clamped FFN hidden", lambda: layer.ffn.step(stream(layer.norm1b).segment(layer.norm2), 1),
          layer.ffn.gate_up.numel() * 2)
        t(name, "step FFN output", lambda: hops.gemv([hops.seg_plain(hh)], layer.ffn.down, y1), layer.ffn.down.numel() * 2)
        t(name, "step token side (both)", lambda: layer.side.step(stream(layer.norm2b), table, p1),
          (layer.side.gate.numel() + layer.side.proj.numel()) * 2)


def dense_kernels(size: str, T: int, iters: int) -> None:
    """The like kernels of the dense family."""
    from . import ops

    dev, t = torch.device("cuda"), Table(iters)
    cfg = dense_config(size, "sdpa")
    W, H, D, G, F = cfg.hidden_dim, cfg.num_heads, cfg.head_dim, cfg.num_kv_heads, cfg.dense_hidden
    bf = dict(device=dev, dtype=torch.bfloat16)
    with torch.no_grad():
        name = f"dense-{size}"
        xb, w = torch.randn(T, W, **bf), torch.ones(W, **bf)
        if W <= 2048:
            t(name, "RMS norm (+ residual)", lambda: ops.add_rmsnorm(xb, xb, w), 8 * T * W)
        qkvg = torch.randn(4 * H * D, W, **bf)
        t(name, "input GEMM", lambda: ops.linear(xb, qkvg), 2 * (T * W + qkvg.numel() + T * 4 * H * D), 8.0 * T * H * D * W)
        q, k, v = (torch.randn(1, h, T, D, **bf) for h in (H, H, H))
        t(name, "attention (library SDPA)", lambda: torch.nn.functional.scaled_dot_product_attention(q, k, v, is_causal=True),
          8 * T * H * D, 2.0 * T * T * H * D)
        pr = torch.randn(T, 4 * H * D, **bf)
        cos, sin = ops.rope_tables(T, D, 1e4, 0, dev)
        t(name, "query / key feature map + rotation", lambda: ops.qk_feature_map(pr, cos, sin, 1, T, H, D), 8 * T * H * D)
        qq, kk, vv, gg = ops.qk_feature_map(pr, cos, sin, 1, T, H, D)
        beta = torch.rand(1, T, H, device=dev)
        fl = T * H * 2.0 * (2 * 64 * D + 3 * 64 * D + 3 * D * D)
        t(name, "gated DeltaNet recurrence", lambda: ops.gated_deltanet(qq, kk, vv, gg, beta=beta, gate_logits=True), 10 * T * H * D, fl)
        from .ops import gla_cuda

        t(name, "gated linear attention", lambda: gla_cuda.gla_attention_core(pr, cos, sin, None, 1, T, H), 10 * T * H * D,
          T * H * 2.0 * (2 * 64 * D + 2 * D * D))
        o = torch.randn(T, H * D, **bf)
        wo = torch.randn(W, H * D, **bf)
        t(name, "output GEMM", lambda: ops.linear(o, wo), 2 * (2 * T * W + wo.numel()), 2.0 * T * H * D * W)
        w13, w2 = torch.randn(2 * F, W, **bf), torch.randn(W, F, **bf)
        t(name, "SwiGLU FFN (both GEMMs)", lambda: ops.swiglu_mlp(xb, w13, w2), 2 * (2 * T * W + 3 * F * W + 2 * T * F), 6.0 * T * F * W)
        x1 = torch.randn(1, 1, W, **bf)
        t(name, "step input projection", lambda: ops.linear(x1, qkvg), qkvg.numel() * 2)
        t(name, "step output projection", lambda: ops.linear(x1, wo), wo.numel() * 2)
        t(name, "step FFN (both)", lambda: ops.swiglu_mlp(x1, w13, w2), 6 * F * W)
        s0 = torch.randn(1, H, D, D, device=dev)
        t(name, "step gated DeltaNet", lambda: ops.gated_deltanet(qq[:, :1], kk[:, :1], vv[:, :1], gg[:, :1], beta=beta[:, :1], initial_state=s0,
                                                                 gate_logits=True), 8 * H * D * D)


# ---------------------------------------------------------------------------------------------------- models
def model_lines(tag: str, model, T: int, new_tokens: int, batches: List[int], graph: bool, iters: int) -> None:
    from .inference import GraphedGreedyDecoder, advance

    dev = torch.device("cuda")
    for B in batches:
        ids = torch.randint(0, model.vocab_size, (B, T), device=dev, generator=torch.Generator(device=dev).manual_seed(1))

        @torch.no_grad()
        def prefill():
            return advance(model, ids, model.init_cache(B), last_token_only=True)

        ms = timeit(prefill, iters)
        emit(workload="hybrid", model=tag, metric="prefill tok/s", value=B * T / ms * 1e3, ms=ms, batch=B, seq_len=T)
    for B in batches:
        ids = torch.randint(0, model.vocab_size, (B, min(T, 2048)), device=dev)
        if graph:
            dec = GraphedGreedyDecoder(model, batch_size=B)
            dec.prefill(ids)
            dec.decode(new_tokens)
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            dec.decode(new_tokens)
            torch.cuda.synchronize()
            dt = time.perf_counter() - t0
        else:
            with torch.no_grad():
                lg, cache = advance(model, ids, model.init_cache(B), last_token_only=True)
                for phase in range(2):
                    torch.cuda.synchronize()
                    t0 = time.perf_counter()
                    for _ in range(new_tokens):
                        lg, cache = advance(model, lg[:, -1].argmax(-1, keepdim=True), cache, last_token_only=True)
                    torch.cuda.synchronize()
                    dt = time.perf_counter() - t0
        emit(workload="hybrid", model=tag, metric="decode tok/s", value=B * new_tokens / dt, ms_per_token=dt / new_tokens * 1e3, batch=B,
             context=min(T, 2048), graph=graph)


def run(sizes: List[str], T: int = 8192, parts: str = "model,kernels", iters: int = 10, new_tokens: int = 128, design: str = "famalorn") -> None:
    dev = torch.device("cuda")
    designs = ["famalorn"] if design == "famalorn" else [design, "famalorn"]
    for size in sizes:
        if "kernels" in parts:
            for d in designs:
                {"famalorn": famalorn_kernels, "bubitar": bubitar_kernels}[d](size, T, iters)
            if design == "famalorn":
                dense_kernels(size, T, iters)
        if "model" not in parts:
            continue
        for d in designs:
            m = build_design(d, size, dev)
            emit(workload="hybrid", model=f"{d}-{size}", parameters=m.num_parameters(), layers=m.num_layers)
            model_lines(f"{d}-{size}", m, T, new_tokens, [1, 4], True, max(3, iters // 2))
            del m
        if design == "famalorn":
            for mixer, graph in (("gated_deltanet", True), ("gla", True), ("sdpa", False)):
                m = build_dense(size, mixer, dev)
                emit(workload="hybrid", model=f"dense-{size}-{mixer}", parameters=m.num_parameters(), layers=m.num_layers)
                model_lines(f"dense-{size}-{mixer}", m, T, new_tokens, [1, 4], graph, max(3, iters // 2))
                del m
        torch.cuda.empty_cache()
