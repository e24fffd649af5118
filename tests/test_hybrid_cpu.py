"""Heterogeneous-layer models on the CPU: the model code, its cache and its entry points against plain statements."""

import io
import json
import os
import subprocess
import sys

import pytest
import torch

import hybrid_oracle as oracle
from hybrid_cases import CONFIGS, build, rel, run_portions, tokens


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def case(request):
    cfg = CONFIGS[request.param]
    W = oracle.make_weights(cfg, seed=3)
    toks = tokens(cfg, 41)
    return cfg, W, toks, oracle.forward(cfg, W, toks)


def test_whole_prompt_matches_plain_statement(case):
    cfg, W, toks, want = case
    assert rel(run_portions(build(cfg, W), toks, []), want) < 2e-5
    assert rel(run_portions(build(cfg, W, dtype=torch.float64), toks, []), want) < 1e-6


@pytest.mark.parametrize("portions", [[1] * 41, [2] * 20, [2, 3, 5, 7, 2, 11], [40], [17, 1, 1, 1, 2, 2]])
def test_portions_do_not_matter(case, portions):
    cfg, W, toks, want = case
    assert rel(run_portions(build(cfg, W), toks, portions), want) < 2e-5


def test_batch_rows_are_independent(case):
    cfg, W, toks, want = case
    m = build(cfg, W)
    other = tokens(cfg, 41, seed=9)
    lg, cache = m(torch.tensor([toks[:30], other[:30]]), cache=m.init_cache(2))
    lg2, _ = m(torch.tensor([toks[30:], other[30:]]), cache=cache)
    got = torch.cat((lg, lg2), 1)
    assert rel(got[0], want) < 2e-5
    assert rel(got[1], oracle.forward(cfg, W, other)) < 2e-5


def test_layers_of_the_residual_stream(case):
    cfg, W, toks, _ = case
    _, layers = oracle.forward(cfg, W, toks, want_layers=True)
    seen = {}
    build(cfg, W)(torch.tensor([toks]), on_layer=lambda i, x: seen.update({i: x.clone()}))
    for i, l in enumerate(layers):
        assert (seen[i].double() - l).abs().max() < 1e-4 * l.abs().max()


def test_cache_growth_keeps_the_keys():
    cfg = CONFIGS["plain"]
    W = oracle.make_weights(cfg, seed=5)
    toks = tokens(cfg, 300)
    want = oracle.forward(cfg, W, toks)
    assert rel(run_portions(build(cfg, W), toks, [250, 3, 2, 40]), want) < 2e-5


def test_layer_state_clone_copy_pack():
    from triune_b200.models.layer_state import LayerState
    from triune_b200.serve.srsm import _pack, _unpack

    cfg = CONFIGS["odd"]
    m = build(cfg, oracle.make_weights(cfg, seed=1), dtype=torch.bfloat16)
    toks = tokens(cfg, 20)
    _, cache = m(torch.tensor([toks[:13]]), cache=m.init_cache(1))
    kept = [(s.clone(), p) for s, p in cache]
    flat, layout = _pack(cache)
    assert flat.dtype == torch.float32 and flat.dim() == 1
    a, _ = m(torch.tensor([toks[13:]]), cache=cache)          # advances the states in place
    b, _ = m(torch.tensor([toks[13:]]), cache=kept)
    c, _ = m(torch.tensor([toks[13:]]), cache=_unpack(flat.clone(), layout))
    assert torch.equal(a, b) and torch.equal(a, c)
    grown = LayerState({"k": torch.zeros(1, 1, 64, 8)}, ("k",))
    assert not grown.reserve(64) and grown.reserve(65) and grown.capacity == 128


def test_config_round_trip_and_validation():
    from triune_b200.config import ModelConfig
    from triune_b200.models.factory import build_model
    from triune_b200.models.famalorn import read_config

    cfg = read_config(CONFIGS["grouped"])
    again = ModelConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))).validate()
    assert again == cfg
    m = build_model(again)
    assert m.num_parameters() >= cfg.param_count()[0]          # alignment rows may add to it
    exact = sum(t.numel() for t in oracle.make_weights(CONFIGS["grouped"]).values())
    assert cfg.param_count()[0] == exact
    bad = json.loads(json.dumps(CONFIGS["grouped"]))
    bad["layers"][1]["mixer"]["left"]["rot"]["dims"] = 7
    with pytest.raises(ValueError):
        read_config(bad)
    bad = json.loads(json.dumps(CONFIGS["grouped"]))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError):
        read_config(bad)


def test_weights_that_do_not_fit_are_refused():
    from triune_b200.models import Famalorn

    cfg = CONFIGS["grouped"]
    W = oracle.make_weights(cfg)
    m = Famalorn(config=cfg)
    with pytest.raises(ValueError):
        m.load_named({k: v for k, v in W.items() if k != "l0.mix.b"})
    with pytest.raises(ValueError):
        m.load_named({**W, "extra": W["head"]})
    with pytest.raises(ValueError):
        m.load_named({**W, "head": W["head"][:-1]})


def save_folder(cfg, W, path):
    from triune_b200.export.safetensors_io import save_file

    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(W, str(path / "model.safetensors"))
    return path


def test_model_folder_loads_through_every_entry_point(tmp_path):
    from triune_b200.export.safetensors_io import load_file
    from triune_b200.inference import load_model_for_inference
    from triune_b200.models.zoo import list_models, load_model
    from triune_b200.serve.engine_state import EngineState

    cfg = CONFIGS["odd"]
    W = oracle.make_weights(cfg, seed=7)
    folder = save_folder(cfg, W, tmp_path / "m")
    toks = tokens(cfg, 19)
    want = oracle.forward(cfg, W, toks)
    for m in (load_model(str(folder)), load_model_for_inference(str(folder), "cpu", torch.float32)):
        assert rel(run_portions(m, toks, [5]), want) < 2e-5
    assert "famalorn" in list_models()
    m.save_pretrained(tmp_path / "copy")
    back = load_file(str(tmp_path / "copy" / "model.safetensors"))
    assert set(back) == set(W) and all(torch.equal(back[k], W[k]) for k in W)
    st = EngineState("cpu")
    assert st.load_model(str(folder))["num_layers"] == len(cfg["layers"])
    a = st.generate("abcdef", session_id="s", max_new_tokens=4, temperature=0.0, template=False)
    b = st.generate("gh", session_id="s", max_new_tokens=3, temperature=0.0, template=False)
    assert len(a["tokens"]) == 4 and len(b["tokens"]) == 3
    st.turbo_mode = True
    t = st.generate("abcdef", max_new_tokens=4, temperature=0.0, template=False, repetition_penalty=1.0)
    assert t["telemetry"]["turbo"] and len(t["tokens"]) == 4


def greedy(cfg, W, toks, n):
    out = list(toks)
    for _ in range(n):
        out.append(int(oracle.forward(cfg, W, out)[-1].argmax()))
    return out[len(toks):]


@pytest.mark.parametrize("name", ["grouped", "odd"])
def test_greedy_generation(name):
    from triune_b200.inference import GraphedGreedyDecoder, generate_tokens

    cfg = CONFIGS[name]
    W = oracle.make_weights(cfg, seed=11)
    toks = tokens(cfg, 15)
    want = greedy(cfg, W, toks, 12)
    m = build(cfg, W, dtype=torch.float64)
    got, _, _ = generate_tokens(m, torch.tensor([toks]), 12, temperature=0.0, repetition_penalty=1.0, count_penalty=0.0,
                                prefill_chunk=7)
    assert got == want
    dec = GraphedGreedyDecoder(m)
    assert dec.generate(torch.tensor([toks]), 12)[0, 15:].tolist() == want
    assert dec.generate(torch.tensor([toks[:9]]), 12)[0, 9:].tolist() == greedy(cfg, W, toks[:9], 12)


def test_checkpoint_of_a_hybrid_model(tmp_path):
    from triune_b200.inference import load_checkpoint_model

    cfg = CONFIGS["grouped"]
    m = build(cfg, oracle.make_weights(cfg, seed=2))
    torch.save({"model_state": m.state_dict(), "config": m.model_config.to_dict()}, tmp_path / "c.pt")
    m2 = load_checkpoint_model(str(tmp_path / "c.pt"))[0]
    ids = torch.tensor([tokens(cfg, 9)])
    assert torch.equal(m(ids)[0], m2(ids)[0])


def test_trace_runner_replays_and_frees(tmp_path):
    from triune_b200.serve.trace import TraceRunner, run

    cfg = CONFIGS["grouped"]
    W = oracle.make_weights(cfg, seed=4)
    m = build(cfg, W)
    a, b = tokens(cfg, 12, 1), tokens(cfg, 8, 2)
    la, lb = oracle.forward(cfg, W, a), oracle.forward(cfg, W, b)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [0, 6]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[7:9], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[9:], "want": [2, 0]}, {"id": "b", "tokens": b, "want": [7]}], "end": ["a", "b"]}]
    out = io.StringIO()
    run(m, tmp_path, [json.dumps(x) for x in lines], out)
    assert out.getvalue().split("\n")[:4] == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "3.f32"]

    def read(i):
        return torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])

    assert rel(read(0), la[[0, 6]]) < 2e-5
    assert rel(read(3), torch.stack((la[11], la[9], lb[7]))) < 2e-5
    r = TraceRunner(m)
    r.step([{"id": "x", "tokens": a, "want": []}], ["x"])
    assert r.caches == {}


def test_trace_program_starts_and_ends(tmp_path):
    cfg = CONFIGS["odd"]
    W = oracle.make_weights(cfg, seed=4)
    folder = save_folder(cfg, W, tmp_path / "m")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    toks = tokens(cfg, 6)
    line = json.dumps({"step": 0, "entries": [{"id": "q", "tokens": toks, "want": [5]}], "end": ["q"]})
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path / "o"),
                        "--max-tokens", "64", "--device", "cpu"], input=line + "\n", capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "done 0" in r.stdout.splitlines()
    got = torch.frombuffer(bytearray((tmp_path / "o" / "0.f32").read_bytes()), dtype=torch.float32)
    assert rel(got[None], oracle.forward(cfg, W, toks)[5:6]) < 2e-5


# ---- each mechanism alone ----------------------------------------------------------------------------------------
def test_far_key_and_sink_show():
    """A query that matches one early key sees it at any distance; a large sink takes the rest of the weight."""
    from triune_b200.ops import hybrid_reference as ref

    T, D, E = 70, 8, 6
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(T, 2, D, generator=g), torch.randn(T, 1, D, generator=g), torch.randn(T, 1, E, generator=g)
    k[3, 0] = 6 * torch.nn.functional.normalize(q[-1, 1], dim=0)
    for sink in (torch.tensor([-2.0, 0.5]), torch.tensor([6.0, 9.0])):
        want = oracle.sink_attention(q.double(), k.double(), v.double(), 0.7, sink.double())
        got = ref.sink_attention(q[None], k.transpose(0, 1)[None], v.transpose(0, 1)[None], sink, 0.7, 1.0, 0, T)[0]
        assert (got.double() - want).abs().max() < 1e-5
    plain = ref.sink_attention(q[None], k.transpose(0, 1)[None], v.transpose(0, 1)[None], None, 0.7, 1.0, 0, T)[0]
    assert (plain.double() - want).abs().max() > 0.1


def test_recurrences_against_plain_scans():
    from triune_b200.ops import hybrid_reference as ref

    g = torch.Generator().manual_seed(1)
    T, H, K, D, E = 23, 6, 3, 5, 7
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v, a, b, A, bias, Dd = r(T, K, D), r(T, K, D), r(T, H, E), r(T, H), r(T, H), r(H), r(H), r(H)
    dt = oracle.softplus(a + bias)
    y, S = oracle.mamba2_scan(v, k, q, dt, A, Dd)
    st = torch.zeros(1, H, D, E, dtype=torch.float64)
    got = ref.recurrent(q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), a, None, A, bias, Dd, st, 1, T, "mamba2", 1e-6, K)
    assert (got.view(T, H, E) - y).abs().max() < 1e-8 and (st[0] - S).abs().max() < 1e-8
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    y, S = oracle.delta_scan(unit(q) * D ** -0.5, unit(k), v, torch.exp(-torch.exp(A) * dt), oracle.sigmoid(b))
    st.zero_()
    got = ref.recurrent(q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), a, b, A, bias, None, st, 1, T, "delta", 1e-6, K)
    assert (got.view(T, H, E) - y).abs().max() < 1e-8 and (st[0] - S).abs().max() < 1e-8


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolution_ring(taps):
    from triune_b200.ops import hybrid_reference as ref

    g = torch.Generator().manual_seed(2)
    T, C = 19, 5
    u, w, b = torch.randn(T, C, generator=g), torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    want = oracle.causal_conv(u.double(), w.double(), b.double())
    for cut in ([19], [1] * 19, [2, 3, 1, 13], [17, 2]):
        ring, at, out = torch.full((1, taps, C), 9.0), 0, []  # stale values: a new sequence must not see them
        for n in cut:
            y, ring = ref.causal_conv(u[at : at + n], w, b, ring, 1, n, at)
            out.append(y)
            at += n
        assert (torch.cat(out).double() - want).abs().max() < 1e-5
