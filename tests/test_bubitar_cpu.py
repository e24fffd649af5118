"""Bubitar models on the CPU: the model code, its cache and its entry points against plain statements."""

import io
import json
import math
import os

import pytest
import torch

import bubitar_oracle as oracle
from bubitar_cases import CONFIGS, YARN
from hybrid_cases import build, rel, run_portions, tokens


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def case(request):
    cfg = CONFIGS[request.param]
    W = oracle.make_weights(cfg, seed=3)
    toks = tokens(cfg, 41)
    return cfg, W, toks, oracle.forward(cfg, W, toks)


def test_whole_prompt_matches_plain_statement(case):
    cfg, W, toks, want = case
    assert rel(run_portions(build(cfg, W), toks, []), want) < 3e-5
    assert rel(run_portions(build(cfg, W, dtype=torch.float64), toks, []), want) < 1e-6


@pytest.mark.parametrize("portions", [[1] * 41, [2] * 20, [2, 3, 5, 7, 2, 11], [40], [17, 1, 1, 1, 2, 2]])
def test_portions_do_not_matter(case, portions):
    cfg, W, toks, want = case
    assert rel(run_portions(build(cfg, W), toks, portions), want) < 3e-5


def test_batch_rows_are_independent(case):
    cfg, W, toks, want = case
    m = build(cfg, W)
    other = tokens(cfg, 41, seed=9)
    lg, cache = m(torch.tensor([toks[:30], other[:30]]), cache=m.init_cache(2))
    lg2, _ = m(torch.tensor([toks[30:], other[30:]]), cache=cache)
    got = torch.cat((lg, lg2), 1)
    assert rel(got[0], want) < 3e-5
    assert rel(got[1], oracle.forward(cfg, W, other)) < 3e-5


def test_layers_of_the_residual_stream(case):
    cfg, W, toks, _ = case
    _, layers = oracle.forward(cfg, W, toks, want_layers=True)
    seen = {}
    build(cfg, W)(torch.tensor([toks]), on_layer=lambda i, x: seen.update({i: x.clone()}))
    for i, l in enumerate(layers):
        assert (seen[i].double() - l).abs().max() < 1e-4 * l.abs().max()


def test_selected_logits(case):
    cfg, W, toks, want = case
    m = build(cfg, W)
    ids = torch.tensor([toks])
    assert rel(m(ids, last_token_only=True)[0][0], want[-1:]) < 3e-5
    assert rel(m(ids, positions=[40, 3])[0][0], want[[40, 3]]) < 3e-5
    assert m(ids, positions=[])[0].shape == (1, 0, cfg["vocab"])


def test_cache_growth_keeps_the_latents():
    cfg = CONFIGS["shared"]
    W = oracle.make_weights(cfg, seed=5)
    toks = tokens(cfg, 300)
    want = oracle.forward(cfg, W, toks)
    assert rel(run_portions(build(cfg, W), toks, [250, 3, 2, 40]), want) < 3e-5


def test_layers_that_share_latents_hold_none_of_their_own():
    from triune_b200.serve.srsm import _pack, _unpack

    cfg = CONFIGS["shared"]
    m = build(cfg, oracle.make_weights(cfg, seed=1), dtype=torch.bfloat16)
    toks = tokens(cfg, 20)
    _, cache = m(torch.tensor([toks[:13]]), cache=m.init_cache(1))
    assert [s.capacity is not None for s, _ in cache] == [True, False, False, True, False]
    assert cache[2][0].nbytes() == 0 and cache[4][0].nbytes() == 0
    kept = [(s.clone(), p) for s, p in cache]
    flat, layout = _pack(cache)
    a, _ = m(torch.tensor([toks[13:]]), cache=cache)          # advances the states in place
    b, _ = m(torch.tensor([toks[13:]]), cache=kept)
    c, _ = m(torch.tensor([toks[13:]]), cache=_unpack(flat.clone(), layout))
    assert torch.equal(a, b) and torch.equal(a, c)


def test_config_round_trip_and_validation():
    from triune_b200.config import ModelConfig
    from triune_b200.models.bubitar import read_config
    from triune_b200.models.factory import build_model

    for raw in CONFIGS.values():
        cfg = read_config(raw)
        again = ModelConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))).validate()
        assert again == cfg
        exact = sum(t.numel() for t in oracle.make_weights(raw).values())
        assert cfg.param_count()[0] == exact
        assert build_model(again).num_parameters() >= exact      # alignment rows may add to it

    def broken(change):
        bad = json.loads(json.dumps(CONFIGS["shared"]))
        change(bad["layers"])
        with pytest.raises((ValueError, KeyError)):
            read_config(bad)

    broken(lambda l: l[1]["mixer"]["rot"].update(dims=7))
    broken(lambda l: l[1]["mixer"].update(decay=[0.5]))
    broken(lambda l: l[1]["mixer"]["decay"].__setitem__(0, 1.5))
    broken(lambda l: l[2]["mixer"].update(kv_from=1))            # not a latent layer
    broken(lambda l: l[2]["mixer"].update(kv_from=4))            # not an earlier one
    broken(lambda l: l[4]["mixer"].update(kv_from=2))            # has none of its own
    broken(lambda l: l[2]["mixer"].update(kv_rank=16))           # another latent
    broken(lambda l: l[2]["mixer"]["rot"].update(base=7.0))      # another rotation
    broken(lambda l: l[0].update(type="other"))
    broken(lambda l: l[0]["mlp"].update(kind="sparse"))
    broken(lambda l: l[0]["mlp"].update(limit=0))


def test_weights_that_do_not_fit_are_refused():
    from triune_b200.models import Bubitar

    cfg = CONFIGS["odd"]
    W = oracle.make_weights(cfg)
    m = Bubitar(config=cfg)
    for bad in ({k: v for k, v in W.items() if k != "l1.mix.dkv.norm"}, {**W, "l3.mix.dkv": W["l1.mix.dkv"]}, {**W, "head": W["head"][:-1]}):
        with pytest.raises(ValueError):
            m.load_named(bad)


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
        assert rel(run_portions(m, toks, [5]), want) < 3e-5
    assert "bubitar" in list_models()
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


def test_command_line_generates(tmp_path, capsys):
    from triune_b200.cli import main

    cfg = CONFIGS["odd"]
    folder = save_folder(cfg, oracle.make_weights(cfg, seed=7), tmp_path / "m")
    assert main(["infer", "--model", str(folder), "--prompt", "abc", "--raw", "--json", "--max-tokens", "3", "--temperature", "0",
                 "--device", "cpu"]) in (0, None)
    assert capsys.readouterr().out


def greedy(cfg, W, toks, n):
    out = list(toks)
    for _ in range(n):
        out.append(int(oracle.forward(cfg, W, out)[-1].argmax()))
    return out[len(toks):]


@pytest.mark.parametrize("name", ["shared", "odd"])
def test_greedy_generation(name):
    from triune_b200.inference import GraphedGreedyDecoder, generate_tokens

    cfg = CONFIGS[name]
    W = oracle.make_weights(cfg, seed=11)
    toks = tokens(cfg, 15)
    want = greedy(cfg, W, toks, 10)
    m = build(cfg, W, dtype=torch.float64)
    got, _, _ = generate_tokens(m, torch.tensor([toks]), 10, temperature=0.0, repetition_penalty=1.0, count_penalty=0.0,
                                prefill_chunk=7)
    assert got == want
    dec = GraphedGreedyDecoder(m)
    assert dec.generate(torch.tensor([toks]), 10)[0, 15:].tolist() == want
    assert dec.generate(torch.tensor([toks[:9]]), 10)[0, 9:].tolist() == greedy(cfg, W, toks[:9], 10)


def test_checkpoint_of_a_model(tmp_path):
    from triune_b200.inference import load_checkpoint_model

    cfg = CONFIGS["shared"]
    m = build(cfg, oracle.make_weights(cfg, seed=2))
    torch.save({"model_state": m.state_dict(), "config": m.model_config.to_dict()}, tmp_path / "c.pt")
    m2 = load_checkpoint_model(str(tmp_path / "c.pt"))[0]
    ids = torch.tensor([tokens(cfg, 9)])
    assert torch.equal(m(ids)[0], m2(ids)[0])


def test_trace_runner_replays_and_frees(tmp_path):
    from triune_b200.serve.trace import TraceRunner, run

    cfg = CONFIGS["shared"]
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

    assert rel(read(0), la[[0, 6]]) < 3e-5
    assert rel(read(3), torch.stack((la[11], la[9], lb[7]))) < 3e-5
    r = TraceRunner(m)
    r.step([{"id": "x", "tokens": a, "want": []}], ["x"])
    assert r.caches == {}


# ---- each mechanism alone ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("rot", [{"dims": 8, "base": 1e3}, {"dims": 16, "base": 5e5, "scaling": YARN}, {"dims": 6, "base": 100.0, "scaling": {
    "factor": 3.0, "original": 30, "fast": 2.0, "slow": 1.9}}, {"dims": 2, "base": 1e4, "scaling": YARN}])
def test_rotation(rot):
    """Turns and amplitudes at near and far positions, and the pairing of the halves."""
    from triune_b200.models.rotary import rotary_frequencies
    from triune_b200.ops import hybrid_reference as ref

    freqs, amp = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    want, wamp = oracle.rotation_table(rot)
    assert amp == pytest.approx(wamp) and torch.allclose(freqs, torch.tensor(want, dtype=torch.float64), rtol=1e-12)
    x = torch.randn(3, 2, rot["dims"] + 3, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    for pos in (0, 1, 77, 100000):
        got = ref.rotate_halves(x[None], ref.rotation_rows(freqs, amp, pos, 3, torch.float64))[0]
        assert (got - oracle.rotate_halves(x, torch.arange(pos, pos + 3), rot)).abs().max() < 1e-9


def test_yarn_borders():
    """Pairs above the fast border keep their frequency, pairs below the slow one are divided, the ramp lies between."""
    from triune_b200.models.rotary import rotary_frequencies

    scaling = {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    f, amp = rotary_frequencies(64, 1e4, scaling)
    plain, _ = rotary_frequencies(64, 1e4)
    turns = 4096 * plain / (2 * math.pi)
    ratio = plain / f
    assert torch.all(ratio[turns > 40] == 1) and torch.allclose(ratio[turns < 0.8], torch.tensor(16.0, dtype=torch.float64))
    assert torch.all(ratio[1:] >= ratio[:-1] - 1e-12) and amp == pytest.approx(0.1 * math.log(16) + 1)


def test_retention_against_the_plain_scan():
    from triune_b200.ops import hybrid_reference as ref

    g = torch.Generator().manual_seed(1)
    T, H, D, E = 23, 3, 6, 5
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, E))
    rot = {"dims": 4, "base": 50.0}
    decay = torch.tensor([0.3, 0.97, 1.0], dtype=torch.float64)
    turn = lambda x: oracle.rotate_halves(x, torch.arange(T), rot)
    y, S = oracle.retention_scan(turn(q), turn(k) * D ** -0.5, v, decay)
    st = torch.zeros(1, H, D, E, dtype=torch.float64)
    f = torch.tensor(oracle.rotation_table(rot)[0], dtype=torch.float64)
    for cut in ([23], [2, 20, 1], [1] * 23):
        st.zero_()
        at, out = 0, []
        for n in cut:
            s = slice(at, at + n)
            out.append(ref.retention(q[s].reshape(n, -1), k[s].reshape(n, -1), v[s].reshape(n, -1), ref.rotation_rows(f, 1.0, at, n, torch.float64),
                                     decay, st, 1, n))
            at += n
        assert (torch.cat(out).view(T, H, E) - y).abs().max() < 1e-10 and (st[0] - S).abs().max() < 1e-10


def test_clamped_activation():
    """Values below, at and above both limits; the gate has no lower limit."""
    from triune_b200.ops import hybrid_reference as ref

    g, u = torch.linspace(-30, 30, 121, dtype=torch.float64), torch.linspace(30, -30, 121, dtype=torch.float64)
    got = ref.gated_activation(g, u, "clamped", 1.5, 1.702)
    gc, uc = torch.clamp(g, max=1.5), torch.clamp(u, -1.5, 1.5)
    assert (got - gc * oracle.sigmoid(1.702 * gc) * (uc + 1)).abs().max() < 1e-12
    assert float(got[0]) != 0.0


def test_sum_with_a_norm_behind_the_sublayer():
    from triune_b200.ops import hybrid_reference as ref

    g = torch.Generator().manual_seed(2)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    x, y, b, w1, w2 = r(4, 10), r(4, 10), r(10), r(10), r(10)
    want = x + oracle.rms_norm(y + b, w1, 1e-3)
    got = x.clone()
    h = ref.add_norm(got, y, b, (w1, 1e-3, "rms"), (w2, 1e-5, "rms"), torch.float64)
    assert torch.allclose(got, want) and torch.allclose(h, oracle.rms_norm(want, w2, 1e-5))
    assert torch.equal(ref.add_norm(x.clone(), y, b, (w1, 1e-3, "rms"), "rows", torch.float64), got)
    assert ref.add_norm(x.clone(), y, None, (w1, 1e-3, "rms"), None, torch.float64) is None


def test_token_side():
    from triune_b200.ops import hybrid as hops

    g = torch.Generator().manual_seed(3)
    gate, table, ids = torch.randn(5, 4, generator=g), torch.randn(9, 12, generator=g), torch.tensor([8, 0, 3, 3, 1])
    want = oracle.gelu_tanh(gate.double()) * table.double()[ids][:, 4:8]
    assert (hops.token_side_hidden(gate, table, ids, 4).double() - want).abs().max() < 1e-6
