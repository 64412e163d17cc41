"""Ragenex and its parts on CPU against the float64 NumPy statement: mechanisms, caches, batches, generation, checkpoints, command line."""
import copy
import json

import numpy as np
import pytest
import torch

import ragenex_oracle as oracle
from helpers import run_tune
from tokenizer_assets import write_sentencepiece_model
from torchtune_b200 import ops
from torchtune_b200.generation import BatchDecoder, generate
from torchtune_b200.models._registry import build_from_config, load_pretrained
from torchtune_b200.models.ragenex import lora_ragenex, ragenex, ragenex_hf_to_tune, ragenex_tune_to_hf
from torchtune_b200.modules import (
    ClampedGLU,
    FeedForward,
    HyperConnectionLayer,
    LightningAttention,
    Linear,
    PassCaches,
    QueryTemperature,
    SpanAttention,
    SpanKVCache,
    StateCache,
    StreamLayerNorm,
    delete_kv_caches,
    disable_kv_cache,
    local_kv_cache,
)
from torchtune_b200.ops import reference
from torchtune_b200.ops.mask import AttentionMask

CPU = torch.device("cpu")
CONFIGS = {
    "plain": oracle.config([oracle.attention_layer(), oracle.lightning_layer(), oracle.attention_layer(heads=4, kv_heads=4, dim=40, vdim=16, ff=None, coef=1.1, every=3)]),
    "looped": oracle.config([oracle.lightning_layer(ff=None), oracle.attention_layer(heads=5, kv_heads=1, dim=16, vdim=24, scale=0.31), oracle.lightning_layer(decay=(0.8, 1.0), dim=12, vdim=8), oracle.attention_layer()],
                            loop=(1, 3, 3), streams=4, eps=1e-2),
    "loop_all": oracle.config([oracle.attention_layer(heads=2, kv_heads=1, dim=8, vdim=8, ff=24, limit=3.0), oracle.lightning_layer(decay=(0.0, 0.5), dim=8, vdim=8, ff=24)], loop=(0, 2, 2), streams=2, width=40),
    "odd": oracle.config([oracle.lightning_layer(decay=(0.9,), dim=5, vdim=7, ff=35), oracle.attention_layer(heads=3, kv_heads=3, dim=11, vdim=9, every=1, ff=22)], width=51, vocab=67, eps=1e-2, streams=1),
    "tiny": oracle.config([oracle.attention_layer(heads=1, kv_heads=1, dim=1, vdim=1, ff=1), oracle.lightning_layer(decay=(0.7,), dim=1, vdim=1, ff=None)], width=8, vocab=5, eps=1e-2, loop=(1, 2, 1)),
}


def _to_torch(w):
    return ragenex_hf_to_tune({k: torch.tensor(v, dtype=torch.float32) for k, v in w.items()})


def _build(cfg, w):
    model = build_from_config(cfg)
    model.load_state_dict(_to_torch(w))
    return model.eval()


def _model(name, seed=0, sharp=2.0):
    cfg = CONFIGS[name]
    w = oracle.weights(cfg, seed=seed, sharp=sharp)
    return cfg, w, _build(cfg, w)


def _seq(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def _t(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32)


def _assert_logits(got, want, tol=5e-4):
    np.testing.assert_allclose(got.detach().double().numpy(), want, atol=tol * max(np.abs(want).max(), 1.0), rtol=0)


# ------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("S", [1, 2, 5])
def test_stream_step(S):
    rng = np.random.default_rng(0)
    x, y, gain, mix, out, read, w = rng.normal(size=(7, S, 20)), rng.normal(size=(7, 20)), rng.normal(size=20), rng.normal(size=(S, S)), rng.normal(size=S), rng.normal(size=S), rng.normal(size=20)
    want = oracle.write_streams(x, mix, out, gain * y)
    a, h = ops.stream_step(_t(x), _t(y), _t(gain), _t(mix), _t(out), _t(read), _t(w), eps=0.03, centered=True)
    np.testing.assert_allclose(a.numpy(), want, atol=1e-5)
    np.testing.assert_allclose(h.numpy(), oracle.layer_norm(oracle.read_streams(want, read), w, 0.03), atol=2e-5)
    a1, _ = ops.stream_step(_t(x[:, :1]), _t(y), _t(gain), _t(mix), _t(out), None, None, eps=0.0, centered=True)
    np.testing.assert_allclose(a1.numpy(), oracle.write_streams(np.repeat(x[:, :1], S, 1), mix, out, gain * y), atol=1e-5)
    _, total = ops.stream_step(_t(x), _t(y), _t(gain), _t(mix), _t(out), None, _t(w), eps=0.03, centered=False, offset=1.0)
    np.testing.assert_allclose(total.numpy(), oracle.rms_norm(want.sum(1), 1.0 + w, 0.03), atol=2e-5)
    norm = StreamLayerNorm(20, eps=0.03)
    norm.load_state_dict({"scale": _t(w)})
    np.testing.assert_allclose(norm(_t(y)).detach().numpy(), oracle.layer_norm(y, w, 0.03), atol=2e-6)


def test_bf16_weights_keep_the_streams_in_fp32():
    b = lambda *n: torch.randn(*n).bfloat16()  # noqa: E731
    x, y, gain, mix, out, read, w = torch.randn(3, 2, 16), b(3, 16), b(16), b(2, 2), b(2), b(2), b(16)
    a, h = ops.stream_step(x, y, gain, mix, out, read, w, eps=1e-6, centered=True)
    d = lambda t: t.double().numpy()  # noqa: E731
    assert a.dtype == torch.float32 and h.dtype == torch.bfloat16
    np.testing.assert_allclose(a.numpy(), oracle.write_streams(d(x), d(mix), d(out), d(gain) * d(y)), atol=1e-5)


def test_query_temperature():
    pos = [0, 3, 4, 5, 8, 9, 1000, 100_000]
    for every in (1, 5):
        np.testing.assert_allclose(QueryTemperature(0.7, every)(torch.tensor(pos)).numpy(), [oracle.temperature(p, 0.7, every) for p in pos], rtol=1e-6)
    with pytest.raises(ValueError):
        QueryTemperature(0.1, 2.5)


@pytest.mark.parametrize("first", [0, 3])
@pytest.mark.parametrize("heads,groups", [(6, 2), (3, 1), (4, 4)])
def test_attention_statement(first, heads, groups):
    rng = np.random.default_rng(2)
    d, dv, n = 5, 7, 9
    s = n - first
    q, k, v = rng.normal(size=(s, heads * d)), rng.normal(size=(n, groups * d)), rng.normal(size=(n, groups * dv))
    visible = torch.arange(n)[None, :] <= first + torch.arange(s)[:, None]
    got = reference.span_attention(_t(q).view(1, s, heads, d), _t(k).view(1, n, groups, d), _t(v).view(1, n, groups, dv), visible[None], 0.6)
    np.testing.assert_allclose(got[0].reshape(s, -1).numpy(), oracle.causal_attention(q, k, v, heads, groups, 0.6, first), atol=1e-5)


@pytest.mark.parametrize("chunk", [1, 4, 16, 64])
def test_lightning_statement(chunk):
    rng = np.random.default_rng(3)
    H, d, dv, s, decay = 4, 6, 5, 37, (0.3, 0.99, 1.0, 0.0)
    q, k, v, state = rng.normal(size=(s, H, d)), rng.normal(size=(s, H, d)), rng.normal(size=(s, H, dv)), rng.normal(size=(H, d, dv))
    for before in (None, state):
        want, after = oracle.decayed_recurrence(q, k, v, decay, before)
        got, st = reference.lightning_attention(_t(q)[None], _t(k)[None], _t(v)[None], decay, None if before is None else _t(before)[None], chunk)
        np.testing.assert_allclose(got[0].numpy(), want, atol=2e-4)
        np.testing.assert_allclose(st[0].numpy(), after, atol=2e-4)


def test_gated_norm_and_clamped_gate():
    rng = np.random.default_rng(4)
    o, g, z = rng.normal(size=(5, 12)), rng.normal(size=12), rng.normal(size=(5, 12))
    np.testing.assert_allclose(reference.gated_norm(_t(o), _t(g), _t(z), 0.02).numpy(), oracle.gated_norm(o, g, z, 0.02), atol=1e-6)
    a, b = 3.0 * rng.normal(size=(2, 50))
    for limit in (0.5, 2.0):
        np.testing.assert_allclose(ops.clamped_glu(_t(a), _t(b), limit, 1.702).numpy(), oracle.clamped_glu(a, b, limit), atol=1e-6)
    with pytest.raises(ValueError):
        FeedForward(gate_proj=Linear(4, 4, bias=False), down_proj=Linear(4, 4, bias=False), activation=ClampedGLU(1.0))


def test_positions_are_added_in_fp32():
    table, pos_table = torch.randn(9, 6).bfloat16(), torch.randn(5, 6).bfloat16()
    ids, pos = torch.tensor([[0, 8, 3]]), torch.tensor([[4, 0, 2]], dtype=torch.int32)
    x = ops.embed_positions(ids, pos, table, pos_table)
    assert x.dtype == torch.float32 and torch.equal(x, table.float()[ids] + pos_table.float()[pos.long()])


# ------------------------------------------------------------------------------------------ whole model
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt(name):
    cfg, w, model = _model(name)
    s = _seq(cfg, 21)
    want, after = oracle.forward(cfg, w, s, return_layers=True)
    assert [i for i, _ in model.run_order()] == oracle.run_order(cfg) and len(after) == len(oracle.run_order(cfg))
    model.output_hidden_states = list(range(len(after) + 1))
    *hidden, logits = model(torch.tensor([s]))
    _assert_logits(logits[0], want)
    for x, e in zip(hidden[1:], after):
        assert x.dtype == torch.float32
        _assert_logits(x[0], e)
    model.output_hidden_states = []
    _assert_logits(model(torch.tensor([s[:1]]))[0], want[:1])


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [(1,) * 17, (16, 1), (2, 2, 13), (7, 2, 8), (15, 2)])
def test_prompt_in_pieces_and_token_by_token(name, cuts):
    cfg, w, model = _model(name)
    s = _seq(cfg, sum(cuts), seed=3)
    want = oracle.forward(cfg, w, s)
    model.setup_caches(1, torch.float32, decoder_max_seq_len=20)
    for again in (False, True):  # the second time on slots and states that were used before
        at = 0
        for n in cuts:
            dense = torch.arange(20)[None, None, :] <= torch.arange(at, at + n)[None, :, None]
            got = model(torch.tensor([s[at : at + n]]), mask=AttentionMask(causal=True) if again else dense, input_pos=torch.arange(at, at + n)[None])
            _assert_logits(got[0], want[at : at + n])
            at += n
        model.reset_caches()


@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_rows_together(name):
    cfg, w, model = _model(name)
    seqs = [_seq(cfg, n, seed=n) for n in (15, 4, 9, 7)]
    cut = [11, 1, 8, 7]
    want = [oracle.forward(cfg, w, s) for s in seqs]
    dec = BatchDecoder(model, CPU, torch.float32, 60)
    for _ in range(2):  # rows, slots and states used again
        h = dec.begin([s[:n] for s, n in zip(seqs, cut)])
        for k in range(4):
            _assert_logits(dec.logits(h[k, h.shape[1] - cut[k] :]), want[k][: cut[k]])
        live, at = [0, 1, 2, 3], list(cut)
        while True:
            gone = [i for i, k in enumerate(live) if at[k] == len(seqs[k])]
            dec.end(gone)
            live = [k for i, k in enumerate(live) if i not in gone]
            if not live:
                break
            h = dec.advance([seqs[k][at[k]] for k in live])
            for i, k in enumerate(live):
                _assert_logits(dec.logits(h[i]), want[k][at[k] : at[k] + 1])
                at[k] += 1
    assert dec.rows == 0


def test_padded_rows_in_pieces():
    """A padded batch cut so that a whole piece of the shorter row is padding: nothing of it stays in the state."""
    cfg, w, model = _model("looped")
    a, b = _seq(cfg, 12), _seq(cfg, 5, seed=2)
    want = [oracle.forward(cfg, w, s) for s in (a, b)]
    rows = torch.tensor([a, [3] * 7 + b])
    start = torch.tensor([0, 7], dtype=torch.int32)
    model.setup_caches(2, torch.float32, decoder_max_seq_len=12)
    at, got = 0, []
    for n in (4, 1, 1, 3, 3):
        slots = torch.arange(at, at + n)
        got.append(model(rows[:, at : at + n], mask=AttentionMask(causal=True, key_start=start, query_start=at), input_pos=(slots[None] - start[:, None]).clamp_min(0)))
        at += n
    got = torch.cat(got, 1)
    _assert_logits(got[0], want[0])
    _assert_logits(got[1, 7:], want[1])


def test_long_decoding():
    cfg, w, model = _model("looped")
    s = _seq(cfg, 90, seed=8)
    want = oracle.forward(cfg, w, s)
    dec = BatchDecoder(model, CPU, torch.float32, 90)
    h = [dec.begin([s[:3]])[0]] + [dec.advance([t])[0] for t in s[3:]]
    _assert_logits(dec.logits(torch.cat(h)), want)
    with pytest.raises(AssertionError, match="full"):
        dec.advance([1])


def test_position_limit():
    cfg = oracle.config([oracle.attention_layer()], max_positions=6)
    w = oracle.weights(cfg)
    model = _build(cfg, w)
    s = _seq(cfg, 6)
    _assert_logits(model(torch.tensor([s]))[0], oracle.forward(cfg, w, s))
    dec = BatchDecoder(model, CPU, torch.float32, 20)
    dec.begin([s[:5], s[:2]])
    dec.advance(s[:2])
    with pytest.raises(ValueError, match="6 positions"):
        dec.advance(s[:2])
    dec.end([0])
    for _ in range(3):  # the shorter row goes on: positions count from its own first token, although its slots are beyond the table
        dec.advance([1])
    dec.end([0])
    with pytest.raises(ValueError, match="6 positions"):
        dec.begin([s + s])
    with pytest.raises(ValueError, match="6 positions"):
        generate(model, torch.tensor(s[:4]) + 1, max_generated_tokens=4)
    assert build_from_config(cfg, max_seq_len=4).max_seq_len == 4 and build_from_config(cfg, max_seq_len=400).max_seq_len == 6


def test_a_far_key_that_stands_out():
    """A sharp query follows the first token however far it is; the temperature makes it sharper with the distance."""
    cfg = oracle.config([oracle.attention_layer(heads=1, kv_heads=1, dim=8, vdim=16, ff=None, scale=1.0, coef=1.0, every=16)], width=24, vocab=12, streams=2, max_positions=130)
    w = oracle.weights(cfg, seed=5, sharp=3.0)
    w["pos"] = w["pos"] * 0.0
    first = {t: oracle.forward(cfg, w, [t] + [5] * 120) for t in range(12)}
    moved = max(first, key=lambda t: np.abs(first[t][-1] - first[5][-1]).max())  # the most visible far key
    assert np.abs(first[moved][-1] - first[5][-1]).max() > 0.5
    cold = oracle.forward({**cfg, "layers": [oracle.attention_layer(heads=1, kv_heads=1, dim=8, vdim=16, ff=None, scale=1.0, coef=0.0)]}, w, [moved] + [5] * 120)
    assert np.abs(cold[-1] - first[moved][-1]).max() > 0.05
    for token in (5, moved):
        seq = [token] + [5] * 120
        model = _build(cfg, w)
        _assert_logits(model(torch.tensor([seq]))[0], first[token])
        dec = BatchDecoder(model, CPU, torch.float32, 130)
        dec.begin([seq[:100]])
        h = [dec.advance([t])[0] for t in seq[100:]]
        _assert_logits(dec.logits(torch.cat(h)), first[token][100:])


def test_a_far_token_in_the_state():
    """With a slow decay the first token still shows after many others, in the prompt and in decoding; with a fast one it does not."""
    for decay, visible in ((1.0, True), (0.5, False)):
        cfg = oracle.config([oracle.lightning_layer(decay=(decay,), dim=8, vdim=16, ff=None)], width=24, vocab=12, streams=2)
        w = oracle.weights(cfg, seed=5)
        w["pos"], w["l0.mix.q"] = w["pos"] * 0.0, w["l0.mix.q"] * 3.0
        a, b = ([t] * 10 + [5] * 60 for t in (3, 5))
        want = oracle.forward(cfg, w, a)
        assert (np.abs(want[-1] - oracle.forward(cfg, w, b)[-1]).max() > 0.05) == visible
        model = _build(cfg, w)
        _assert_logits(model(torch.tensor([a]))[0], want)
        dec = BatchDecoder(model, CPU, torch.float32, 70)
        h = [dec.begin([a[:12]])[0]] + [dec.advance([t])[0] for t in a[12:]]
        _assert_logits(dec.logits(torch.cat(h)), want)


def test_every_pass_has_its_own_cache():
    """The passes of a looped layer see different inputs: with one shared cache or state decoding would differ."""
    cfg, w, model = _model("looped")
    model.setup_caches(1, torch.float32, decoder_max_seq_len=8)
    s = _seq(cfg, 8)
    model(torch.tensor([s]), mask=AttentionMask(causal=True), input_pos=torch.arange(8)[None])
    counts = [len(list(layer.attn.kv_cache)) for layer in model.layers]
    assert counts == [1, 3, 3, 1]
    keys = [c.k for c in model.layers[1].attn.kv_cache]
    states = [c.state for c in model.layers[2].attn.kv_cache]
    for a in (keys, states):
        assert (a[0] - a[1]).abs().max() > 0.1 and (a[1] - a[2]).abs().max() > 0.1
    with pytest.raises(RuntimeError, match="once caches exist"):
        model.set_loop(0, 1, 2)


def test_loop_is_checked():
    from torchtune_b200.models.llama3 import llama3

    model = llama3(vocab_size=16, num_layers=2, num_heads=2, num_kv_heads=1, embed_dim=16, max_seq_len=8)
    with pytest.raises(ValueError, match="cannot run several times"):
        model.set_loop(0, 1, 2)
    with pytest.raises(ValueError, match="cannot run"):
        model.set_loop(1, 3, 2)
    assert model.run_order() == [(0, 0), (1, 0)]


# ------------------------------------------------------------------------------------------ masks and caches
def test_masks_that_say_the_same_agree():
    cfg, w, model = _model("plain")
    s = torch.tensor([_seq(cfg, 12)])
    want = model(s)
    dense = torch.tril(torch.ones(12, 12, dtype=torch.bool))[None]
    for mask in (dense, dense[:, None], AttentionMask(causal=True), AttentionMask(causal=True, key_start=torch.tensor([0], dtype=torch.int32)), AttentionMask(causal=False, bool_mask=dense)):
        assert torch.allclose(model(s, mask=mask), want, atol=1e-5)
    with pytest.raises(ValueError, match="whole rows"):
        model(s, mask=AttentionMask(causal=True, window=4))
    with pytest.raises(ValueError, match="whole rows"):
        model(s, mask=dense & (torch.arange(12)[None, :] != 3))


def test_caches():
    kv = SpanKVCache(3, 4, 1, 2, 3, torch.float32)
    kv.k.copy_(torch.arange(24.0).view(3, 4, 1, 2))
    kv.v.copy_(torch.arange(36.0).view(3, 4, 1, 3))
    kv.advance(2)
    k, v = kv.k.clone(), kv.v.clone()
    kv.keep_rows([1, 2])
    assert torch.equal(kv.k[0, :2], k[1, :2]) and torch.equal(kv.v[1, :2], v[2, :2])
    assert kv.reserve(3, 2) == 2
    with pytest.raises(AssertionError):
        kv.reserve(1, 3)
    with pytest.raises(ValueError):
        kv.reserve(4, 1)
    st = StateCache(3, 4, 1, 2, 3)
    assert st.state.dtype == torch.float32
    st.state.copy_(torch.arange(18.0).view(3, 1, 2, 3))
    st.advance(3)
    saved, before = st.snapshot(), st.state.clone()
    st.state.mul_(2)
    st.advance(1)
    with pytest.raises(ValueError, match="forget"):
        st.rewind(2)
    st.restore(saved)
    assert st.size == 3 and torch.equal(st.state, before)
    st.keep_rows([2])
    assert torch.equal(st.state[0], before[2])
    both = PassCaches([SpanKVCache(1, 4, 1, 2, 2, torch.float32), SpanKVCache(1, 4, 1, 2, 2, torch.float32)])
    both.advance(2)
    both.slot = torch.tensor([2])
    assert [c.size for c in both] == [2, 2] and both[1].slot is both.slot and both.size == 2 and both.reserve(1, 2) == 2
    saved = both.snapshot()
    both.rewind(1)
    both.restore(saved)
    assert both[1].size == 2
    both.reset()
    assert both[0].size == both[1].size == 0


def test_cache_utilities():
    cfg, w, model = _model("looped")
    s = torch.tensor([_seq(cfg, 6)])
    want = model(s)
    args = dict(mask=AttentionMask(causal=True), input_pos=torch.arange(6)[None])
    with local_kv_cache(model, batch_size=1, device=CPU, dtype=torch.float32, decoder_max_seq_len=8):
        assert model.caches_are_enabled()
        with disable_kv_cache(model):
            assert torch.allclose(model(s), want, atol=1e-5)
        assert torch.allclose(model(s, **args), want, atol=1e-5)
        assert all(layer.attn.kv_cache.size == 6 for layer in model.layers)
    assert not model.caches_are_setup()
    model.setup_caches(1, torch.float32, decoder_max_seq_len=8)
    model.load_state_dict(model.state_dict())  # joined projection weights stay the model's parameters
    assert torch.allclose(model(s, **args), want, atol=1e-5)
    delete_kv_caches(model)


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("cached", [True, False])
def test_greedy_generation(cached):
    cfg, w, model = _model("looped")
    prompts = [[t or 1 for t in p] for p in (_seq(cfg, 6, seed=1), _seq(cfg, 3, seed=2))]  # 0 is the padding
    want = [oracle.greedy(cfg, w, p, 5) for p in prompts]
    batch = torch.tensor([prompts[0], [0, 0, 0] + prompts[1]])
    if cached:
        model.setup_caches(2, torch.float32, decoder_max_seq_len=12)
    out, logits = generate(model, batch, max_generated_tokens=5, pad_id=0, top_k=1)
    assert out[0].tolist() == want[0] and out[1, 3:].tolist() == want[1] and logits.shape == (2, 5, cfg["vocab"])
    if cached:
        model.reset_caches()
        one, _ = generate(model, torch.tensor(prompts[1]), max_generated_tokens=5, pad_id=0, top_k=1, stop_tokens=[want[1][4]])
        assert one[0].tolist() == want[1][:5]


def test_single_conversation_decoder():
    from torchtune_b200.engine.inference import CachedDecoder

    cfg, w, model = _model("plain")
    prompt = _seq(cfg, 5)
    model.setup_caches(1, torch.float32, decoder_max_seq_len=12)
    dec = CachedDecoder(model, CPU, 12, 1.0, 1, [])
    with torch.inference_mode():
        assert prompt + dec.run(torch.tensor([prompt]), 4) == oracle.greedy(cfg, w, prompt, 4)


def test_generate_recipe(tmp_path, tune_path, monkeypatch, caplog):
    cfg = oracle.config([oracle.attention_layer(), oracle.lightning_layer()], vocab=200, loop=(0, 2, 2))
    folder = oracle.save(tmp_path / "ckpt", cfg, oracle.weights(cfg))
    (tmp_path / "tok").mkdir()
    sp = write_sentencepiece_model(tmp_path / "tok", vocab_size=200)
    run_tune(tune_path, f"run generate --config ragenex/generation checkpoint_dir={folder} output_dir={tmp_path / 'out'} device=cpu dtype=fp32 "
                        f"tokenizer.path={sp} max_new_tokens=6 prompt.user=hello top_k=1", monkeypatch)
    assert "tokens/sec" in caplog.text


# ------------------------------------------------------------------------------------------ configuration and weights
def test_checkpoint_round_trip(tmp_path):
    from torchtune_b200 import training

    cfg = CONFIGS["looped"]
    w = oracle.weights(cfg, seed=9)
    folder = oracle.save(tmp_path / "a", cfg, w)
    ck = training.FullModelHFCheckpointer(str(folder), ["model.safetensors"], "RAGENEX", output_dir=str(tmp_path / "out"))
    sd = ck.load_checkpoint()["model"]
    back = ragenex_tune_to_hf(sd)
    assert set(back) == set(w) and all(np.array_equal(back[k].double().numpy(), w[k]) for k in w)
    model = load_pretrained(folder, dtype=torch.float32, device=CPU, max_seq_len=64)
    assert not model.training and type(model.layers[0]) is HyperConnectionLayer and set(model.state_dict()) == set(sd)
    assert type(model.layers[0].attn) is LightningAttention and type(model.layers[1].attn) is SpanAttention and model.span_masks
    s = _seq(cfg, 8)
    _assert_logits(model(torch.tensor([s]))[0], oracle.forward(cfg, w, s))
    ck.save_checkpoint({"model": model.state_dict()}, epoch=0)
    again = load_pretrained(tmp_path / "out" / "epoch_0", dtype=torch.float32, device=CPU)
    assert torch.equal(again(torch.tensor([s])), model(torch.tensor([s])))
    with pytest.raises(ValueError, match="unexpected tensor"):
        ragenex_hf_to_tune({"l0.mix.z": torch.zeros(1)})
    extra = {**w, "l0.norm2": w["l0.norm1"], "l0.hc2.in": w["l0.hc1.in"]}  # layer 0 has no feed-forward block
    more = load_pretrained(oracle.save(tmp_path / "b", cfg, extra), dtype=torch.float32, device=CPU)
    assert torch.equal(more(torch.tensor([s])), model(torch.tensor([s])))


def test_configuration_is_checked(tmp_path):
    good = CONFIGS["looped"]
    path = tmp_path / "config.json"
    path.write_text(json.dumps(good))
    with torch.device("meta"):
        assert len(ragenex(config=str(path)).layers) == 4 and len(ragenex(config=str(tmp_path)).layers) == 4

    def bad(change, match):
        cfg = copy.deepcopy(good)
        change(cfg)
        with pytest.raises(ValueError, match=match), torch.device("meta"):
            ragenex(config=cfg)

    bad(lambda c: c["layers"][0].update(type="conv"), "mixer type")
    bad(lambda c: c["layers"][1].update(mlp={"kind": "experts", "ff": 8}), "feed-forward kind")
    bad(lambda c: c["layers"][1]["mixer"].update(kv_heads=2), "evenly")
    bad(lambda c: c["layers"][0]["mixer"].update(heads=4), "decays")
    bad(lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 1.5, 0.1]), "between 0 and 1")
    bad(lambda c: c.update(streams=-1), "streams")
    bad(lambda c: c["loop"].update(stop=9), "outside")
    without = {k: v for k, v in good.items() if k != "loop"}
    assert ragenex(config=without).run_order() == ragenex(config={**good, "loop": None}).run_order() == [(i, 0) for i in range(4)]


def test_adapters_and_gradients():
    """Adapters attach to the named projections and train; the adapted model decodes like its full forward."""
    cfg = CONFIGS["looped"]
    model = lora_ragenex(["q_proj", "k_proj", "v_proj", "gate_proj", "output_proj"], True, config=cfg, max_seq_len=64, lora_rank=4, lora_alpha=8)
    for p in model.parameters():
        p.data = torch.randn_like(p) * 0.1
    names = [n for n, _ in model.named_parameters() if "lora_a" in n]
    assert any("layers.0.attn.gate_proj" in n for n in names) and not any("layers.1.attn.gate_proj" in n for n in names) and any("layers.1.mlp.w1" in n for n in names)
    s = torch.tensor([_seq(cfg, 7)])
    full = model(s)
    full.sum().backward()
    for n, p in model.named_parameters():
        assert p.grad is not None and torch.isfinite(p.grad).all(), n
    assert model.layers[0].attn.gate_proj.lora_a.weight.grad.abs().sum() > 0 and model.layers[1].sa_streams.mix.grad.abs().sum() > 0
    with torch.no_grad():
        model.setup_caches(1, torch.float32, decoder_max_seq_len=7)
        parts = [model(s[:, i : i + 1], mask=AttentionMask(causal=True), input_pos=torch.tensor([[i]])) for i in range(7)]
    assert torch.allclose(torch.cat(parts, 1), full, atol=1e-4)
    with pytest.raises(ValueError, match="unknown attention modules"):
        lora_ragenex(["kv_down"], config=cfg, lora_rank=4, lora_alpha=8)


def test_trace_replay_bookkeeping(tmp_path):
    """Names, wanted places and ended requests, on CPU."""
    from torchtune_b200.generation.trace import TraceReplay

    cfg, w, model = _model("looped")
    seqs = {"p": _seq(cfg, 9), "q": _seq(cfg, 5, seed=1)}
    want = {k: oracle.forward(cfg, w, v) for k, v in seqs.items()}
    replay = TraceReplay(BatchDecoder(model, CPU, torch.float32, 30), tmp_path)
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])  # noqa: E731
    with torch.inference_mode():
        replay.run({"step": 0, "entries": [{"id": "q", "tokens": seqs["q"][:4], "want": [3, 0]}, {"id": "p", "tokens": seqs["p"][:7], "want": [2]}], "end": []})
        _assert_logits(torch.tensor(read(0)), np.stack([want["q"][3], want["q"][0], want["p"][2]]))
        replay.run({"step": 1, "entries": [{"id": "p", "tokens": seqs["p"][7:8], "want": []}, {"id": "q", "tokens": seqs["q"][4:], "want": [0]}], "end": ["q"]})
        _assert_logits(torch.tensor(read(1)), want["q"][4:])
        replay.run({"step": 2, "entries": [{"id": "p", "tokens": seqs["p"][8:], "want": [0]}], "end": ["p"]})
        _assert_logits(torch.tensor(read(2)), want["p"][8:])
        replay.run({"step": 3, "entries": [{"id": "q", "tokens": seqs["q"], "want": [4]}], "end": ["q"]})
        _assert_logits(torch.tensor(read(3)), want["q"][4:])
