"""Begapel and its parts on CPU against the float64 NumPy statement: mechanisms, caches, batches, generation, checkpoints, command line."""
import copy
import json

import numpy as np
import pytest
import torch

import begapel_oracle as oracle
from helpers import run_tune
from tokenizer_assets import write_sentencepiece_model
from torchtune_b200 import ops
from torchtune_b200.generation import BatchDecoder, RowLayout, generate
from torchtune_b200.models._registry import architecture_of, build_from_config, load_pretrained
from torchtune_b200.models.begapel import begapel, begapel_hf_to_tune, begapel_tune_to_hf, lora_begapel
from torchtune_b200.modules import LatentCache, ResidualStreamLayer, StreamRMSNorm, delete_kv_caches, disable_kv_cache, local_kv_cache
from torchtune_b200.modules.latent_attention import PreciseRotaryPositionalEmbeddings
from torchtune_b200.ops import reference
from torchtune_b200.ops.mask import AttentionMask

CPU = torch.device("cpu")
CONFIGS = {
    "plain": oracle.config([oracle.layer(), oracle.layer(heads=2, dim=40, rot=16, vdim=24, rank=64, ff=None)]),
    "shared": oracle.config([oracle.layer(ff=None), oracle.layer(kv_from=0, heads=5, dim=16, vdim=32, scale=0.31), oracle.layer(rank=80, base=77.0), oracle.layer(kv_from=2, rank=80, base=77.0),
                             oracle.layer(kv_from=0)], width=104, mult=1.0, cap=3.0),
    "odd": oracle.config([oracle.layer(heads=3, dim=10, rot=6, vdim=7, rank=21, ff=35), oracle.layer(kv_from=0, heads=1, dim=5, rot=6, vdim=9, rank=21, ff=22)], width=51, vocab=67, eps=1e-2),
    "one_head": oracle.config([oracle.layer(heads=1, dim=1, rot=2, vdim=1, rank=1, ff=1)], width=8, vocab=5),
}


def _to_torch(w):
    return begapel_hf_to_tune({k: torch.tensor(v, dtype=torch.float32) for k, v in w.items()})


def _build(cfg, w):
    model = build_from_config(cfg, max_seq_len=256)
    model.load_state_dict(_to_torch(w))
    return model.eval()


def _model(name, seed=0, sharp=2.0):
    cfg = CONFIGS[name]
    w = oracle.weights(cfg, seed=seed, sharp=sharp)
    return cfg, w, _build(cfg, w)


def _seq(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def _assert_logits(got, want, tol=2e-4):
    np.testing.assert_allclose(got.detach().double().numpy(), want, atol=tol * max(np.abs(want).max(), 1.0), rtol=0)


# ------------------------------------------------------------------------------------------ mechanisms
def test_stream_norm_and_residual_step():
    rng = np.random.default_rng(0)
    x, y, g, n = rng.normal(size=(4, 6, 20)), 0.05 * rng.normal(size=(4, 6, 20)), rng.normal(size=20), rng.normal(size=20)
    t = lambda a: torch.tensor(a, dtype=torch.float32)  # noqa: E731
    for offset in (0.0, 1.0):
        a, h = ops.residual_norm(t(x), t(y), t(g), t(n), eps=0.03, mult=0.4, offset=offset)
        want = x + 0.4 * oracle.rms_norm(y, g, 0.03, offset)
        np.testing.assert_allclose(a.numpy(), want, atol=1e-6)
        np.testing.assert_allclose(h.numpy(), oracle.rms_norm(want, n, 0.03, offset), atol=2e-6)
    norm, post = StreamRMSNorm(20, eps=0.03, zero_centered=True), StreamRMSNorm(20, eps=0.03, zero_centered=True)
    assert not norm.scale.any() and not post.scale.any()
    norm.load_state_dict({"scale": t(n)})
    post.load_state_dict({"scale": t(g)})
    np.testing.assert_allclose(norm(t(x)).detach().numpy(), oracle.rms_norm(x, n, 0.03, 1.0), atol=2e-6)
    a, h = StreamRMSNorm.chain(t(x), t(y), post, 0.4, norm)
    np.testing.assert_allclose(a.detach().numpy(), oracle.residual_step(x, y, g, 0.03, 0.4), atol=1e-6)
    other = StreamRMSNorm(20, eps=0.5)  # another eps and offset in front of the next sublayer
    a2, h2 = StreamRMSNorm.chain(t(x), t(y), post, 0.4, other)
    assert torch.equal(a, a2)
    np.testing.assert_allclose(h2.detach().numpy(), oracle.rms_norm(a.detach().double().numpy(), np.ones(20), 0.5, 0.0), atol=2e-6)
    assert torch.equal(StreamRMSNorm.chain(t(x), t(y), post, 0.4, None)[0], a) and StreamRMSNorm.chain(t(x), t(y), post, 0.4, None)[1] is None


def test_a_bf16_gain_keeps_the_stream_in_fp32():
    x, y = torch.randn(3, 16), torch.randn(3, 16).bfloat16()
    g = torch.randn(16).bfloat16()
    a, h = ops.residual_norm(x, y, g, g, eps=1e-6, mult=0.5, offset=1.0)
    assert a.dtype == torch.float32 and h.dtype == torch.bfloat16
    np.testing.assert_allclose(a.numpy(), oracle.residual_step(x.double().numpy(), y.double().numpy(), g.double().numpy(), 1e-6, 0.5), atol=1e-6)


def test_rotation_table():
    z = np.random.default_rng(1).normal(size=(5, 2, 12))
    pos = [0, 3, 17, 120, 255]
    rope = PreciseRotaryPositionalEmbeddings(8, 256, 50.0)
    got = reference.rope_interleaved(torch.tensor(z[None, ..., :8], dtype=torch.float32), rope.cache, torch.tensor([pos]))
    np.testing.assert_allclose(got[0].numpy(), oracle.rotate_pairs(z, pos, 8, 50.0)[..., :8], atol=1e-6)
    assert rope.cache.dtype == torch.float32
    with torch.device("meta"):
        PreciseRotaryPositionalEmbeddings(8, 256, 50.0)


@pytest.mark.parametrize("first", [0, 3])
def test_attention_statement(first):
    rng = np.random.default_rng(2)
    H, d, r, dv, rank, n, s = 3, 5, 4, 6, 7, 9, 9 - first
    q, c, kr = rng.normal(size=(s, H, d + r)), rng.normal(size=(n, rank)), rng.normal(size=(n, r))
    uk, uv = rng.normal(size=(H * d, rank)), rng.normal(size=(H * dv, rank))
    t = lambda a: torch.tensor(a, dtype=torch.float32)[None]  # noqa: E731
    visible = torch.arange(n)[None, :] <= first + torch.arange(s)[:, None]
    got = reference.latent_attention(t(q), t(c @ uk.T).view(1, n, H, d), t(kr), t(c @ uv.T).view(1, n, H, dv), visible[None], 0.6)
    np.testing.assert_allclose(got[0].reshape(s, H * dv).numpy(), oracle.causal_latent_attention(q, c, kr, uk, uv, H, d, dv, 0.6, first), atol=1e-5)


def test_partial_rotation_of_the_rotated_part():
    """A rotation over fewer dimensions than the rotated part leaves the rest as it is."""
    cfg = oracle.config([oracle.layer(rot=12, rot_dims=4)])
    w = oracle.weights(cfg)
    s = _seq(cfg, 12)
    _assert_logits(_build(cfg, w)(torch.tensor([s]))[0], oracle.forward(cfg, w, s))


# ------------------------------------------------------------------------------------------ whole model
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt(name):
    cfg, w, model = _model(name)
    s = _seq(cfg, 21)
    want, streams = oracle.forward(cfg, w, s, return_layers=True)
    n = len(cfg["layers"])
    model.output_hidden_states = list(range(n + 1))
    *hidden, logits = model(torch.tensor([s]))
    _assert_logits(logits[0], want)
    for i, x in enumerate(streams):
        assert hidden[i + 1].dtype == torch.float32
        _assert_logits(hidden[i + 1][0], x)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [(1,) * 17, (16, 1), (2, 2, 13), (7, 2, 8), (15, 2)])
def test_prompt_in_pieces_and_token_by_token(name, cuts):
    cfg, w, model = _model(name)
    s = _seq(cfg, sum(cuts), seed=3)
    want = oracle.forward(cfg, w, s)
    model.setup_caches(1, torch.float32, decoder_max_seq_len=20)
    for again in (False, True):  # the second time on slots that were used before
        at = 0
        for n in cuts:
            dense = torch.arange(20)[None, None, :] <= torch.arange(at, at + n)[None, :, None]
            got = model(torch.tensor([s[at : at + n]]), mask=AttentionMask(causal=True) if again else dense, input_pos=torch.arange(at, at + n)[None])
            _assert_logits(got[0], want[at : at + n])
            at += n
        model.reset_caches()


@pytest.mark.parametrize("name", ["plain", "shared", "odd"])
def test_unequal_rows_together(name):
    cfg, w, model = _model(name)
    seqs = [_seq(cfg, n, seed=n) for n in (15, 4, 9, 7)]
    cut = [11, 1, 8, 7]
    want = [oracle.forward(cfg, w, s) for s in seqs]
    dec = BatchDecoder(model, CPU, torch.float32, 60)
    for _ in range(2):  # rows and slots used again
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


def test_long_decoding():
    cfg, w, model = _model("shared")
    s = _seq(cfg, 90, seed=8)
    want = oracle.forward(cfg, w, s)
    dec = BatchDecoder(model, CPU, torch.float32, 90)
    h = [dec.begin([s[:3]])[0]] + [dec.advance([t])[0] for t in s[3:]]
    _assert_logits(dec.logits(torch.cat(h)), want)
    with pytest.raises(AssertionError, match="full"):
        dec.advance([1])


def test_a_short_row_may_outlive_a_long_one():
    """Slots are bounded by the longest prompt plus what the last row may still grow, not by the longest sequence."""
    cfg, w, model = _model("plain")
    dec = BatchDecoder(model, CPU, torch.float32, 24)
    long, short = _seq(cfg, 20), _seq(cfg, 23, seed=4)
    dec.begin([long, short[:1]])
    dec.end([0])
    h = [dec.advance([t])[0] for t in short[1:]]
    _assert_logits(dec.logits(torch.cat(h)), oracle.forward(cfg, w, short)[1:])


def test_a_far_key_that_stands_out():
    """Sharp scores over two kinds of tokens: the answer follows the first token however far it is."""
    cfg = oracle.config([oracle.layer(heads=1, dim=8, rot=2, vdim=16, rank=16, ff=None, scale=1.0)], width=24, vocab=12, mult=1.0)
    w = oracle.weights(cfg, seed=5)
    w["l0.mix.q"] = w["l0.mix.q"] * 3.0
    first = {}
    for token in range(12):
        seq = [token] + [5] * 120
        first[token] = oracle.forward(cfg, w, seq)
    moved = max(first, key=lambda t: np.abs(first[t][-1] - first[5][-1]).max())  # the most visible far key
    assert np.abs(first[moved][-1] - first[5][-1]).max() > 0.5
    for token in (5, moved):
        seq = [token] + [5] * 120
        model = _build(cfg, w)
        _assert_logits(model(torch.tensor([seq]))[0], first[token])
        dec = BatchDecoder(model, CPU, torch.float32, 130)
        dec.begin([seq[:100]])
        h = [dec.advance([t])[0] for t in seq[100:]]
        _assert_logits(dec.logits(torch.cat(h)), first[token][100:])


def test_shared_latents_come_from_the_named_layer():
    cfg, w, model = _model("shared")
    s = _seq(cfg, 10)
    w2 = dict(w)
    w2["l2.mix.dkv"] = w["l2.mix.dkv"][:, ::-1].copy()  # layers 2 and 3 read it, 0, 1 and 4 do not
    model.load_state_dict(_to_torch(w2))
    _assert_logits(model(torch.tensor([s]))[0], oracle.forward(cfg, w2, s))
    assert np.abs(oracle.forward(cfg, w2, s) - oracle.forward(cfg, w, s)).max() > 0.1


# ------------------------------------------------------------------------------------------ masks and caches
def test_masks_that_say_the_same_agree():
    cfg, w, model = _model("plain")
    s = torch.tensor([_seq(cfg, 12)])
    want = model(s)
    dense = torch.tril(torch.ones(12, 12, dtype=torch.bool))[None]
    assert torch.allclose(model(s, mask=dense), want) and torch.allclose(model(s, mask=AttentionMask(causal=True)), want)
    assert torch.allclose(model(s, mask=AttentionMask(causal=True, key_start=torch.tensor([0], dtype=torch.int32))), want)
    # packed documents: each its own causal sequence
    docs = torch.tensor([[0] * 5 + [1] * 7])
    pos = torch.tensor([[0, 1, 2, 3, 4, 0, 1, 2, 3, 4, 5, 6]])
    packed = model(s, mask=AttentionMask(causal=True, doc_ids=docs), input_pos=pos)
    _assert_logits(packed[0, 5:], oracle.forward(cfg, w, s[0, 5:].tolist()))


def test_key_start_mask_for_other_attention():
    """The same description works for ordinary attention."""
    q, k, v = torch.randn(2, 2, 4, 8), torch.randn(2, 7, 2, 8), torch.randn(2, 7, 2, 8)
    start = torch.tensor([0, 3], dtype=torch.int32)
    got = ops.attention(q, k, v, AttentionMask(causal=True, key_start=start, query_start=4))
    j, own = torch.arange(7), 4 + torch.arange(2)
    dense = (j[None, None] <= own[None, :, None]) & (j[None, None] >= start[:, None, None])
    assert torch.allclose(got, ops.attention(q, k, v, AttentionMask(causal=False, bool_mask=dense)))


def test_row_layout():
    real = torch.tensor([[0, 0, 1, 1, 1], [1, 1, 1, 1, 1], [0, 1, 1, 1, 1]], dtype=torch.bool)
    lay = RowLayout(real)
    assert lay.start.tolist() == [2, 0, 1]
    assert lay.positions(0, 5).tolist() == [[0, 0, 0, 1, 2], [0, 1, 2, 3, 4], [0, 0, 1, 2, 3]]
    assert lay.positions(6, 1).tolist() == [[4], [6], [5]]
    m = lay.mask(5, 2)
    assert m.dense(3, 2, 8, CPU)[0].int().tolist() == [[0, 0, 1, 1, 1, 1, 0, 0], [0, 0, 1, 1, 1, 1, 1, 0]]
    lay.keep([1, 2])
    assert lay.start.tolist() == [0, 1] and lay.batch == 2
    inside = RowLayout(torch.tensor([[0, 1, 0, 1]], dtype=torch.bool))  # the pad id occurs as a token
    assert inside.start.tolist() == [1]


def test_cache_rows_and_limits():
    c = LatentCache(3, 4, 2, torch.float32)
    c.latent.copy_(torch.arange(24.0).view(3, 4, 2))
    c.advance(2)
    before = c.latent.clone()
    c.keep_rows([1, 2])
    assert torch.equal(c.latent[0, :2], before[1, :2]) and torch.equal(c.latent[1, :2], before[2, :2])
    assert c.reserve(3, 2) == 2
    with pytest.raises(AssertionError):
        c.reserve(1, 3)
    with pytest.raises(ValueError):
        c.reserve(4, 1)
    c.reset()
    assert c.size == 0


def test_cache_utilities():
    cfg, w, model = _model("shared")
    s = torch.tensor([_seq(cfg, 6)])
    want = model(s)
    with local_kv_cache(model, batch_size=1, device=CPU, dtype=torch.float32, decoder_max_seq_len=8):
        assert model.caches_are_enabled() and model.layers[1].attn.kv_cache is None
        with disable_kv_cache(model):
            assert torch.allclose(model(s), want, atol=1e-5)
        assert torch.allclose(model(s, mask=AttentionMask(causal=True), input_pos=torch.arange(6)[None]), want, atol=1e-5)
        assert model.layers[0].attn.kv_cache.size == 6
    assert not model.caches_are_setup()
    model.setup_caches(1, torch.float32, decoder_max_seq_len=8)
    # joined projection weights stay the model's parameters
    model.load_state_dict(model.state_dict())
    assert torch.allclose(model(s, mask=AttentionMask(causal=True), input_pos=torch.arange(6)[None]), want, atol=1e-5)
    delete_kv_caches(model)


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("cached", [True, False])
def test_greedy_generation(cached):
    cfg, w, model = _model("shared")
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
    cfg = oracle.config([oracle.layer(), oracle.layer(kv_from=0)], vocab=200)
    folder = oracle.save(tmp_path / "ckpt", cfg, oracle.weights(cfg))
    (tmp_path / "tok").mkdir()
    sp = write_sentencepiece_model(tmp_path / "tok", vocab_size=200)
    run_tune(tune_path, f"run generate --config begapel/generation checkpoint_dir={folder} output_dir={tmp_path / 'out'} device=cpu dtype=fp32 "
                        f"tokenizer.path={sp} max_new_tokens=6 prompt.user=hello top_k=1", monkeypatch)
    assert "tokens/sec" in caplog.text


# ------------------------------------------------------------------------------------------ configuration and weights
def test_checkpoint_round_trip(tmp_path):
    from torchtune_b200 import training

    cfg = CONFIGS["shared"]
    w = oracle.weights(cfg, seed=9)
    folder = oracle.save(tmp_path / "a", cfg, w)
    ck = training.FullModelHFCheckpointer(str(folder), ["model.safetensors"], "BEGAPEL", output_dir=str(tmp_path / "out"))
    sd = ck.load_checkpoint()["model"]
    back = begapel_tune_to_hf(sd)
    assert set(back) == set(w) and all(np.array_equal(back[k].double().numpy(), w[k]) for k in w)
    model = load_pretrained(folder, dtype=torch.float32, device=CPU, max_seq_len=64)
    assert not model.training and type(model.layers[0]) is ResidualStreamLayer and set(model.state_dict()) == set(sd)
    s = _seq(cfg, 8)
    _assert_logits(model(torch.tensor([s]))[0], oracle.forward(cfg, w, s))
    ck.save_checkpoint({"model": model.state_dict()}, epoch=0)
    again = load_pretrained(tmp_path / "out" / "epoch_0", dtype=torch.float32, device=CPU)
    assert torch.equal(again(torch.tensor([s])), model(torch.tensor([s])))
    with pytest.raises(ValueError, match="unexpected tensor"):
        begapel_hf_to_tune({"l0.mix.z": torch.zeros(1)})


def test_configuration_is_checked(tmp_path):
    good = CONFIGS["shared"]
    path = tmp_path / "config.json"
    path.write_text(json.dumps(good))
    with torch.device("meta"):
        assert len(begapel(config=str(path)).layers) == 5 and len(begapel(config=str(tmp_path)).layers) == 5

    def bad(change, match):
        cfg = copy.deepcopy(good)
        change(cfg)
        with pytest.raises(ValueError, match=match), torch.device("meta"):
            begapel(config=cfg)

    bad(lambda c: c["layers"][0].update(type="conv"), "mixer type")
    bad(lambda c: c["layers"][1].update(mlp={"kind": "experts", "ff": 8}), "feed-forward kind")
    bad(lambda c: c["layers"][1]["mixer"].update(kv_from=3), "does not come before")
    bad(lambda c: c["layers"][4]["mixer"].update(kv_from=1), "none of its own")
    bad(lambda c: c["layers"][1]["mixer"].update(kv_rank=7), "differ in kv_rank")
    bad(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "rotated dimensions")
    with pytest.raises(ValueError, match="architecture"):
        architecture_of({"architecture": "Other"})


def test_adapters_and_gradients():
    """Adapters attach to the named projections and train; the adapted model decodes like its full forward."""
    cfg = CONFIGS["shared"]
    model = lora_begapel(["q_proj", "kv_down", "k_up", "v_up"], True, config=cfg, max_seq_len=64, lora_rank=4, lora_alpha=8)
    for p in model.parameters():
        p.data = torch.randn_like(p) * 0.1
    names = [n for n, _ in model.named_parameters() if "lora_a" in n]
    assert any("layers.0.attn.kv_down" in n for n in names) and not any("layers.1.attn.kv_down" in n for n in names) and any("layers.1.mlp.w1" in n for n in names)
    s = torch.tensor([_seq(cfg, 7)])
    full = model(s)
    full.sum().backward()
    assert model.layers[0].attn.kv_down.lora_a.weight.grad.abs().sum() > 0
    with torch.no_grad():
        model.setup_caches(1, torch.float32, decoder_max_seq_len=7)
        parts = [model(s[:, i : i + 1], mask=AttentionMask(causal=True), input_pos=torch.tensor([[i]])) for i in range(7)]
    assert torch.allclose(torch.cat(parts, 1), full, atol=1e-4)
    with pytest.raises(ValueError, match="unknown attention modules"):
        lora_begapel(["v_proj"], config=cfg, lora_rank=4, lora_alpha=8)


def test_trace_runner_arguments():
    from torchtune_b200.generation import trace

    with pytest.raises(SystemExit):
        trace.main(["--model", "x", "--dtype", "float16", "--out", "y", "--max-tokens", "1"])


def test_trace_replay_bookkeeping(tmp_path):
    """Names, wanted places and ended requests, on CPU."""
    from torchtune_b200.generation.trace import TraceReplay

    cfg, w, model = _model("plain")
    seqs = {"p": _seq(cfg, 9), "q": _seq(cfg, 5, seed=1)}
    want = {k: oracle.forward(cfg, w, v) for k, v in seqs.items()}
    replay = TraceReplay(BatchDecoder(model, CPU, torch.float32, 30), tmp_path)
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])  # noqa: E731
    with torch.inference_mode():
        replay.run({"step": 0, "entries": [{"id": "q", "tokens": seqs["q"][:4], "want": [3, 0]}, {"id": "p", "tokens": seqs["p"][:7], "want": [2]}], "end": []})
        _assert_logits(torch.tensor(read(0)), np.stack([want["q"][3], want["q"][0], want["p"][2]]))
        replay.run({"step": 1, "entries": [{"id": "p", "tokens": seqs["p"][7:8], "want": []}, {"id": "q", "tokens": seqs["q"][4:], "want": [0]}], "end": ["q"]})
        _assert_logits(torch.tensor(read(1)), want["q"][4:])
        with pytest.raises(ValueError):
            replay.run({"step": 2, "entries": [{"id": "q", "tokens": [1], "want": []}], "end": []})
        replay.run({"step": 2, "entries": [{"id": "p", "tokens": seqs["p"][8:], "want": []}], "end": ["p"]})
        assert not (tmp_path / "2.f32").exists() and replay.live == []
        replay.run({"step": 3, "entries": [{"id": "q", "tokens": seqs["q"], "want": [4]}], "end": ["q"]})
        _assert_logits(torch.tensor(read(3)), want["q"][4:])
