"""CUDA kernels of latent attention and of the 32-bit residual stream against float64 statements."""
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest
import torch

import begapel_oracle as oracle

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda"
BF16, F32 = torch.bfloat16, torch.float32


def _rand(*shape, dtype=BF16, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dtype).to(DEV)


def _np(t):
    return t.detach().double().cpu().numpy()


def _close(got, want, dtype, tol16=2e-2, tol32=2e-5):
    want = torch.as_tensor(want)
    err = (got.detach().double().cpu() - want).abs().max().item()
    scale = max(want.abs().max().item(), 1e-3)
    assert err <= (tol32 if dtype == F32 else tol16) * scale, (err, scale)


def _errors():
    from torchtune_b200.ops._lib import check_device_errors

    torch.cuda.synchronize()
    check_device_errors()


# ------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [64, 200, 513, 2048, 5120])
@pytest.mark.parametrize("offset", [0.0, 1.0])
def test_residual_norm(dtype, width, offset):
    from torchtune_b200 import ops

    rows, eps, mult = 37, 1e-3, 0.37
    x, y = _rand(rows, width, dtype=F32), _rand(rows, width, dtype=dtype, scale=0.02, seed=1)
    wp, wn = _rand(width, dtype=dtype, seed=2), _rand(width, dtype=dtype, seed=3)
    with torch.no_grad():
        x1, h = ops.residual_norm(x, y, wp, wn, eps=eps, mult=mult, offset=offset)
        x2, none = ops.residual_norm(x, y, wp, None, eps=eps, mult=mult, offset=offset)
        same, h0 = ops.residual_norm(x, None, None, wn, eps=eps, mult=mult, offset=offset)
    want = _np(x) + mult * oracle.rms_norm(_np(y), _np(wp), eps, offset)
    assert x1.dtype == F32 and h.dtype == dtype and none is None
    _close(x1, want, F32)
    assert torch.equal(x1, x2)
    _close(h, oracle.rms_norm(want, _np(wn), eps, offset), dtype, tol16=5e-3)
    _close(h0, oracle.rms_norm(_np(x), _np(wn), eps, offset), dtype, tol16=5e-3)


def test_softcap_and_wide_logits():
    from torchtune_b200 import ops

    for v, k in ((96, 64), (501, 100)):
        x, w = _rand(5, k), _rand(v, k, seed=1)
        with torch.no_grad():
            z = ops.linear_wide(x, w)
            assert z.dtype == F32 and z.shape == (5, v)
            _close(z, _np(x) @ _np(w).T, F32)
            _close(ops.softcap(z.clone(), 7.0), oracle.soft_cap(_np(z), 7.0), F32)


# ------------------------------------------------------------------------------------------ prepare
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("heads,dim,rot,dims,rank", [(3, 24, 8, 8, 48), (5, 12, 6, 4, 10), (16, 128, 64, 64, 512)])
def test_prepare(dtype, heads, dim, rot, dims, rank):
    from torchtune_b200.modules.latent_attention import PreciseRotaryPositionalEmbeddings
    from torchtune_b200.ops import latent

    b, s, slots, base, eps, first = 2, 3, 9, 300.0, 1e-4, 4
    table = PreciseRotaryPositionalEmbeddings(dims, 64, base).cache.to(DEV)
    width = heads * (dim + rot)
    packed = _rand(b * s, width + rank + rot, dtype=dtype, seed=3)
    q, kv = packed.split([width, rank + rot], dim=1)
    q_in, kv_in = _np(q), _np(kv)
    gain = _rand(rank, dtype=dtype, seed=4)
    pos = torch.tensor([7, 0, 31, 5, 6, 60], dtype=torch.int32, device=DEV)
    want_q = q_in.reshape(b * s, heads, dim + rot).copy()
    want_q[..., dim:] = oracle.rotate_pairs(want_q[..., dim:], pos.tolist(), dims, base)
    want_c = oracle.rms_norm(kv_in[:, :rank], _np(gain), eps, 0.0)
    want_r = oracle.rotate_pairs(kv_in[:, rank:], pos.tolist(), dims, base)
    slot = torch.tensor([first], dtype=torch.int32, device=DEV)
    for device_slot in (None, slot):
        for to_lat in (False, True):
            p2 = packed.clone()
            q2, kv2 = p2.split([width, rank + rot], dim=1)
            buf = torch.full((b, slots, rank + rot), 9.0, dtype=dtype, device=DEV)
            q_out = torch.zeros(b * s, heads, rank + rot, dtype=dtype, device=DEV) if to_lat else None
            latent.prepare(q2, kv2, gain, buf, table, pos, s=s, slot=device_slot, slot_host=first if device_slot is None else 0, heads=heads, dim=dim, rot=rot, rot_dims=dims, rank=rank,
                           eps=eps, q_out=q_out)
            got = q_out[:, :, rank:] if to_lat else q2.reshape(b * s, heads, dim + rot)[..., dim:]
            _close(got, want_q[..., dim:], dtype, tol16=5e-3, tol32=1e-6)
            if to_lat:
                assert torch.equal(q2, q)
            else:
                assert torch.equal(q2.reshape(b * s, heads, dim + rot)[..., :dim], q.reshape(b * s, heads, dim + rot)[..., :dim])
            rows = buf[:, first : first + s].reshape(b * s, -1)
            _close(rows[:, :rank], want_c, dtype, tol16=5e-3, tol32=1e-6)
            _close(rows[:, rank:], want_r, dtype, tol16=5e-3, tol32=1e-6)
            assert bool((buf[:, :first] == 9).all()) and bool((buf[:, first + s :] == 9).all())
    _errors()


# ------------------------------------------------------------------------------------------ attention
def _attend(q, k, kr, v, scale, lo, hi):
    """q [b, s, h, d+r], k [b, sk, h, d], kr [b, sk, r], v [b, sk, h, dv]; key range lo..hi per (b, query)."""
    b, s, h, _ = q.shape
    d = k.shape[-1]
    sc = (torch.einsum("bqhd,bkhd->bhqk", q[..., :d], k) + torch.einsum("bqhr,bkr->bhqk", q[..., d:], kr)) * scale
    j = torch.arange(k.shape[1])
    vis = (j >= lo[..., None]) & (j <= hi[..., None])
    sc = sc.masked_fill(~vis[:, None], -1e300)
    p = torch.softmax(sc, -1) * vis.any(-1)[:, None, :, None]
    return torch.einsum("bhqk,bkhd->bqhd", p, v)


PREFILL = [
    # b, s, first, heads, dim, rot, vdim, rank
    (1, 1, 0, 2, 56, 32, 72, 88),
    (2, 130, 0, 3, 24, 8, 40, 48),
    (1, 300, 0, 2, 128, 64, 128, 64),
    (2, 257, 0, 1, 64, 64, 128, 64),
    (1, 129, 250, 2, 72, 24, 56, 128),
    (1, 513, 0, 2, 192, 64, 128, 64),
    (3, 5, 126, 2, 40, 8, 16, 16),
]


@pytest.mark.parametrize("shape", PREFILL)
@pytest.mark.parametrize("kind", ["bf16", "any", "fp32"])
@pytest.mark.parametrize("padded", [False, True])
def test_prefill(shape, kind, padded, monkeypatch):
    from torchtune_b200.ops import latent

    b, s, first, H, d, r, dv, rank = shape
    dtype = F32 if kind == "fp32" else BF16
    if kind == "any":
        monkeypatch.setattr(latent, "prefill_supported", lambda *a: False)
    sk, slots = first + s, first + s + 40
    q = _rand(b * s, H * (d + r), dtype=dtype, seed=1)
    kv = _rand(b * sk, H * (d + dv), dtype=dtype, seed=2)
    kn, v = kv.split([H * d, H * dv], dim=1)
    buf = _rand(b, slots, rank + r, dtype=dtype, seed=3)
    g = _rand(b * s, H * dv + 16, dtype=dtype, seed=4)[:, : H * dv]
    # one far key per sequence dominates for the last query
    q.view(b, s, H, d + r)[:, -1] *= 4
    start = torch.tensor([(7 * i + 3) % s if padded else 0 for i in range(b)], dtype=torch.int32)
    lo = start[:, None].expand(b, s)
    hi = (first + torch.arange(s))[None].expand(b, s)
    scale = 0.9 / (d + r) ** 0.5
    bounds = latent.Bounds(lo=start.to(DEV), lo_row=1) if padded else latent.Bounds()
    out = latent.prefill(q, kn, v, buf, g, b=b, s=s, sk=sk, slot0=first, heads=H, dim=d, rot=r, vdim=dv, rank=rank, scale=scale, bounds=bounds)
    want = _attend(q.double().cpu().view(b, s, H, d + r), kn.double().cpu().reshape(b, sk, H, d), buf[:, :sk, rank:].double().cpu(), v.double().cpu().reshape(b, sk, H, dv), scale, lo, hi)
    want = want.reshape(b * s, H * dv) * torch.sigmoid(g.double().cpu())
    _errors()
    _close(out, want, dtype)
    # explicit bounds say the same
    wide = latent.Bounds(lo=lo.contiguous().to(DEV), lo_row=s, lo_query=1, hi=hi.to(torch.int32).contiguous().to(DEV), hi_row=s, hi_query=1)
    again = latent.prefill(q, kn, v, buf, g, b=b, s=s, sk=sk, slot0=first, heads=H, dim=d, rot=r, vdim=dv, rank=rank, scale=scale, bounds=wide)
    assert torch.equal(out, again)


DECODE = [
    # b, heads, rank, rot, newest slot, slots
    (1, 6, 104, 24, 0, 64),
    (1, 6, 104, 24, 127, 300),
    (2, 6, 104, 24, 128, 300),
    (3, 20, 48, 8, 259, 300),
    (1, 16, 512, 64, 1500, 2048),
    (2, 40, 512, 64, 700, 701),
    (5, 16, 256, 128, 383, 384),
    (1, 3, 16, 24, 129, 130),
]


@pytest.mark.parametrize("shape", DECODE)
@pytest.mark.parametrize("kind", ["bf16", "any", "fp32"])
@pytest.mark.parametrize("vdim", [40, 128])
def test_decode_and_value(shape, kind, vdim, monkeypatch):
    from torchtune_b200.ops import latent

    b, H, rank, r, newest, slots = shape
    dtype = F32 if kind == "fp32" else BF16
    if kind == "any":
        monkeypatch.setattr(latent, "decode_supported", lambda *a: False)
    q = _rand(b, H, rank + r, dtype=dtype, seed=1)
    buf = _rand(b, slots, rank + r, dtype=dtype, seed=2)
    w = _rand(H * vdim, rank, dtype=dtype, seed=3, scale=rank**-0.5)
    g = _rand(b, H * vdim + 8, dtype=dtype, seed=4)[:, : H * vdim]
    scale = 1.5 / (rank + r) ** 0.5
    slot = torch.tensor([newest], dtype=torch.int32, device=DEV)
    for start in ([0] * b, [min(newest, 130 * i + 1) for i in range(b)]):
        lo = torch.tensor(start, dtype=torch.int32)
        bounds = latent.Bounds(lo=lo.to(DEV), lo_row=1)
        kr, c = buf[..., rank:].double().cpu(), buf[..., :rank].double().cpu()
        lat = _attend(q.double().cpu()[:, None], c[:, :, None].expand(b, slots, H, rank), kr, c[:, :, None].expand(b, slots, H, rank), scale, lo[:, None], torch.full((b, 1), newest))[:, 0]
        want = torch.einsum("bhk,hnk->bhn", lat, w.double().cpu().view(H, vdim, rank)).reshape(b, H * vdim) * torch.sigmoid(g.double().cpu())
        for device_slot, keys in ((None, newest + 1), (slot, slots)):
            o, ml = latent.decode(q, buf, rank=rank, rot=r, scale=scale, slot=device_slot, slot_host=newest, bounds=bounds, keys=keys)
            out = latent.value(o, ml, w, g, vdim=vdim)
            _errors()
            _close(out, want, dtype)
        monkeypatch.setattr(latent, "VALUE_GROUPED_ROWS", 1)
        if dtype == BF16:
            _close(latent.value(o, ml, w, g, vdim=vdim), want, dtype)
        monkeypatch.setattr(latent, "VALUE_GROUPED_ROWS", 32)


def test_decode_single_key_stands_out():
    """One cached row scores far above all others, at the first, last and tile-border slots: its value comes back alone."""
    from torchtune_b200.ops import latent

    H, rank, r, slots = 4, 64, 8, 400
    for at in (0, 127, 128, 255, 256, 399):
        buf = _rand(1, slots, rank + r, seed=at) * 0.1
        q = torch.zeros(1, H, rank + r, dtype=BF16, device=DEV)
        q[..., rank] = 30.0
        buf[0, :, rank] = 0.0
        buf[0, at, rank] = 30.0
        for newest in sorted({at, slots - 1}):
            o, ml = latent.decode(q, buf, rank=rank, rot=r, scale=1.0, slot=None, slot_host=newest, bounds=latent.Bounds(), keys=newest + 1)
            eye = torch.eye(rank, dtype=BF16, device=DEV).repeat(H, 1)
            out = latent.value(o, ml, eye, None, vdim=rank).view(H, rank)
            _close(out, _np(buf[0, at, :rank])[None].repeat(H, 0), BF16, tol16=5e-3)
        if at > 0:  # the same key just outside the range
            o, ml = latent.decode(q, buf, rank=rank, rot=r, scale=1.0, slot=None, slot_host=at - 1, bounds=latent.Bounds(), keys=at)
            out = latent.value(o, ml, eye, None, vdim=rank).view(H, rank)
            _close(out, _np(buf[0, :at, :rank]).mean(0)[None].repeat(H, 0), BF16, tol16=2e-2)
    _errors()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("rows", [1, 3, 9, 130])
@pytest.mark.parametrize("heads,dim,rot,rank", [(3, 24, 8, 48), (16, 128, 64, 512), (5, 12, 6, 10)])
def test_absorb(dtype, rows, heads, dim, rot, rank):
    from torchtune_b200.ops import latent

    q = _rand(rows, heads * (dim + rot) + 8, dtype=dtype, seed=1)[:, : heads * (dim + rot)]
    w = _rand(heads * dim, rank, dtype=dtype, seed=2, scale=dim**-0.5)
    out = torch.zeros(rows, heads, rank + rot, dtype=dtype, device=DEV)
    latent.absorb(q.contiguous() if rows == 130 else q, w, out, heads=heads, dim=dim, rot=rot, rank=rank)
    want = np.einsum("rhd,hdn->rhn", _np(q).reshape(rows, heads, dim + rot)[..., :dim], _np(w).reshape(heads, dim, rank))
    _errors()
    _close(out[..., :rank], want, dtype, tol16=1e-2)
    assert not out[..., rank:].any()


# ------------------------------------------------------------------------------------------ whole model
MODELS = {
    "plain": lambda: oracle.config([oracle.layer(), oracle.layer(heads=2, dim=40, rot=16, vdim=24, rank=64, ff=None)]),
    "shared": lambda: oracle.config([oracle.layer(ff=None), oracle.layer(kv_from=0, heads=5, dim=16, vdim=32), oracle.layer(rank=80), oracle.layer(kv_from=2, rank=80), oracle.layer(kv_from=0)],
                                    width=104, mult=1.0),
    "odd": lambda: oracle.config([oracle.layer(heads=3, dim=10, rot=6, vdim=7, rank=21, ff=35), oracle.layer(kv_from=0, heads=1, dim=5, rot=6, vdim=9, rank=21, ff=22)], width=51, vocab=67),
    "large_heads": lambda: oracle.config([oracle.layer(heads=18, dim=128, rot=64, vdim=128, rank=512, ff=64)], width=64),
}


def _load(tmp_path, name, dtype, sharp=2.0):
    from torchtune_b200.models._registry import load_pretrained

    cfg = MODELS[name]()
    w = oracle.weights(cfg, seed=len(name), sharp=sharp)
    return cfg, w, load_pretrained(oracle.save(tmp_path / name, cfg, w), dtype=dtype, device=torch.device(DEV), max_seq_len=512)


def _rms_error(got, want):
    d = got.detach().double().cpu().numpy() - want
    d -= d.mean(-1, keepdims=True)
    return (np.sqrt((d * d).mean(-1)) / want.std()).max()


@pytest.mark.parametrize("name", list(MODELS))
@pytest.mark.parametrize("dtype,tol", [(F32, 3e-5), (BF16, 6e-2)])
def test_model(tmp_path, name, dtype, tol):
    from torchtune_b200.generation import BatchDecoder

    cfg, w, model = _load(tmp_path, name, dtype)
    rng = np.random.default_rng(1)
    seqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in (140, 9, 1, 133)]
    want = [oracle.forward(cfg, w, s) for s in seqs]
    with torch.inference_mode():
        for s, e in zip(seqs, want):  # no cache
            assert _rms_error(model(torch.tensor([s], device=DEV))[0], e) < tol
        dec = BatchDecoder(model, torch.device(DEV), dtype, 400)
        for s, e in zip(seqs, want):  # prompt, then one by one; caches reused from request to request
            n = max(1, len(s) - 6)
            h = [dec.begin([s[:n]])[0]] + [dec.advance([t])[0] for t in s[n:]]
            assert _rms_error(dec.logits(torch.cat(h)), e) < tol
            dec.end([0])
        # unequal rows together; the shorter ones end earlier
        cut = [len(s) - k for s, k in zip(seqs, (20, 4, 0, 9))]
        h = dec.begin([s[:n] for s, n in zip(seqs, cut)])
        live, at, L = [0, 1, 2, 3], list(cut), h.shape[1]
        for k in range(4):
            assert _rms_error(dec.logits(h[k, L - cut[k] :]), want[k][: cut[k]]) < tol
        while live:
            gone = [i for i, k in enumerate(live) if at[k] == len(seqs[k])]
            dec.end(gone)
            live = [k for i, k in enumerate(live) if i not in gone]
            if not live:
                break
            h = dec.advance([seqs[k][at[k]] for k in live])
            for i, k in enumerate(live):
                assert _rms_error(dec.logits(h[i]), want[k][at[k] : at[k] + 1]) < tol
                at[k] += 1
        # several tokens at a time behind a prompt
        s, e = seqs[0], want[0]
        with torch.device(DEV):
            from torchtune_b200.modules import delete_kv_caches

            delete_kv_caches(model)
            model.setup_caches(1, dtype, decoder_max_seq_len=len(s))
        done = 0
        for n in (2, 63, 2, 64, 9):
            x = torch.tensor([s[done : done + n]], device=DEV)
            from torchtune_b200.ops.mask import AttentionMask

            got = model(x, mask=AttentionMask(causal=True), input_pos=torch.arange(done, done + n, device=DEV)[None])
            assert _rms_error(got[0], e[done : done + n]) < tol
            done += n
    _errors()


def test_greedy_generation_matches(tmp_path):
    """fp32 generation through ``generate`` picks the oracle's tokens, alone and in a padded batch."""
    from torchtune_b200.generation import generate
    from torchtune_b200.modules import local_kv_cache

    cfg, w, model = _load(tmp_path, "shared", F32)
    prompts = [[5, 9, 2, 33, 8], [7, 1]]
    want = [oracle.greedy(cfg, w, p, 6) for p in prompts]
    pad = cfg["vocab"] + 1
    batch = torch.tensor([prompts[0], [pad] * 3 + prompts[1]], device=DEV)
    with local_kv_cache(model, batch_size=2, device=torch.device(DEV), dtype=F32, decoder_max_seq_len=16):
        safe = batch.masked_fill(batch == pad, 0)
        assert not (safe[:, 0] == 0).all()
        out, _ = generate(model, safe, max_generated_tokens=6, pad_id=0, top_k=1)
        model.reset_caches()
        alone, _ = generate(model, torch.tensor(prompts[0], device=DEV), max_generated_tokens=6, pad_id=0, top_k=1)
    assert out[0].tolist() == want[0] and out[1, 3:].tolist() == want[1] and alone[0].tolist() == want[0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    cfg = MODELS["shared"]()
    w = oracle.weights(cfg, seed=6)
    folder = oracle.save(tmp_path / "m", cfg, w)
    rng = np.random.default_rng(2)
    seqs = {k: rng.integers(0, cfg["vocab"], n).tolist() for k, n in (("x", 11), ("y", 4), ("z", 7))}
    want = {k: oracle.forward(cfg, w, s) for k, s in seqs.items()}
    steps = [
        {"step": 0, "entries": [{"id": "x", "tokens": seqs["x"][:8], "want": [7, 0]}, {"id": "y", "tokens": seqs["y"][:3], "want": [1]}], "end": []},
        {"step": 1, "entries": [{"id": "y", "tokens": seqs["y"][3:], "want": [0]}, {"id": "x", "tokens": seqs["x"][8:9], "want": []}], "end": ["y"]},
        {"step": 2, "entries": [{"id": "x", "tokens": seqs["x"][9:10], "want": []}], "end": []},
        {"step": 3, "entries": [{"id": "x", "tokens": seqs["x"][10:], "want": [0]}], "end": ["x"]},
        {"step": 4, "entries": [{"id": "z", "tokens": seqs["z"], "want": [6, 2]}], "end": ["z"]},
    ]
    out = tmp_path / "out"
    out.mkdir()
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "20"], input="\n".join(map(json.dumps, steps)),
                         capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    expect = {0: [want["x"][7], want["x"][0], want["y"][1]], 1: [want["y"][3]], 3: [want["x"][10]], 4: [want["z"][6], want["z"][2]]}
    assert sorted(p.name for p in out.iterdir()) == sorted(f"{i}.f32" for i in expect)
    for i, rows in expect.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(len(rows), -1))
        assert _rms_error(got, np.stack(rows)) < (3e-5 if dtype == "float32" else 6e-2)
