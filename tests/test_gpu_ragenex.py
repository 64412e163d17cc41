"""CUDA kernels of span attention, lightning attention and hyper-connected streams against float64 statements, and the Ragenex decoder built
from them."""
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest
import torch

import ragenex_oracle as oracle

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


# ------------------------------------------------------------------------------------------ streams
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [64, 203, 1028, 2048, 4096, 8200])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 7])
def test_stream_step(dtype, width, S):
    from torchtune_b200 import ops

    rows, eps = 19, 1e-3
    x, y = _rand(rows, S, width, dtype=F32), _rand(rows, width, dtype=dtype, seed=1)
    gain, wn = _rand(width, dtype=dtype, seed=2), _rand(width, dtype=dtype, seed=3)
    mix, out, read = _rand(S, S, dtype=dtype, seed=4), _rand(S, dtype=dtype, seed=5), _rand(S, dtype=dtype, seed=6)
    for one in (False, True):  # one stream stands for S equal ones
        xi = x[:, :1].contiguous() if one else x
        streams = np.repeat(_np(xi), S, 1) if one else _np(xi)
        want = oracle.write_streams(streams, _np(mix), _np(out), _np(gain) * _np(y))
        with torch.no_grad():
            x1, h = ops.stream_step(xi, y, gain, mix, out, read, wn, eps=eps, centered=True)
            x2, none = ops.stream_step(xi, y, gain, mix, out, None, None, eps=eps, centered=True)
            gone, total = ops.stream_step(xi, y, gain, mix, out, None, wn, eps=eps, centered=True, keep=False)
            same, h0 = ops.stream_step(xi, None, None, None, None, read, wn, eps=eps, centered=True)
            _, rms = ops.stream_step(xi, y, gain, mix, out, read, wn, eps=eps, centered=False, offset=1.0)
        assert x1.dtype == F32 and x1.shape == (rows, S, width) and h.dtype == dtype and none is None and gone is None and same.shape == xi.shape
        _close(x1, want, F32)
        assert torch.equal(x1, x2)
        _close(h, oracle.layer_norm(oracle.read_streams(want, _np(read)), _np(wn), eps), dtype, tol16=6e-3)
        _close(total, oracle.layer_norm(want.sum(1), _np(wn), eps), dtype, tol16=6e-3)
        _close(h0, oracle.layer_norm(oracle.read_streams(streams, _np(read)), _np(wn), eps), dtype, tol16=6e-3)
        _close(rms, oracle.rms_norm(oracle.read_streams(want, _np(read)), 1.0 + _np(wn), eps), dtype, tol16=6e-3)


def test_layer_norm_of_a_shifted_row():
    """A mean far above the spread: the deviations are squared, not the values."""
    from torchtune_b200 import ops

    x = _rand(3, 1, 2048, dtype=F32, scale=0.01) + 30.0
    w = torch.ones(2048, device=DEV)
    with torch.no_grad():
        h = ops.stream_step(x, None, None, None, None, None, w, eps=1e-8, centered=True)[1]
    _close(h, oracle.layer_norm(_np(x)[:, 0], 1.0, 1e-8), F32, tol32=3e-4)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [40, 51, 1536])
def test_embed_positions(dtype, width):
    from torchtune_b200 import ops

    table, pos_table = _rand(33, width, dtype=dtype), _rand(17, width, dtype=dtype, seed=1)
    ids, pos = torch.tensor([[0, 32, 5], [7, 7, 1]], device=DEV), torch.tensor([[0, 16, 3], [2, 9, 9]], dtype=torch.int32, device=DEV)
    with torch.no_grad():
        x = ops.embed_positions(ids, pos, table, pos_table)
    assert x.dtype == F32 and torch.equal(x, table.float()[ids] + pos_table.float()[pos.long()])


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_clamped_glu(dtype):
    from torchtune_b200 import ops

    for width in (96, 35):
        both = _rand(21, 2 * width + 8, dtype=dtype, scale=2.0)
        g, u = both[:, :width], both[:, width : 2 * width]
        for limit in (0.7, 3.0):
            with torch.no_grad():
                _close(ops.clamped_glu(g, u, limit, 1.702), oracle.clamped_glu(_np(g), _np(u), limit), dtype, tol16=6e-3)


def test_feed_forward_with_the_gate_in_the_gemm():
    """Enough rows for the CTA-pair GEMM: same result as the separate steps."""
    from torchtune_b200.modules import ClampedGLU, FeedForward, Linear
    from torchtune_b200.ops import _cuda

    torch.manual_seed(0)
    dim, ff = 512, 1024
    mlp = FeedForward(gate_proj=Linear(dim, ff, bias=False), down_proj=Linear(ff, dim, bias=False), up_proj=Linear(dim, ff, bias=False), activation=ClampedGLU(0.9)).to(DEV, BF16)
    x = _rand(4096, dim)
    with torch.no_grad():
        fused = _cuda.gate_up_swiglu(x, mlp.w1.weight, mlp.w3.weight, (0.9, 1.702))
        assert fused is not None
        want = oracle.clamped_glu(_np(x) @ _np(mlp.w1.weight).T, _np(x) @ _np(mlp.w3.weight).T, 0.9)
        _close(fused, want, BF16)
        _close(mlp(x), want @ _np(mlp.w2.weight).T, BF16)
        _close(mlp(x[:5]), (want @ _np(mlp.w2.weight).T)[:5], BF16)
    _errors()


# ------------------------------------------------------------------------------------------ span attention
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("heads,groups,dim,vdim", [(6, 2, 24, 40), (5, 1, 7, 9), (16, 4, 128, 128), (4, 4, 40, 16)])
def test_span_prepare(dtype, heads, groups, dim, vdim):
    from torchtune_b200.ops import span

    b, s, slots, first, eps, coef, every = 2, 3, 9, 4, 1e-2, 0.6, 5
    widths = [heads * dim, groups * dim, groups * vdim]
    packed = _rand(b * s, sum(widths), dtype=dtype, seed=3)
    gq, gk = _rand(widths[0], dtype=dtype, seed=4), _rand(widths[1], dtype=dtype, seed=5)
    pos = torch.tensor([3, 4, 5, 98, 99, 100], dtype=torch.int32, device=DEV)
    slot = torch.tensor([first], dtype=torch.int32, device=DEV)
    for gains, c in (((gq, gk), coef), ((None, None), 0.0), ((gq, gk), 0.0), ((None, None), coef)):
        for device_slot in (None, slot):
            q, k, v = packed.clone().split(widths, dim=1)
            qn, kn, vn = _np(q), _np(k), _np(v)
            if gains[0] is not None:
                qn, kn = oracle.rms_norm(qn, _np(gq), eps), oracle.rms_norm(kn, _np(gk), eps)
            qn = qn * np.array([oracle.temperature(p, c, every) for p in pos.tolist()])[:, None]
            keys, values = (torch.full((b, slots, groups, d), 9.0, dtype=dtype, device=DEV) for d in (dim, vdim))
            got = span.prepare(q, k, v, *gains, keys, values, pos, s=s, slot=device_slot, slot_host=first if device_slot is None else 0, eps=eps, coef=c, every=every)
            _close(got, qn, dtype, tol16=6e-3, tol32=1e-6)
            _close(keys[:, first : first + s].reshape(b * s, -1), kn, dtype, tol16=6e-3, tol32=1e-6)
            assert torch.equal(values[:, first : first + s].reshape(b * s, -1), v) and np.array_equal(_np(v), vn)
            for t in (keys, values):
                assert bool((t[:, :first] == 9).all()) and bool((t[:, first + s :] == 9).all())
    _errors()


def _attend(q, k, v, scale, lo, hi):
    """q [b, s, h, d], k [b, sk, g, d], v [b, sk, g, dv]; key range lo..hi per (b, query)."""
    n = q.shape[2] // k.shape[2]
    k, v = k.repeat_interleave(n, 2), v.repeat_interleave(n, 2)
    sc = torch.einsum("bqhd,bkhd->bhqk", q, k) * scale
    j = torch.arange(k.shape[1])
    vis = (j >= lo[..., None]) & (j <= hi[..., None])
    p = torch.softmax(sc.masked_fill(~vis[:, None], -1e300), -1) * vis.any(-1)[:, None, :, None]
    return torch.einsum("bhqk,bkhd->bqhd", p, v)


SPAN_PREFILL = [
    # b, s, first, heads, groups, dim, vdim
    (1, 1, 0, 2, 1, 56, 72),
    (2, 130, 0, 6, 2, 24, 40),
    (1, 300, 0, 4, 4, 128, 128),
    (2, 257, 0, 3, 1, 64, 120),
    (1, 129, 250, 4, 2, 72, 56),
    (1, 513, 0, 2, 1, 200, 128),
    (3, 5, 126, 8, 2, 40, 16),
]


@pytest.mark.parametrize("shape", SPAN_PREFILL)
@pytest.mark.parametrize("kind", ["bf16", "any", "fp32"])
@pytest.mark.parametrize("padded", [False, True])
def test_span_prefill(shape, kind, padded, monkeypatch):
    from torchtune_b200.ops import latent, span

    b, s, first, H, G, d, dv = shape
    dtype = F32 if kind == "fp32" else BF16
    if kind == "any":
        monkeypatch.setattr(span, "prefill_supported", lambda *a: False)
    sk, slots = first + s, first + s + 40
    q = _rand(b * s, H * d + 8, dtype=dtype, seed=1)[:, : H * d]
    keys, values = _rand(b, slots, G, d, dtype=dtype, seed=2), _rand(b, slots, G, dv, dtype=dtype, seed=3)
    q[s - 1 :: s] *= 4  # sharp scores for the last queries
    start = torch.tensor([(7 * i + 3) % s if padded else 0 for i in range(b)], dtype=torch.int32)
    lo, hi = start[:, None].expand(b, s), (first + torch.arange(s))[None].expand(b, s)
    scale = 0.9 / d**0.5
    bounds = latent.Bounds(lo=start.to(DEV), lo_row=1) if padded else latent.Bounds()
    args = dict(b=b, s=s, sk=sk, slot0=first, heads=H, scale=scale)
    out = span.prefill(q, keys, values, bounds=bounds, **args)
    want = _attend(q.double().cpu().view(b, s, H, d), keys[:, :sk].double().cpu(), values[:, :sk].double().cpu(), scale, lo, hi).reshape(b * s, H * dv)
    _errors()
    _close(out, want, dtype)
    wide = latent.Bounds(lo=lo.contiguous().to(DEV), lo_row=s, lo_query=1, hi=hi.to(torch.int32).contiguous().to(DEV), hi_row=s, hi_query=1)
    assert torch.equal(out, span.prefill(q, keys, values, bounds=wide, **args))


SPAN_DECODE = [
    # b, heads, groups, dim, vdim, newest slot, slots
    (1, 6, 2, 24, 40, 0, 64),
    (1, 6, 1, 104, 128, 127, 300),
    (2, 8, 4, 64, 72, 128, 300),
    (3, 40, 2, 48, 8, 259, 300),
    (1, 16, 4, 128, 128, 1500, 2048),
    (2, 34, 1, 256, 256, 700, 701),
    (5, 4, 4, 128, 64, 383, 384),
    (1, 20, 1, 16, 392, 129, 130),
]


@pytest.mark.parametrize("shape", SPAN_DECODE)
@pytest.mark.parametrize("kind", ["bf16", "any", "fp32"])
def test_span_decode(shape, kind, monkeypatch):
    from torchtune_b200.ops import latent, span

    b, H, G, d, dv, newest, slots = shape
    dtype = F32 if kind == "fp32" else BF16
    if kind == "any":
        monkeypatch.setattr(span, "decode_supported", lambda *a: False)
    q = _rand(b, H * d + 16, dtype=dtype, seed=1)[:, : H * d].view(b, H, d)
    keys, values = _rand(b, slots, G, d, dtype=dtype, seed=2), _rand(b, slots, G, dv, dtype=dtype, seed=3)
    scale = 1.5 / d**0.5
    slot = torch.tensor([newest], dtype=torch.int32, device=DEV)
    for start in ([0] * b, [min(newest, 130 * i + 1) for i in range(b)]):
        lo = torch.tensor(start, dtype=torch.int32)
        bounds = latent.Bounds(lo=lo.to(DEV), lo_row=1)
        want = _attend(q.double().cpu()[:, None], keys.double().cpu(), values.double().cpu(), scale, lo[:, None], torch.full((b, 1), newest)).reshape(b, H * dv)
        for device_slot, visible in ((None, newest + 1), (slot, slots)):
            out = span.decode(q, keys, values, scale=scale, slot=device_slot, slot_host=newest, bounds=bounds, keys_visible=visible)
            _errors()
            _close(out, want, dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_span_decode_single_key_stands_out(dtype):
    """One cached key scores far above all others, at the first, last and tile-border slots: its value comes back alone; just outside the
    range it has no part."""
    from torchtune_b200.ops import latent, span

    H, G, d, slots = 4, 2, 64, 400
    for at in (0, 127, 128, 255, 256, 399):
        values = _rand(1, slots, G, 72, seed=at, dtype=dtype)
        q, keys = torch.zeros(1, H, d, dtype=dtype, device=DEV), torch.zeros(1, slots, G, d, dtype=dtype, device=DEV)
        q[..., 5] = 30.0
        keys[0, at, :, 5] = 30.0
        run = lambda newest, lo=0: span.decode(q, keys, values, scale=1.0, slot=None, slot_host=newest, bounds=latent.Bounds(lo=torch.tensor([lo], dtype=torch.int32, device=DEV), lo_row=1),  # noqa: E731
                                               keys_visible=newest + 1).view(H, 72)
        per_head = lambda t: _np(t).repeat(2, 0)  # noqa: E731
        for newest in sorted({at, slots - 1}):
            _close(run(newest), per_head(values[0, at]), dtype, tol16=5e-3)
            _close(run(newest, at), per_head(values[0, at]), dtype, tol16=5e-3)
        if at > 0:
            _close(run(at - 1), per_head(values[0, :at].double().mean(0)), dtype)
        if at < slots - 1:
            _close(run(slots - 1, at + 1), per_head(values[0, at + 1 :].double().mean(0)), dtype)
    _errors()


# ------------------------------------------------------------------------------------------ lightning attention
def _recurrence(q, k, v, decay, state, starts, first, H):
    """Per row through the oracle; k of padding is left out."""
    b = state.shape[0]
    s = q.shape[0] // b
    outs, states = [], []
    for i in range(b):
        r = slice(i * s, (i + 1) * s)
        qi, ki, vi = (oracle.silu(_np(t[r])).reshape(s, H, -1) for t in (q, k, v))
        ki = ki * (first + np.arange(s) >= starts[i])[:, None, None]
        o, st = oracle.decayed_recurrence(qi, ki, vi, decay, _np(state[i]))
        outs.append(o.reshape(s, -1)), states.append(st)
    return np.concatenate(outs), np.stack(states)


LIGHTNING = [
    # b, s, decay, dim, vdim
    (1, 1, (0.5, 0.99), 128, 128),
    (3, 1, (0.9,), 7, 9),
    (2, 9, (0.3, 1.0, 0.0), 24, 40),
    (1, 40, (0.999, 0.7), 40, 130),
    (2, 129, (0.999, 0.7), 16, 24),
    (1, 128, (0.0, 1.0, 0.97), 128, 128),
    (2, 300, (0.9, 0.995), 72, 104),
    (1, 700, (0.6, 0.9999), 128, 64),
    (1, 65, (0.98,), 200, 16),
]


@pytest.mark.parametrize("shape", LIGHTNING)
@pytest.mark.parametrize("kind", ["bf16", "runs", "recurrent", "fp32"])
def test_lightning(shape, kind, monkeypatch):
    from torchtune_b200.ops import recurrent

    b, s, decay, d, dv = shape
    H, dtype = len(decay), F32 if kind == "fp32" else BF16
    if kind == "recurrent":
        monkeypatch.setattr(recurrent, "chunks_supported", lambda *a: False)
    if kind == "runs":  # one chunk per run: the states in front of the runs carry everything
        monkeypatch.setattr(recurrent, "run_chunks", lambda *a: 1)
    widths = [H * d, H * d, H * dv]
    packed = _rand(b * s, sum(widths) + 16, dtype=dtype, seed=1)
    before = _rand(b, H, d, dv, dtype=F32, seed=2)
    for fresh, padded in ((True, False), (False, False), (True, True)):
        first = 0 if fresh else 5
        starts = [(37 * i + 11) % s if padded else 0 for i in range(b)]
        state = before.clone()
        q, k, v, _ = packed.clone().split(widths + [16], dim=1)
        want, after = _recurrence(q, k, v, decay, torch.zeros_like(before) if fresh else before, starts, first, H)
        o = recurrent.lightning(q, k, v, decay, state, b=b, s=s, heads=H, dim=d, vdim=dv, fresh=fresh, first=first,
                                starts=torch.tensor(starts, dtype=torch.int32, device=DEV) if padded else None)
        _errors()
        _close(o, want, dtype, tol16=1e-2)
        _close(state, after, dtype, tol16=6e-3)
    free, _ = _recurrence(*packed.split(widths + [16], dim=1)[:3], decay, torch.zeros_like(before), [0] * b, 0, H)
    q, k, v, _ = packed.clone().split(widths + [16], dim=1)
    _close(recurrent.lightning(q, k, v, decay, None, b=b, s=s, heads=H, dim=d, vdim=dv, fresh=True, first=0, starts=None), free, dtype, tol16=1e-2)
    _errors()


def test_lightning_state_keeps_32_bits():
    """Many chunks with almost no decay and a state much larger than what a token adds: the chunked state follows the exact one to far more
    digits than a bf16 operand would leave."""
    from torchtune_b200.ops import recurrent

    b, s, H, d, dv, decay = 1, 1024, 2, 64, 64, (0.99995, 1.0)
    q, k, v = (_rand(b * s, H * n, seed=i) + 1.0 for i, n in enumerate((d, d, dv)))
    state = _rand(b, H, d, dv, dtype=F32, seed=9) * 1e4
    activated = [torch.nn.functional.silu(t.float()).to(BF16) for t in (q, k, v)]  # as the kernels see them
    qi, ki, vi = (_np(t).reshape(s, H, -1) for t in activated)
    o, after = oracle.decayed_recurrence(qi, ki, vi, decay, _np(state[0]))
    got_state = state.clone()
    out = recurrent.lightning(q, k, v, decay, got_state, b=b, s=s, heads=H, dim=d, vdim=dv, fresh=False, first=1, starts=None)
    _errors()
    _close(got_state, after[None], F32, tol32=2e-4)
    _close(out, o.reshape(s, -1), BF16, tol16=5e-3)


def test_lightning_token_that_stands_out():
    """One token writes to the state, a later one reads it: what comes back is its value times the decay of the distance, across chunk and run
    borders."""
    from torchtune_b200.ops import recurrent

    H, d, dv, s = 2, 32, 40, 520
    decay = (0.995, 1.0)
    for at, ask in ((0, 519), (127, 128), (126, 127), (128, 255), (255, 256), (383, 519), (3, 4), (200, 200)):
        q, k, v = (torch.full((s, H * n), -200.0, dtype=BF16, device=DEV) for n in (d, d, dv))  # SiLU of -200 is 0
        v[at] = _rand(H * dv, seed=at).abs() + 1.0
        k[at], q[ask] = 2.0, 3.0
        want = np.zeros((s, H, dv))
        qk = d * oracle.silu(2.0) * oracle.silu(3.0)
        for h in range(H):
            want[ask, h] = qk * decay[h] ** (ask - at) * oracle.silu(_np(v[at])).reshape(H, dv)[h]
        for per in (1, 2, 9):
            recurrent_per = recurrent.run_chunks
            recurrent.run_chunks = lambda *a: per
            try:
                o = recurrent.lightning(q.clone(), k.clone(), v.clone(), decay, None, b=1, s=s, heads=H, dim=d, vdim=dv, fresh=True, first=0, starts=None)
            finally:
                recurrent.run_chunks = recurrent_per
            _close(o, want.reshape(s, -1), BF16, tol16=1e-2)
    _errors()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [96, 51, 2048])
def test_gated_norm(dtype, width):
    from torchtune_b200.ops import recurrent

    rows, eps = 13, 1e-2
    gain, gate = _rand(width, dtype=dtype, seed=1), _rand(rows, width + 8, dtype=dtype, seed=2)[:, :width]
    for o in (_rand(rows, width, dtype=F32, scale=0.1), _rand(rows, width, dtype=dtype)):
        _close(recurrent.gated_norm(o, gain, gate, eps), oracle.gated_norm(_np(o), _np(gain), _np(gate), eps), dtype, tol16=6e-3)


# ------------------------------------------------------------------------------------------ whole model
MODELS = {
    "plain": lambda: oracle.config([oracle.attention_layer(), oracle.lightning_layer(), oracle.attention_layer(heads=4, kv_heads=4, dim=40, vdim=16, ff=None)]),
    "looped": lambda: oracle.config([oracle.lightning_layer(ff=None), oracle.attention_layer(heads=5, kv_heads=1, dim=64, vdim=72, coef=0.3, every=17), oracle.lightning_layer(decay=(0.8, 0.99), dim=40, vdim=16),
                                     oracle.attention_layer()], loop=(0, 3, 2), streams=4, width=136, eps=3e-2),
    "odd": lambda: oracle.config([oracle.lightning_layer(decay=(0.9, 0.98, 0.7), dim=13, vdim=11, ff=35), oracle.attention_layer(heads=3, kv_heads=3, dim=11, vdim=9, every=1, ff=22)], width=51, vocab=67, streams=1,
                                 loop=(1, 2, 2), eps=1e-2),
    "large": lambda: oracle.config([oracle.attention_layer(heads=36, kv_heads=2, dim=128, vdim=128, ff=64), oracle.lightning_layer(decay=(0.97, 0.9999), dim=128, vdim=128, ff=64)], width=72, streams=2),
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
@pytest.mark.parametrize("dtype,tol", [(F32, 5e-5), (BF16, 8e-2)])
def test_model(tmp_path, name, dtype, tol):
    from torchtune_b200.generation import BatchDecoder
    from torchtune_b200.modules import delete_kv_caches
    from torchtune_b200.ops.mask import AttentionMask

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
        delete_kv_caches(model)
        with torch.device(DEV):
            model.setup_caches(1, dtype, decoder_max_seq_len=len(s))
        done = 0
        for n in (2, 63, 2, 64, 9):
            x = torch.tensor([s[done : done + n]], device=DEV)
            got = model(x, mask=AttentionMask(causal=True), input_pos=torch.arange(done, done + n, device=DEV)[None])
            assert _rms_error(got[0], e[done : done + n]) < tol
            done += n
    _errors()


@pytest.mark.parametrize("dtype,tol", [(F32, 5e-5), (BF16, 8e-2)])
def test_long_decoding(tmp_path, dtype, tol):
    """Far more decoded tokens than the prompt has, over several key tiles, replayed as one graph."""
    from torchtune_b200.generation import BatchDecoder

    cfg, w, model = _load(tmp_path, "plain", dtype)
    s = np.random.default_rng(5).integers(0, cfg["vocab"], 290).tolist()
    with torch.inference_mode():
        dec = BatchDecoder(model, torch.device(DEV), dtype, 290)
        h = [dec.begin([s[:2]])[0]] + [dec.advance([t])[0] for t in s[2:]]
        assert _rms_error(dec.logits(torch.cat(h)), oracle.forward(cfg, w, s)) < tol
    _errors()


def test_greedy_generation_matches(tmp_path):
    """fp32 generation through ``generate`` picks the oracle's tokens, alone and in a padded batch (decode steps are a replayed graph)."""
    from torchtune_b200.generation import generate
    from torchtune_b200.modules import local_kv_cache

    cfg, w, model = _load(tmp_path, "looped", F32)
    prompts = [[5, 9, 2, 33, 8], [7, 1]]
    want = [oracle.greedy(cfg, w, p, 6) for p in prompts]
    batch = torch.tensor([prompts[0], [0] * 3 + prompts[1]], device=DEV)
    with local_kv_cache(model, batch_size=2, device=torch.device(DEV), dtype=F32, decoder_max_seq_len=16):
        out, _ = generate(model, batch, max_generated_tokens=6, pad_id=0, top_k=1)
        model.reset_caches()
        alone, _ = generate(model, torch.tensor(prompts[0], device=DEV), max_generated_tokens=6, pad_id=0, top_k=1)
    uncached, _ = generate(model, batch, max_generated_tokens=6, pad_id=0, top_k=1)
    assert out[0].tolist() == want[0] and out[1, 3:].tolist() == want[1] and alone[0].tolist() == want[0] and torch.equal(uncached, out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    cfg = MODELS["looped"]()
    w = oracle.weights(cfg, seed=6)
    folder = oracle.save(tmp_path / "m", cfg, w)
    rng = np.random.default_rng(2)
    seqs = {k: rng.integers(0, cfg["vocab"], n).tolist() for k, n in (("x", 31), ("y", 4), ("z", 7))}
    want = {k: oracle.forward(cfg, w, s) for k, s in seqs.items()}
    steps = [
        {"step": 0, "entries": [{"id": "x", "tokens": seqs["x"][:28], "want": [27, 0]}, {"id": "y", "tokens": seqs["y"][:3], "want": [1]}], "end": []},
        {"step": 1, "entries": [{"id": "y", "tokens": seqs["y"][3:], "want": [0]}, {"id": "x", "tokens": seqs["x"][28:29], "want": []}], "end": ["y"]},
        {"step": 2, "entries": [{"id": "x", "tokens": seqs["x"][29:30], "want": []}], "end": []},
        {"step": 3, "entries": [{"id": "x", "tokens": seqs["x"][30:], "want": [0]}], "end": ["x"]},
        {"step": 4, "entries": [{"id": "z", "tokens": seqs["z"], "want": [6, 2]}], "end": ["z"]},
    ]
    out = tmp_path / "out"
    out.mkdir()
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"], input="\n".join(map(json.dumps, steps)),
                         capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    expect = {0: [want["x"][27], want["x"][0], want["y"][1]], 1: [want["y"][3]], 3: [want["x"][30]], 4: [want["z"][6], want["z"][2]]}
    assert sorted(p.name for p in out.iterdir()) == sorted(f"{i}.f32" for i in expect)
    for i, rows in expect.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(len(rows), -1))
        assert _rms_error(got, np.stack(rows)) < (5e-5 if dtype == "float32" else 8e-2)
