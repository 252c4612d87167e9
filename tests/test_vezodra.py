"""Vezodra in the ragged engine against the plain evaluation in ``vezodra_oracle.py`` (float64, whole sequences, no cache):
every mechanism alone, prefill against token-by-token decoding, prompt portions down to two tokens, unequal batches, reuse of
cache pages and state slots, window edges, the softmax's added one, keys and writes far back, the first tokens, long decoding,
repeated spans, other sizes, and greedy generation through the scheduler.  Runs on the PyTorch branch of every op without a GPU;
``test_vezodra_gpu.py`` runs the same cases on the CUDA kernels."""
import copy
import math

import pytest
import torch

import vezodra_oracle as O
from shuffle_exchange_b200.inference.v2.config_v2 import RaggedInferenceEngineConfig
from shuffle_exchange_b200.inference.v2.engine_factory import build_engine_from_state_dict
from shuffle_exchange_b200.inference.v2.kernels import mixer_ops as M
from shuffle_exchange_b200.inference.v2.kernels import parallel_ops as P
from shuffle_exchange_b200.inference.v2.modules import heuristics
from shuffle_exchange_b200.inference.v2.modules.configs import (DSSelfAttentionConfig, MaskingType, PositionalEmbeddingType,
                                                               RotateHalfConfig)
from shuffle_exchange_b200.inference.v2.modules.implementations import DSRotarySinkAttention
from shuffle_exchange_b200.inference.v2.ragged.ragged_manager import DSStateManagerConfig
from shuffle_exchange_b200.inference.v2.scheduler import generate

DEV = "cuda" if torch.cuda.is_available() else "cpu"
F64 = torch.float64

ATT = {"type": "attention", "mixer": {"dim": 8, "heads": 6, "kv_heads": 2, "rot": {"base": 700.0, "dims": 4}, "scale": 0.4,
                                      "vdim": 8}, "mlp": {"ff": 40, "kind": "dense"}}
PAIR = {"type": "parallel",
        "mixer": {"left": {"dim": 8, "heads": 4, "kv_heads": 2, "mask": {"size": 7},
                           "rot": {"base": 90.0, "dims": 8, "scaling": {"factor": 3.0}}, "scale": 0.5, "vdim": 12},
                  "right": {"dim": 8, "heads": 3}},
        "mlp": {"ff": 24, "kind": "dense"}}


def make_cfg(layers, width=24, vocab=53, eps=1e-5, taps=3, loop=None):
    cfg = {"architecture": "Vezodra", "canon": {"taps": taps}, "layers": copy.deepcopy(layers), "norm": {"eps": eps},
           "vocab": vocab, "width": width}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


STACK = make_cfg([PAIR, ATT, dict(PAIR, mlp=None), PAIR], loop=(1, 3, 2))


def make_engine(cfg, W, dtype=torch.float32, blocks=64, block_size=4, max_live=4, max_tokens=256):
    sm = DSStateManagerConfig(max_tracked_sequences=max_live, max_ragged_sequence_count=max_live,
                              max_ragged_batch_size=max_tokens, max_context=blocks * block_size, num_kv_blocks=blocks)
    return build_engine_from_state_dict(cfg, W, RaggedInferenceEngineConfig(state_manager=sm, kv_block_size=block_size),
                                        dtype=dtype)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed(engine, uid, toks, sizes):
    """Give ``toks`` to the engine in portions of the given sizes (cycled); returns the logits of every token."""
    out, lo, i = [], 0, 0
    while lo < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - lo)
        i += 1
        out.append(engine.put([uid], [torch.tensor(toks[lo: lo + n])], logit_positions=[list(range(n))]))
        lo += n
    return torch.cat(out).double().cpu()


def row_errors(got, want):
    """Difference with the mean over the vocabulary taken off, relative to the spread of the expected logits."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def close(got, want, tol=2e-4):
    err = row_errors(got, want)
    assert err.max() < tol, f"worst row {int(err.argmax())}: {float(err.max()):.3e}"


def cuts_of(T, kind):
    return {"whole": [T], "ones": [1] * T, "mixed": [2, 1, 3] + [T - 6]}[kind]


@pytest.fixture(scope="module")
def stack():
    W = O.random_weights(STACK, seed=4)
    toks = tokens(47, STACK["vocab"], 5)
    return W, toks, O.forward(STACK, W, toks)


# ------------------------------------------------------------------------------------------------ stream, norms, filter
def _open_layers(x, add, w1, w2, filt, cuts, slot=1, wide_slots=3):
    """One sequence in portions through :func:`open_parallel_layer`, on a slot that holds another sequence's rows."""
    W, keep = x.shape[1], filt.shape[1] - 1
    state = torch.full((wide_slots, keep, W), 9.0, device=DEV) if keep else None
    outs, outs2, streams, lo = [], [], [], 0
    for n in cuts:
        sl = slice(lo, lo + n)
        r = x[sl].clone().to(DEV)
        part = P.StreamSum(y=add.y[sl].to(DEV), a=add.a[sl].to(DEV), wa=None if add.wa is None else add.wa.to(DEV),
                           b=None if add.b is None else add.b[sl].to(DEV), wb=None if add.wb is None else add.wb.to(DEV),
                           mult=add.mult)
        info = torch.tensor([[0, n, lo, slot]], dtype=torch.int32, device=DEV)
        t2s = torch.zeros(n, dtype=torch.int32, device=DEV)
        o, o2 = P.open_parallel_layer(r, part, w1.to(DEV), filt.t().contiguous().to(DEV), state, w2.to(DEV), 1e-3,
                                      torch.float32, info, t2s, n == 1)
        outs.append(o.cpu()), outs2.append(o2.cpu()), streams.append(r.cpu())
        lo += n
    if keep:
        assert torch.all(state[[0, 2]] == 9.0)
    return (torch.cat(t).double() for t in (outs, outs2, streams))


@pytest.mark.parametrize("W,taps", [(40, 4), (40, 3), (24, 2), (16, 1), (10, 4), (24, 6), (1032, 4), (7, 9)])
@pytest.mark.parametrize("pair", [True, False], ids=["averaged_pair", "single_mixer"])
def test_sums_norms_and_input_filter(W, taps, pair):
    g = torch.Generator().manual_seed(W + taps)
    T = 29
    x, y, a, b = (torch.randn(T, W, generator=g) for _ in range(4))
    w1, w2, wa, wb = (1.0 + 0.3 * torch.randn(W, generator=g) for _ in range(4))
    filt = torch.randn(W, taps, generator=g) * 0.5
    add = P.StreamSum(y=y, a=a, wa=wa, b=b, wb=wb, mult=0.5) if pair else P.StreamSum(y=y, a=a)
    X = x.double() + y.double() + (0.5 * (O.rms_norm(a.double(), wa.double(), 1e-3) + O.rms_norm(b.double(), wb.double(), 1e-3))
                                   if pair else a.double())
    h = O.rms_norm(X, w1.double(), 1e-3)
    want, want2 = h + O.causal_filter(h, filt.double()), O.rms_norm(X, w2.double(), 1e-3)
    for kind in ("whole", "ones", "mixed"):
        got, got2, stream = _open_layers(x, add, w1, w2, filt, cuts_of(T, kind))
        assert torch.allclose(stream, X, atol=1e-5)
        assert torch.allclose(got, want, atol=3e-5) and torch.allclose(got2, want2, atol=1e-5), kind


def test_filter_over_a_batch_of_unequal_sequences():
    """Sequences that bring 1 to 11 rows each, some continuing and some new, in one batch: neighbours' rows are never read."""
    g = torch.Generator().manual_seed(3)
    W, taps, eps = 24, 4, 1e-5
    lens, seen, slots = [1, 2, 11, 3, 1, 9], [0, 1, 0, 5, 2, 17], [4, 0, 6, 1, 5, 2]
    full = [torch.randn(n + s, W, generator=g) for n, s in zip(lens, seen)]
    w1, filt = 1.0 + 0.3 * torch.randn(W, generator=g), torch.randn(W, taps, generator=g)
    hs = [O.rms_norm(f.double(), w1.double(), eps) for f in full]
    state = torch.full((7, taps - 1, W), 7.0)
    for h, s, slot in zip(hs, seen, slots):
        if s:
            k = min(s, taps - 1)
            state[slot, taps - 1 - k:] = h[s - k: s].float()
    state = state.to(DEV)
    first = [sum(lens[:i]) for i in range(len(lens))]
    info = torch.tensor([[f, n, s, slot] for f, n, s, slot in zip(first, lens, seen, slots)], dtype=torch.int32, device=DEV)
    t2s = torch.arange(len(lens)).repeat_interleave(torch.tensor(lens)).to(torch.int32).to(DEV)
    rows = torch.cat([f[s:] for f, s in zip(full, seen)]).to(DEV)
    out, out2 = P.open_parallel_layer(rows, None, w1.to(DEV), filt.t().contiguous().to(DEV), state, None, eps, torch.float32,
                                      info, t2s, False)
    assert out2 is None
    want = torch.cat([(h + O.causal_filter(h, filt.double()))[s:] for h, s in zip(hs, seen)])
    assert torch.allclose(out.double().cpu(), want, atol=2e-5)
    for h, slot in zip(hs, slots):
        k = min(h.shape[0], taps - 1)
        assert torch.allclose(state[slot, taps - 1 - k:].double().cpu(), h[-k:], atol=1e-5)
    assert torch.all(state[3] == 7.0)


def test_final_norm_of_selected_rows_leaves_the_stream_alone():
    g = torch.Generator().manual_seed(8)
    x, y, a = (torch.randn(9, 40, generator=g) for _ in range(3))
    w = torch.randn(40, generator=g)
    rows = torch.tensor([7, 0, 3], dtype=torch.int32, device=DEV)
    r = x.clone().to(DEV)
    got = P.stream_norm_rows(r, P.StreamSum(y=y.to(DEV), a=a.to(DEV)), rows, w.to(DEV), 1e-4, torch.float32)
    want = O.rms_norm((x + y + a).double()[[7, 0, 3]], w.double(), 1e-4)
    assert torch.allclose(got.double().cpu(), want, atol=1e-5) and torch.equal(r.cpu(), x)
    P.stream_add(r, P.StreamSum(y=y.to(DEV)), 1e-4, torch.float32)
    assert torch.allclose(r.cpu(), x + y)


# ------------------------------------------------------------------------------------------------ rotation, attention
@pytest.mark.parametrize("dims,base,factor", [(8, 700.0, 1.0), (64, 5e4, 8.0), (6, 10.0, 2.5), (0, 10.0, 1.0)])
def test_rotation_frequencies(dims, base, factor):
    f = DSRotarySinkAttention.rotary_table(dims, base, factor)
    want = O.rotary_angles(2, {"dims": dims, "base": base, "scaling": {"factor": factor}})[1]
    assert f.dtype == torch.float32 and torch.allclose(f.double(), want, rtol=1e-7, atol=0)


@pytest.mark.parametrize("Hq,G,d,dv,dims,interleaved,norm,keys_are_values", [
    (6, 2, 8, 8, 4, True, False, True), (4, 2, 8, 12, 8, False, True, False), (3, 1, 5, 3, 4, False, True, False),
    (2, 2, 10, 10, 10, True, True, True), (4, 4, 64, 64, 64, True, False, True), (5, 5, 40, 24, 16, False, True, False),
    (1, 1, 12, 12, 0, True, False, True), (2, 1, 6, 7, 6, False, False, False)])
def test_rotated_rows_and_cache_append(Hq, G, d, dv, dims, interleaved, norm, keys_are_values, block_size=4):
    g = torch.Generator().manual_seed(d)
    T, pad = 19, 8
    v0 = (Hq + G) * d + pad
    width = (v0 + G * dv + 7) // 8 * 8
    x = torch.randn(T, width, generator=g)
    q_w, k_w = torch.randn(Hq * d, generator=g), torch.randn(G * d, generator=g)
    temp = torch.randn(Hq, generator=g)
    rot = {"dims": dims, "base": 300.0, "scaling": {"factor": 1.5}}
    X = x.double()
    q, k = X[:, pad: pad + Hq * d], X[:, pad + Hq * d: pad + (Hq + G) * d]
    v = k.clone() if keys_are_values else X[:, v0: v0 + G * dv]
    if norm:
        q, k = O.rms_norm(q, q_w.double(), 1e-3), O.rms_norm(k, k_w.double(), 1e-3)
    want_q = O.rotate(q.reshape(T, Hq, d), rot, interleaved) * temp.double()[:, None]
    want_k = O.rotate(k.reshape(T, G, d), rot, interleaved)
    freqs = DSRotarySinkAttention.rotary_table(dims, 300.0, 1.5).to(DEV)
    for cuts in ([T], [1, 2, 5, 11]):
        pages = (T + block_size - 1) // block_size
        kc = torch.full((pages + 1, block_size, G, d), 9.0, device=DEV)
        vc = torch.full((pages + 1, block_size, G, dv), 9.0, device=DEV)
        tables = torch.arange(pages, 0, -1, dtype=torch.int32, device=DEV).view(1, pages)
        got, lo = [], 0
        for n in cuts:
            t2s = torch.zeros(n, dtype=torch.int32, device=DEV)
            pos = torch.arange(lo, lo + n, dtype=torch.int32, device=DEV)
            got.append(P.rope_append(x[lo: lo + n].to(DEV), pad, pad + Hq * d, pad + Hq * d if keys_are_values else v0,
                                     q_w.to(DEV) if norm else None, k_w.to(DEV) if norm else None, freqs, interleaved,
                                     temp.to(DEV), kc, vc, t2s, pos, tables, Hq, G, d, dv, 1e-3).cpu())
            lo += n
        assert torch.allclose(torch.cat(got).double(), want_q, atol=3e-5)
        order = tables[0].long().cpu()
        assert torch.allclose(kc.cpu()[order].reshape(-1, G, d)[:T].double(), want_k, atol=3e-5)
        assert torch.allclose(vc.cpu()[order].reshape(-1, G, dv)[:T].double(), v.reshape(T, G, dv), atol=1e-6)
        assert torch.all(kc[0] == 9.0)


class _Batch:
    """The metadata of one ragged batch without an engine."""

    def __init__(self, portions, tables):
        seqs, pos = [], []
        for s, (lo, n) in enumerate(portions):
            seqs += [s] * n
            pos += list(range(lo, lo + n))
        self._t2s = torch.tensor(seqs, dtype=torch.int32, device=DEV)
        self._pos = torch.tensor(pos, dtype=torch.int32, device=DEV)
        self._tables = tables

    def token_to_seq(self): return self._t2s
    def token_positions(self): return self._pos
    def block_tables(self): return self._tables


def _attention_module(window=0, unit=False, from_keys=False, H=4, G=2, d=8, dv=None, dims=8, gate=False, scale=0.5):
    from shuffle_exchange_b200.inference.v2.inference_utils import DtypeEnum
    return heuristics.instantiate_attention(DSSelfAttentionConfig(
        max_tokens=64, n_heads_q=H, n_heads_kv=G, head_size=d, v_head_size=dv or d, max_sequences=4, scale_factor=scale,
        input_dtype=DtypeEnum.fp32, output_dtype=DtypeEnum.fp32,
        masking_type=MaskingType.sliding_window if window else MaskingType.causal,
        masking_args={"size": window} if window else {},
        positional_embedding_type=PositionalEmbeddingType.rotate_half if dims else PositionalEmbeddingType.none,
        positional_embedding_config=RotateHalfConfig(theta_base=50.0, rotate_dim=dims), split_cache=True, unit_sink=unit,
        values_from_keys=from_keys, output_gate=gate, output_gate_per_head=gate), None)


def _run_module(mod, x, cuts, block_size=4, weights=None):
    c = mod._config
    pages = (x.shape[0] + block_size - 1) // block_size
    kc = torch.full((pages, block_size, c.n_heads_kv, c.head_size), 5.0, device=DEV)
    vc = torch.full((pages, block_size, c.n_heads_kv, c.v_head_size), 5.0, device=DEV)
    tables = torch.arange(pages - 1, -1, -1, dtype=torch.int32, device=DEV).view(1, pages)
    out, lo = [], 0
    for n in cuts:
        out.append(mod(x[lo: lo + n].to(DEV).contiguous(), (kc, vc), _Batch([(lo, n)], tables), None, weights).cpu())
        lo += n
    return torch.cat(out).double()


@pytest.mark.parametrize("window", [1, 2, 5, 9, 64])
def test_one_key_that_stands_out_just_inside_and_just_outside_the_window(window):
    """Key 3 scores far above every other: the queries up to ``3 + window - 1`` return its value and the next one does not."""
    H = G = 1
    d = 4
    T = 3 + min(window, 12) + 4
    x = torch.zeros(T, 3 * d)
    x[:, :d] = torch.tensor([1.0, 0, 0, 0])                      # queries
    x[3, d: 2 * d] = torch.tensor([60.0, 0, 0, 0])               # key 3
    x[:, 2 * d:] = torch.arange(T, dtype=torch.float32)[:, None] + 1.0
    mod = _attention_module(window=window, H=H, G=G, d=d, dims=0, scale=1.0)
    for cuts in ([T], [1] * T, [4, T - 4]):
        out = _run_module(mod, x, cuts)
        for t in range(T):
            inside = 3 <= t < 3 + window
            if inside:
                assert torch.allclose(out[t], torch.full((d,), 4.0, dtype=F64), atol=1e-5), (t, out[t])
            else:
                keys = [j for j in range(t + 1) if t - j < window]
                assert torch.allclose(out[t], torch.full((d,), sum(k + 1.0 for k in keys) / len(keys), dtype=F64), atol=1e-5)


def test_one_joins_the_softmax_denominator_before_any_shift():
    """Scores of -3 with two keys: weights e^-3 / (1 + 2 e^-3); scores of +50: the one does not matter; -200: all vanish."""
    d = 2
    for score in (-3.0, 0.0, 50.0, -200.0):
        x = torch.zeros(2, 2 * d)
        x[:, 0], x[:, d] = score, 1.0
        x[1, d + 1] = 2.0
        mod = _attention_module(unit=True, from_keys=True, H=1, G=1, d=d, dims=0, scale=1.0)
        for cuts in ([2], [1, 1]):
            out = _run_module(mod, x, cuts)
            e = math.exp(score)
            want = torch.tensor([[e / (1 + e), 0.0], [2 * e / (1 + 2 * e), 2 * e / (1 + 2 * e)]], dtype=F64)
            assert torch.allclose(out, want, atol=1e-6), score


def test_gate_per_head_and_values_that_are_not_rotated():
    g = torch.Generator().manual_seed(2)
    H, G, d, T = 4, 2, 8, 23
    mod = _attention_module(unit=True, from_keys=True, H=H, G=G, d=d, dims=4, gate=True)
    assert mod.gate_column == 48 and mod.projection_width == 56
    x = torch.randn(T, mod.projection_width, generator=g)
    X = x.double()
    q, k = X[:, : H * d].view(T, H, d), X[:, H * d: (H + G) * d].view(T, G, d)
    rot = {"dims": 4, "base": 50.0}
    want = O.attend(O.rotate(q, rot, False), O.rotate(k, rot, False), k, 0.5, 0, True)
    want = (want * torch.sigmoid(X[:, 48: 48 + H])[:, :, None]).reshape(T, H * d)
    for cuts in ([T], [1, 2, 20]):
        assert torch.allclose(_run_module(mod, x, cuts), want, atol=2e-5)


# ------------------------------------------------------------------------------------------------ delta rule with removal
def _removal_case(H, n, rank, T, seed):
    g = torch.Generator().manual_seed(seed)
    B = (H * n + 7) // 8 * 8
    proj = torch.randn(T, 5 * B + rank, generator=g)
    P_ = {"w1": torch.eye(rank, dtype=F64), "w2": torch.randn(H * n, rank, generator=g).double() / math.sqrt(rank),
          "w0": torch.randn(H * n, generator=g).double() - 1.0, "a.b": torch.randn(H * n, generator=g).double()}
    return proj, B, P_


def _removal_oracle(proj, B, P_, H, n, rank):
    T, X = proj.shape[0], proj.double()
    cols = [X[:, i * B: i * B + H * n] for i in range(5)]
    r, k, v = (c.reshape(T, H, n) for c in cols[:3])
    low = X[:, 5 * B: 5 * B + rank]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(low) @ P_["w2"].T + P_["w0"])).view(T, H, n)
    rate = torch.sigmoid(cols[3] + P_["a.b"]).view(T, H, n)
    return torch.stack([O.removal_recurrence(r[:, i], k[:, i], v[:, i], decay[:, i], rate[:, i]) for i in range(H)],
                       dim=1).reshape(T, H * n)


def _removal_run(proj, B, P_, H, n, rank, cuts, slot=1):
    state = torch.full((3, H, n, n), 5.0, device=DEV)
    w2, w0, ab = (t.float().contiguous().to(DEV) for t in (P_["w2"].T, P_["w0"], P_["a.b"]))
    outs, lo = [], 0
    for c in cuts:
        info = torch.tensor([[0, c, lo, slot]], dtype=torch.int32, device=DEV)
        buf = P.removal_prepare(proj[lo: lo + c].to(DEV), 0, B, 2 * B, 3 * B, 5 * B, w2, w0, ab, H, n, math.exp(-0.5), 1e-6)
        outs.append(P.removal_recurrence(buf, state, info, c == 1).cpu())
        lo += c
    assert torch.all(state[[0, 2]] == 5.0)
    return torch.cat(outs).double()


@pytest.mark.parametrize("H,n,rank", [(3, 8, 6), (1, 5, 1), (2, 40, 16), (1, 130, 20), (2, 64, 8), (2, 33, 3), (1, 132, 4)])
def test_delta_rule_with_separate_decay_and_removal(H, n, rank):
    T = 27
    proj, B, P_ = _removal_case(H, n, rank, T, n)
    want = _removal_oracle(proj, B, P_, H, n, rank)
    for cuts in ([T], [1] * T, [1, 2, 8, 9, 7], [16, 11]):
        got = _removal_run(proj, B, P_, H, n, rank, cuts)
        assert torch.allclose(got, want, atol=1e-4, rtol=1e-4), float((got - want).abs().max())


def test_both_terms_read_the_old_state_and_the_write_uses_the_raw_key():
    """Two steps by hand: k = 2 e0 written with value 3, then the same key again with removal rate a and decay w: the state's
    entry becomes w * 6 - a * 6 + 2 * v, not (w - a w) * 6 nor a write of the unit key."""
    n, a_raw, w0 = 4, 0.3, -0.7
    proj = torch.zeros(2, 5 * 8 + 1)
    proj[:, 0] = 1.0                                              # r = e0
    proj[:, 8] = 2.0                                              # k = 2 e0
    proj[0, 16], proj[1, 16] = 3.0, 5.0                           # v
    P_ = {"w2": torch.zeros(n, 1, dtype=F64), "w0": torch.full((n,), w0, dtype=F64), "a.b": torch.full((n,), a_raw, dtype=F64)}
    sig = lambda z: 1 / (1 + math.exp(-z))
    w, a = math.exp(-math.exp(-0.5) * sig(w0)), sig(a_raw)
    u2 = 4.0 / (4.0 + 1e-6)                                       # square of the unit key's entry
    want0 = 6.0
    want1 = w * 6.0 - a * u2 * 6.0 + 10.0
    for cuts in ([2], [1, 1]):
        got = _removal_run(proj, 8, P_, 1, n, 1, cuts)
        assert abs(got[0, 0] - want0) < 1e-5 and abs(got[1, 0] - want1) < 1e-5
    assert torch.allclose(got, _removal_oracle(proj, 8, P_, 1, n, 1), atol=1e-5)


def test_an_old_write_on_a_channel_that_keeps_is_read_hundreds_of_tokens_later():
    """Decays of ~1 (w0 = -40) and no removal (a.b = -40): what the first token wrote is still there at token 400; on a
    channel with full decay exp(-e^-0.5) per token it is gone."""
    n, T = 4, 400
    proj = torch.zeros(T, 5 * 8 + 1)
    proj[0, 8:10] = 1.0                                           # k of the first token: channels 0 and 1
    proj[0, 16:20] = torch.tensor([1.0, 2.0, 3.0, 4.0])
    proj[T - 2, 1] = 1.0                                          # read channel 1, then channel 0
    proj[T - 1, 0] = 1.0
    w0 = torch.full((n,), -40.0, dtype=F64)
    w0[1] = 40.0
    P_ = {"w2": torch.zeros(n, 1, dtype=F64), "w0": w0, "a.b": torch.full((n,), -40.0, dtype=F64)}
    for cuts in ([T], [200, 2] + [1] * 198):
        got = _removal_run(proj, 8, P_, 1, n, 1, cuts)
        assert torch.allclose(got[T - 1], torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=F64), atol=1e-4)
        assert got[T - 2].abs().max() < 1e-6


def test_recurrence_over_a_batch_of_unequal_sequences():
    H, n, rank = 2, 8, 3
    lens, slots = [1, 17, 2, 8], [2, 0, 3, 1]
    cases = [_removal_case(H, n, rank, L + 4, 70 + L) for L in lens]
    B, P_ = cases[0][1], cases[0][2]
    want = [_removal_oracle(c[0], B, P_, H, n, rank) for c in cases]
    w2, w0, ab = (t.float().contiguous().to(DEV) for t in (P_["w2"].T, P_["w0"], P_["a.b"]))
    state = torch.full((5, H, n, n), 5.0, device=DEV)

    def step(rows, seen):
        first = [sum(r.shape[0] for r in rows[:i]) for i in range(len(rows))]
        info = torch.tensor([[f, r.shape[0], s, slot] for f, r, s, slot in zip(first, rows, seen, slots)], dtype=torch.int32,
                            device=DEV)
        buf = P.removal_prepare(torch.cat(rows).to(DEV), 0, B, 2 * B, 3 * B, 5 * B, w2, w0, ab, H, n, math.exp(-0.5), 1e-6)
        o = P.removal_recurrence(buf, state, info, all(r.shape[0] == 1 for r in rows)).double().cpu()
        return [o[f: f + r.shape[0]] for f, r in zip(first, rows)]
    got = [[x] for x in step([c[0][:L] for c, L in zip(cases, lens)], [0] * 4)]
    for i in range(4):                                            # then every sequence decodes, all in one batch
        for lst, x in zip(got, step([c[0][L + i: L + i + 1] for c, L in zip(cases, lens)], [L + i for L in lens])):
            lst.append(x)
    for lst, w in zip(got, want):
        assert torch.allclose(torch.cat(lst), w, atol=1e-4, rtol=1e-4)
    assert torch.all(state[4] == 5.0)


# ------------------------------------------------------------------------------------------------ layers and the stack
@pytest.mark.parametrize("layer", [ATT, PAIR, dict(ATT, mlp=None), dict(PAIR, mlp=None)],
                         ids=["attention", "pair", "attention_alone", "pair_alone"])
def test_one_layer_of_each_kind(layer):
    cfg = make_cfg([layer])
    W = O.random_weights(cfg, seed=1)
    toks = tokens(23, cfg["vocab"], 2)
    want = O.forward(cfg, W, toks)
    eng = make_engine(cfg, W)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [3, 1, 2]), want)


def test_stream_after_every_layer_run(stack):
    W, toks, _ = stack
    handed = []
    O.forward(STACK, W, toks, handed)
    eng = make_engine(STACK, W)
    eng.model().layer_outputs = []
    feed(eng, 1, toks, [len(toks)])
    assert len(handed) == len(eng.model().layer_outputs) == 6
    for got, want in zip(eng.model().layer_outputs, handed):
        assert torch.allclose(got.double().cpu(), want, atol=2e-4, rtol=1e-4)


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (0, 3, 3), (1, 2, 4), (2, 3, 2), (0, 1, 2)])
def test_repeated_spans_keep_a_cache_and_a_state_per_pass(loop):
    cfg = make_cfg([PAIR, ATT, dict(PAIR, mlp=None)], loop=loop)
    W = O.random_weights(cfg, seed=6)
    toks = tokens(25, cfg["vocab"], 7)
    want = O.forward(cfg, W, toks)
    eng = make_engine(cfg, W)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [5, 1, 2, 1]), want)
    n_runs = len(O.runs(cfg))
    assert len(eng.model().kv_cache_config(4).layer_shapes) == n_runs


def test_what_lies_just_outside_the_window_does_not_matter_and_just_inside_does():
    """One pair whose recurrent half is muted and whose input filter is zero: the last position's logits change with the
    token ``size - 1`` back and not with the token ``size`` back, in a prompt and decoded alone."""
    size = 7
    layer = dict(PAIR, mlp=None)
    layer["mixer"] = dict(PAIR["mixer"], left=dict(PAIR["mixer"]["left"], scale=2.0))
    cfg = make_cfg([layer], taps=2)
    W = O.random_weights(cfg, seed=13)
    W["l0.canon1"] = torch.zeros_like(W["l0.canon1"])
    W["l0.mix.right.out"] = torch.zeros_like(W["l0.mix.right.out"])
    toks = tokens(21, cfg["vocab"], 14)
    base = O.forward(cfg, W, toks)
    eng, uid = make_engine(cfg, W, max_live=2), 0
    for back, matters in ((size, False), (size - 1, True), (size + 3, False), (1, True)):
        other = list(toks)
        other[-1 - back] = (other[-1 - back] + 17) % cfg["vocab"]
        want = O.forward(cfg, W, other)
        assert bool((want[-1] - base[-1]).abs().max() > 1e-3) == matters
        for sizes in ([len(toks)], [len(toks) - 3, 1], [4, 2, 5]):
            uid += 1
            got = feed(eng, uid, other, sizes)
            close(got, want)
            assert bool((got[-1] - base[-1]).abs().max() > 1e-3) == matters
            eng.flush(uid)


def test_far_keys_and_old_writes_decide_the_logits():
    """Attention with its score scale raised tenfold, so that single keys carry most of a query's weight wherever they lie among
    hundreds, and a delta rule whose channels barely decay: prompt rows, portions cut at page and window borders and beside
    them, and decode tokens follow the plain evaluation."""
    att = dict(ATT, mixer=dict(ATT["mixer"], scale=4.0), mlp=None)
    pair = dict(PAIR, mlp=None)
    pair["mixer"] = {"left": dict(PAIR["mixer"]["left"], scale=3.0, mask={"size": 64}), "right": PAIR["mixer"]["right"]}
    cfg = make_cfg([att, pair], vocab=31)
    W = O.random_weights(cfg, seed=21)
    W["l1.mix.right.w0"] = torch.full_like(W["l1.mix.right.w0"], -9.0)
    W["l1.mix.right.a.b"] = torch.full_like(W["l1.mix.right.a.b"], -9.0)
    toks = tokens(300, cfg["vocab"], 22)
    want = O.forward(cfg, W, toks)
    eng = make_engine(cfg, W, block_size=8, blocks=128, max_tokens=320)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [245] + [1] * 55), want)
    close(feed(eng, 3, toks, [64, 37, 3, 2, 40, 4, 127, 1, 7, 15]), want)
    other = tokens(40, cfg["vocab"], 23) + toks[40:]                 # another beginning gives other logits at the end
    assert (O.forward(cfg, W, other)[-1] - want[-1]).abs().max() > 1e-2


# ------------------------------------------------------------------------------------------------ cache, state, batches
def test_prefill_equals_token_by_token_decoding(stack):
    W, toks, want = stack
    eng = make_engine(STACK, W)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [1]), want)


@pytest.mark.parametrize("sizes", [[2], [3, 5], [7, 1, 1, 2], [16, 2, 9], [40, 1], [1, 2]])
def test_prompt_portions(stack, sizes):
    W, toks, want = stack
    eng = make_engine(STACK, W)
    close(feed(eng, 1, toks, sizes), want)


def test_unequal_requests_in_one_batch_equal_each_alone():
    W = O.random_weights(STACK, seed=9)
    reqs = {u: tokens(n, STACK["vocab"], 10 + u) for u, n in ((1, 19), (2, 3), (3, 31), (4, 8))}
    want = {u: O.forward(STACK, W, t) for u, t in reqs.items()}
    eng = make_engine(STACK, W)
    at = {u: 0 for u in reqs}
    got = {u: [] for u in reqs}
    plan = [{1: 5, 3: 2}, {1: 1, 2: 3, 3: 9, 4: 2}, {1: 13, 3: 1, 4: 1}, {3: 1, 4: 1}, {3: 1, 4: 4}, {3: 17}]
    for step in plan:                                              # 2 is left out, 1 ends, a step of single tokens only
        uids = list(step)
        toks = [torch.tensor(reqs[u][at[u]: at[u] + n]) for u, n in step.items()]
        out = eng.put(uids, toks, logit_positions=[list(range(n)) for n in step.values()]).double().cpu()
        k = 0
        for u, n in step.items():
            got[u].append(out[k: k + n])
            k, at[u] = k + n, at[u] + n
    for u in reqs:
        assert at[u] == len(reqs[u])
        close(torch.cat(got[u]), want[u])


def test_a_step_that_asks_for_no_logits_still_advances(stack):
    W, toks, want = stack
    eng = make_engine(STACK, W)
    for lo, n in ((0, 9), (9, 1), (10, 2)):
        out = eng.put([1], [torch.tensor(toks[lo: lo + n])], logit_positions=[[]])
        assert out.shape == (0, STACK["vocab"])
    close(feed_rest(eng, 1, toks, 12), want[12:])


def feed_rest(eng, uid, toks, lo):
    return eng.put([uid], [torch.tensor(toks[lo:])], logit_positions=[list(range(len(toks) - lo))]).double().cpu()


def test_pages_and_state_slots_are_reused():
    """As many pages as the longest request and its neighbour need, two state slots: every later request gets pages and a
    slot that an earlier one filled, in another order, and must come out as if alone -- also one shorter than the filter."""
    W = O.random_weights(STACK, seed=3)
    eng = make_engine(STACK, W, blocks=10, block_size=4, max_live=2)
    for i, n in enumerate((20, 23, 1, 26, 2, 29)):
        toks = tokens(n, STACK["vocab"], 20 + i)
        other = tokens(6, STACK["vocab"], 40 + i)
        eng.put([100 + i], [torch.tensor(other)])                 # a neighbour that holds the other slot and two pages
        got = feed(eng, i, toks, [7, 1, 2] if i % 2 else [1, 1, 4])
        close(got, O.forward(STACK, W, toks))
        eng.flush(i)
        eng.flush(100 + i)
        assert eng.free_blocks == 10


def test_long_decoding(stack):
    W, _, _ = stack
    toks = tokens(150, STACK["vocab"], 6)
    want = O.forward(STACK, W, toks)
    eng = make_engine(STACK, W)
    close(feed(eng, 1, toks, [9] + [1] * 200), want)


ODD = [
    # nothing a multiple of 8, one head, a window of one token, part of the channels rotated, no scaling entry
    (make_cfg([{"type": "parallel",
                "mixer": {"left": {"dim": 5, "heads": 1, "kv_heads": 1, "mask": {"size": 1},
                                   "rot": {"base": 77.0, "dims": 4}, "scale": 1.7, "vdim": 3},
                          "right": {"dim": 7, "heads": 1}}, "mlp": {"ff": 9, "kind": "dense"}},
               {"type": "attention", "mixer": {"dim": 6, "heads": 3, "kv_heads": 1, "rot": {"base": 12.0, "dims": 2},
                                               "scale": 0.9, "vdim": 6}, "mlp": {"ff": 11, "kind": "dense"}}],
              width=10, vocab=17, eps=1e-3, taps=5), 3),
    # many heads of unequal kinds, values wider than keys, one tap, key sizes above 32
    (make_cfg([{"type": "parallel",
                "mixer": {"left": {"dim": 16, "heads": 8, "kv_heads": 8, "mask": {"size": 16},
                                   "rot": {"base": 1e4, "dims": 8, "scaling": {"factor": 16.0}}, "scale": 0.2, "vdim": 40},
                          "right": {"dim": 36, "heads": 2}}, "mlp": None},
               dict(ATT, mlp={"ff": 64, "kind": "dense"})], width=64, vocab=29, taps=1, loop=(0, 2, 2)), 8),
    # a stack of one kind; long filter; a window longer than the sequence
    (make_cfg([{"type": "parallel",
                "mixer": {"left": {"dim": 4, "heads": 2, "kv_heads": 1, "mask": {"size": 500},
                                   "rot": {"base": 30.0, "dims": 4, "scaling": {"factor": 1.0}}, "scale": 0.5, "vdim": 4},
                          "right": {"dim": 4, "heads": 4}}, "mlp": None}] * 2, width=8, vocab=11, taps=11), 1),
    (make_cfg([ATT, ATT], width=16, vocab=23, taps=2), 4),
]


@pytest.mark.parametrize("cfg,rank", ODD, ids=["no_multiples_of_8_window_1", "one_tap_wide_values", "pairs_only_long_filter",
                                               "attention_only"])
def test_other_sizes(cfg, rank):
    W = O.random_weights(cfg, seed=8, rank=rank)
    toks = tokens(21, cfg["vocab"], 9)
    want = O.forward(cfg, W, toks)
    eng = make_engine(cfg, W, block_size=8)
    close(feed(eng, 1, toks, [len(toks)]), want)
    close(feed(eng, 2, toks, [4, 1, 2]), want)


def test_configuration_is_read_into_the_layer_specs():
    from shuffle_exchange_b200.inference.v2.checkpoint.huggingface_engine import PlainModelConfig
    from shuffle_exchange_b200.inference.v2.model_implementations.vezodra import VezodraPolicy
    spec = VezodraPolicy(PlainModelConfig(STACK)).spec(PlainModelConfig(STACK))
    p, a, q, _ = spec.layers
    left, right = p.parts
    assert (a.kind, a.n_heads, a.n_heads_kv, a.key_dim, a.value_dim, a.attn_scale, a.rot_dims, a.rot_base, a.rot_divisor) == (
        "rotary_attention", 6, 2, 8, 8, 0.4, 4, 700.0, 1.0)
    assert a.rot_interleaved and a.values_from_keys and a.unit_sink and a.head_scale and a.gate_per_head and a.window == 0
    assert (p.kind, left.kind, left.n_heads, left.n_heads_kv, left.key_dim, left.value_dim, left.window, left.rot_divisor) == (
        "pair", "rotary_attention", 4, 2, 8, 12, 7, 3.0)
    assert left.qk_row_norm and not (left.rot_interleaved or left.values_from_keys or left.unit_sink or left.out_gate)
    assert (right.kind, right.n_heads, right.key_dim, right.value_dim) == ("removal_delta", 3, 8, 8)
    assert right.decay_rate == pytest.approx(math.exp(-0.5), rel=1e-12)
    assert (p.ff_dim, p.ff_activation, q.ff_dim) == (24, "silu", 0)
    assert (spec.block_form, spec.input_conv_taps, spec.norm_eps) == ("parallel", 3, 1e-5)
    assert [i for i, _ in spec.runs()] == [0, 1, 2, 1, 2, 3]
    with pytest.raises(ValueError, match="taps"):
        W = O.random_weights(make_cfg([ATT], taps=4))
        make_engine(make_cfg([ATT], taps=3), W)


def test_bf16_serving_stays_near_the_exact_evaluation(stack):
    W, toks, want = stack
    eng = make_engine(STACK, W, dtype=torch.bfloat16)
    for uid, sizes in ((1, [len(toks)]), (2, [5, 1, 2])):
        assert row_errors(feed(eng, uid, toks, sizes), want).max() < 0.06


# ------------------------------------------------------------------------------------------------ generation
def _check_greedy(prompt, out, W, cfg):
    seq = list(prompt)
    for tok in out:
        logits = O.forward(cfg, W, seq)[-1]
        top2 = logits.topk(2).values
        if top2[0] - top2[1] > 1e-3:                           # a near tie may go either way in 32-bit
            assert tok == int(logits.argmax())
        seq.append(tok)


def test_greedy_generation_through_the_scheduler():
    W = O.random_weights(STACK, seed=12)
    prompts = [tokens(n, STACK["vocab"], 30 + n) for n in (5, 17, 2, 9, 12)]          # five requests, four may be live
    eng = make_engine(STACK, W, blocks=40, block_size=4, max_live=4, max_tokens=16)
    got = generate(eng, prompts, max_new_tokens=6, max_batch_tokens=16, max_prompt_portion=7)
    for p, out in zip(prompts, got):
        _check_greedy(p, out, W, STACK)
        assert len(out) == 6
    assert eng.free_blocks == 40 and eng._state_manager.n_tracked_sequences == 0


def write_checkpoint(folder, cfg, W):
    """``config.json`` + ``model.safetensors`` (bf16): 8-byte header length, JSON header, tensor bytes."""
    import json
    import struct
    with open(folder / "config.json", "w") as f:
        json.dump(cfg, f)
    meta, blobs, off = {}, [], 0
    for name, t in W.items():
        b = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        meta[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    header = json.dumps(meta).encode()
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(header)) + header + b"".join(blobs))


def _run_command(cmd, stdin=None):
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", cmd[0]), *cmd[1:]], input=stdin, capture_output=True,
                       text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    return r.stdout.splitlines()


def test_command_line_generation_from_a_checkpoint_folder(tmp_path):
    import json
    W = O.random_weights(STACK, seed=14)
    write_checkpoint(tmp_path, STACK, W)
    prompts = [[5, 17, 3], [9, 9, 1, 2, 3, 4, 5, 6, 7]]
    cmd = ["sxb_generate", "--model", str(tmp_path), "--max-new-tokens", "4", "--dtype", "float32"]
    for p in prompts:
        cmd += ["--prompt", ",".join(map(str, p))]
    lines = [json.loads(x) for x in _run_command(cmd) if x.startswith("{")]
    assert [x["prompt"] for x in lines] == prompts
    for p, x in zip(prompts, lines):
        _check_greedy(p, x["generated"], W, STACK)
        assert len(x["generated"]) == 4


def test_replaying_a_schedule_of_steps_from_a_checkpoint_folder(tmp_path):
    """``bin/trace_run``: five requests through a pool of four 64-token pages and four state slots -- portions beside single
    tokens, a request left out of a step, requests that end and whose pages and slot the next one takes; every wanted position
    must equal the plain evaluation of its request alone."""
    import json
    import numpy as np
    W = O.random_weights(STACK, seed=15)
    model = tmp_path / "model"
    model.mkdir()
    write_checkpoint(model, STACK, W)
    reqs = {name: tokens(n, STACK["vocab"], 50 + n) for name, n in (("a", 40), ("b", 9), ("c", 23), ("d", 1), ("e", 30))}
    plan = [({"a": 17, "b": 2}, []), ({"a": 3, "b": 7, "c": 5, "d": 1}, ["b", "d"]), ({"a": 1, "c": 2, "e": 11}, []),
            ({"a": 19, "e": 1}, ["a"]), ({"c": 1, "e": 1}, []), ({"c": 15, "e": 17}, ["c", "e"])]
    at = {k: 0 for k in reqs}
    steps, wanted = [], []
    for i, (portion, end) in enumerate(plan):
        entries = []
        for name, n in portion.items():
            want = sorted({0, n - 1, n // 2})
            entries.append({"id": name, "tokens": reqs[name][at[name]: at[name] + n], "want": want})
            wanted += [(i, name, at[name] + w) for w in want]
            at[name] += n
        steps.append(json.dumps({"step": i, "entries": entries, "end": end}))
    assert at == {k: len(v) for k, v in reqs.items()}
    out = tmp_path / "out"
    cmd = ["trace_run", "--model", str(model), "--dtype", "float32", "--out", str(out), "--max-tokens", "256"]
    lines = _run_command(cmd + ([] if torch.cuda.is_available() else ["--device", "cpu"]), "\n".join(steps) + "\n")
    assert [x for x in lines if x.startswith("done")] == [f"done {i}" for i in range(len(plan))]
    full = {name: O.forward(STACK, W, t) for name, t in reqs.items()}
    got = {i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, STACK["vocab"])).double()
           for i in range(len(plan))}
    row = {i: 0 for i in got}
    for i, name, p in wanted:
        close(got[i][row[i]: row[i] + 1], full[name][p: p + 1])
        row[i] += 1
    assert all(row[i] == got[i].shape[0] for i in got)
