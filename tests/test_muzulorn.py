"""The Muzulorn design in the engine against the plain numpy statement of it (tests/plain/muzulorn_plain.py).

Every test makes its own small configuration and random weights.  Each body runs twice: with the PyTorch stand-ins
for the kernels on the CPU (the parts, the cache manager, the batching), and on the GPU with the real kernels (marked
``gpu``).  The configurations differ from one another in everything a configuration can say: the order of the three kinds of
mixers, one to six streams, keys and values read by one, two or no later layer, key sizes unlike value sizes, query and
key latents of any size, part or all or none of the shared key part rotated, windows shorter and longer than a page and none, states
in one, some or as many groups as heads, convolutions of one to five taps, routers that choose one, some or all of
their experts, with and without the shared one, layers without a feed-forward, a model without pairs of tokens.
"""

import json
import os

import numpy as np
import pytest
import torch

import sllm_b200.models  # noqa: F401  (registers the parts and the architecture)
from tests import traces
from tests.plain import muzulorn_plain as plain
from tests.test_kidolorn import CLOSE_CALL, CUTS, _bf16_exact, _portions, _requests, _step, _to, compare, dev, dtypes_on, make_model  # noqa: F401
from tests.test_sezopel import _paged, _relative, _term


def _att(heads, kv, dim, vdim, scale, bias_max, softcap=None, q_temp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max}
    if softcap is not None:
        m["softcap"] = softcap
    if q_temp is not None:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, rot=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return m


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _layer(mixer, mlp):
    typ = "mamba2" if "state" in mixer else "latent_attention" if "kv_rank" in mixer else "attention"
    return {"type": typ, "mixer": mixer, "mlp": mlp}


def _config(vocab, width, streams, mult, layers, pairs=None, eps=1e-5):
    c = {"architecture": "Muzulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "residual_mult": mult, "layers": layers}
    if pairs is not None:
        c["embedding"] = {"bigram": {"buckets": pairs[0], "mul_prev": pairs[1], "mul_cur": pairs[2]}}
    return c


CONFIG_A = _config(290, 80, 3, 0.7, [              # keys and values read one and four layers on; every kind of mixer and of feed-forward
    _layer(_att(6, 2, 24, 40, 0.2, 21, 5.0, (0.4, 16)), _moe(6, 2, 40, 24)),
    _layer(_att(6, 2, 24, 40, 0.3, 33, 3.0, (0.7, 9), kv_from=0), None),
    _layer(_ssm(6, 16, 20, 3, 3, 4), _dense(72)),
    _layer(_lat(4, 24, 8, 40, 36, 48, 0.15, 19, (1000.0, 8)), _moe(4, 4, 16)),
    _layer(_att(6, 2, 24, 40, 0.25, 40, 8.0, None, kv_from=0), _moe(5, 1, 24, 40)),
], pairs=(101, 29, 3))
CONFIG_B = _config(210, 128, 4, 0.5, [             # cached heads of 64 and 128 on pages of 16: the tensor-core attention forms on the GPU (bfloat16)
    _layer(_ssm(4, 32, 64, 1, 4, 1), _moe(8, 2, 32, 64)),
    _layer(_att(8, 2, 64, 48, 0.12, 50, 10.0, (0.3, 32)), _dense(192)),
    _layer(_att(4, 1, 96, 128, 0.1, 17, None, (0.5, 20)), _dense(128)),
    _layer(_lat(8, 16, 16, 32, 64, 48, 0.2, 40, (10000.0, 16)), _moe(8, 3, 32, 32)),
    _layer(_att(8, 2, 64, 48, 0.15, 100, 5.0, None, kv_from=1), None),
    _layer(_lat(2, 32, 32, 32, 32, 96, 0.15, 70, (500.0, 32)), _dense(64)),
    _layer(_att(4, 1, 96, 128, 0.08, 64, 15.0, None, kv_from=2), _dense(320)),
], pairs=(997, 1000003, 7919), eps=1e-6)
ODD = _config(77, 50, 2, 1.3, [                    # sizes that are multiples of nothing; one head; a window of one and two tokens
    _layer(_lat(3, 10, 6, 14, 11, 21, 0.4, 2, (50.0, 6)), _dense(33)),
    _layer(_ssm(5, 9, 7, 5, 5, 3), _moe(3, 2, 14, 9)),
    _layer(_att(3, 3, 10, 7, 0.3, 12, 4.0, (1.0, 7)), None),
    _layer(_lat(1, 12, 6, 9, 5, 13, 0.3, 1, (50.0, 4)), _moe(3, 3, 10, 7)),
    _layer(_ssm(1, 18, 33, 1, 2, 1), _dense(9)),
    _layer(_att(3, 3, 10, 7, 0.4, 200, 2.0, None, kv_from=2), _moe(4, 1, 11)),
], pairs=(5, 3, 2), eps=1e-4)
BARE = _config(90, 64, 1, 1.0, [                   # one stream, no pairs of tokens, no caps and factors, no feed-forwards, no window, nothing rotated
    _layer(_att(4, 4, 32, 32, 0.2, 30), None),
    _layer(_ssm(2, 16, 16, 2, 1, 2), None),
    _layer(_lat(5, 16, 0, 16, 24, 16, 0.25, None), None)])
SIX = _config(120, 72, 6, 0.4, [_layer(_ssm(4, 24, 32, 2, 4, 2), _dense(100)), _layer(_lat(2, 32, 16, 16, 40, 64, 0.2, 33, (100.0, 8)), _moe(16, 5, 8, 8))],
              pairs=(64, 2, 1))
MID = _config(1000, 352, 4, 0.6, [                 # a few hundred channels, no power of two: the products' tensor-core forms between tiny and real
    _layer(_att(12, 3, 64, 64, 0.1, 90, 12.0, (0.5, 24)), _dense(1024)),
    _layer(_ssm(10, 48, 64, 2, 4, 2), _moe(8, 3, 96, 160)),
    _layer(_att(12, 3, 64, 64, 0.12, 48, 20.0, None, kv_from=0), _dense(512)),
    _layer(_lat(5, 48, 16, 64, 112, 80, 0.125, 45, (20000.0, 16)), _moe(8, 2, 96, 96)),
], pairs=(5000, 37, 19))
CONFIGS = {"A": (CONFIG_A, 16), "B": (CONFIG_B, 16), "odd": (ODD, 8), "bare": (BARE, 4), "six": (SIX, 32), "mid": (MID, 16)}


def plain_logits(d, reqs, margins=None):
    cfg, w = plain.load_model(d)
    out = {}
    for r, ids in reqs.items():
        m = []
        out[r] = plain.forward(ids, cfg, w, margins=m).astype(np.float32)
        if margins is not None:
            margins[r] = np.min(np.stack(m), axis=0) if m else np.full(len(ids), np.inf)
    return out


def models_for(tmp_path, config, dev, reqs, seed=5, edit=None):
    """(dtype, model folder, plain logits, routers' margins) for every dtype the device runs."""
    d = make_model(tmp_path, config, seed=seed, edit=edit)
    margins = {}
    want = plain_logits(d, reqs, margins)
    for dtype in dtypes_on(dev):
        yield dtype, d, want, margins


def _bind(part, w, prefix=""):
    part.bind(lambda rel: torch.from_numpy(np.ascontiguousarray(w[prefix + rel], dtype=np.float32)))
    return part


# ---- configuration, plan, weights ---------------------------------------------------------------------------

def test_config_plan_and_cache_needs():
    from sllm_b200.config import ConfigError, architecture_of
    from sllm_b200.models.causal_lm import CausalLM
    from sllm_b200.parts import PagedKV, SlotState
    arch = architecture_of(CONFIG_A)
    cfg = arch.config_cls.from_dict(CONFIG_A)
    assert cfg.to_dict() == CONFIG_A
    p = arch.plan(cfg)
    assert len(p.layers) == 5 and [e.cache_from for e in p.run_list] == [None, 0, None, None, 0] and p.position is None
    assert p.streams == 3 and (p.token_pairs.name, p.token_pairs.buckets, p.token_pairs.mul_prev, p.token_pairs.mul_cur) == ("bigram", 101, 29, 3)
    assert p.ignored_names == ("l1.norm2", "l1.hc2.in", "l1.hc2.out", "l1.hc2.mix") and "ffn" not in p.layers[1].parts
    m = CausalLM(p, dtype=torch.float32, device="cpu")
    assert m.cache_needs() == [("own", (PagedKV(2, 40, None), SlotState((1,), "previous_token"))), ("borrow", 0),
                               ("own", (SlotState((6, 20, 16), "ssm"), SlotState((6 * 16 + 2 * 3 * 20, 2), "conv"))),
                               ("own", PagedKV(1, 56, 19, values=False)), ("borrow", 0)]
    assert CausalLM(p, dtype=torch.bfloat16, device="cpu").cache_needs()[3] == ("own", PagedKV(1, 64, 19, values=False))
    shapes = {s.name: tuple(s.shape) for s in m.tensor_specs()}
    assert set(n for n in shapes if n.startswith("l1.")) == {"l1.norm1", "l1.hc1.in", "l1.hc1.out", "l1.hc1.mix", "l1.mix.q", "l1.mix.q.b",
                                                            "l1.mix.q.norm", "l1.mix.rel", "l1.mix.o", "l1.mix.o.b"}
    assert shapes["embed"] == shapes["head"] == (290, 80) and shapes["bigram"] == (102, 80) and shapes["final.norm"] == (80,)
    assert shapes["l0.mix.k.norm"] == (48,) and shapes["l0.mix.q.norm"] == (144,) and shapes["l0.mix.v.b"] == (80,) and shapes["l0.mix.rel"] == (None, 6)
    assert shapes["l0.mlp.shared.sg"] == (1, 80) and shapes["l0.mlp.shared.down"] == (80, 24) and shapes["l0.mlp.router.b"] == (6,)
    assert "l3.mlp.shared.sg" not in shapes and shapes["l3.mlp.e3.gate"] == (16, 80)
    assert shapes["l2.mix.in"] == (96 + 96 + 120 + 6, 80) and shapes["l2.mix.conv"] == (216, 3) and shapes["l2.mix.norm"] == (96,)
    assert shapes["l3.mix.dq"] == (36, 80) and shapes["l3.mix.uq"] == (4 * 32, 36) and shapes["l3.mix.dkv"] == (56, 80) and shapes["l3.mix.g"] == (160, 80)

    def edited(path, value):
        c = json.loads(json.dumps(CONFIG_A))
        at = c
        for k in path[:-1]:
            at = at[k]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return c
    for bad in (edited(("layers", 0, "mixer", "kv_heads"), 4), edited(("layers", 4, "mixer", "kv_from"), 2), edited(("layers", 4, "mixer", "kv_from"), 1),
                edited(("layers", 4, "mixer", "kv_from"), 4), edited(("layers", 4, "mixer", "dim"), 32), edited(("layers", 1, "mixer", "vdim"), 24),
                edited(("layers", 1, "mixer", "kv_heads"), 1), edited(("layers", 0, "mixer", "scale"), None), edited(("layers", 0, "mixer", "bias_max"), None),
                edited(("layers", 0, "mixer", "q_temp", "every"), None), edited(("layers", 2, "mixer", "groups"), 4), edited(("layers", 2, "mixer", "norm_groups"), 5),
                edited(("layers", 2, "mixer", "state"), None), edited(("layers", 3, "mixer", "rot", "dims"), 7), edited(("layers", 3, "mixer", "rot", "dims"), 10),
                edited(("layers", 3, "mixer", "q_rank"), None), edited(("layers", 3, "mixer", "mask", "size"), None), edited(("layers", 0, "mlp", "kind"), "other"),
                edited(("layers", 0, "mlp", "router", "top"), 7), edited(("layers", 0, "mlp", "shared", "ff"), None), edited(("layers", 0, "type"), "other"),
                edited(("streams",), None), edited(("residual_mult",), None), edited(("norm",), None), edited(("layers",), []),
                edited(("embedding", "bigram", "buckets"), None)):
        with pytest.raises(ConfigError):
            arch.config_cls.from_dict(bad)


# ---- each mechanism alone: an operation or a part against the plain function ------------------------------------------

@pytest.mark.parametrize("H,copies,buckets,mul_prev,mul_cur", [(50, 3, 7, 5, 3), (64, 1, 101, 29, 1), (300, 4, 65536, 2654435761, 40503), (33, None, 1, 4, 9), (16, 6, 12, 0, 1)])
def test_rows_by_pairs_of_tokens_across_portions_and_slots(dev, H, copies, buckets, mul_prev, mul_cur):
    """Every copy of a token's stream is its embedding row plus its pair's; the token before comes from the same portion, from the request's
    state, or does not exist.  Two requests in portions down to one token, one slot that another request used before."""
    import sllm_b200.ops as ops
    from sllm_b200.config.plan import TokenPairs
    rng = np.random.default_rng(H)
    V = 41
    w = _bf16_exact({"embed": rng.standard_normal((V, H)), "bigram": rng.standard_normal((buckets + 1, H))})
    lens, slots = {0: 110, 1: 21}, {0: 2, 1: 0}
    ids = {s: rng.integers(0, V, n).tolist() for s, n in lens.items()}
    ids[0][:6] = [V - 1, V - 1, 0, 0, V - 1, 3]
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    want = {s: plain.embedding(i, cfg, w) for s, i in ids.items()}
    before = torch.full((4, 1), 17.0, device=dev)                   # (what another request left: a first token must not see it)
    to = _to(dev)
    for td in (torch.float32,) if dev == "cpu" else (torch.float32, torch.bfloat16):
        table, pair = to(w["embed"]).to(td), to(w["bigram"]).to(td)

        def run(rows, step):
            step.token_ids = torch.tensor(sum((ids[s][a:b] for s, a, b in rows), []), dtype=torch.int32, device=dev)
            x = ops.embed_streams(table, step, 1.0, copies, pair, before, TokenPairs("bigram", buckets, mul_prev, mul_cur))
            if copies is None:
                return x.cpu().numpy()
            assert tuple(x.shape[1:]) == (copies, H) and all(torch.equal(x[:, 0], x[:, c]) for c in range(copies))
            return x[:, 0].cpu().numpy()
        got = _portions(dev, lens, slots, CUTS, run)
        for s in lens:
            np.testing.assert_allclose(got[s], want[s], rtol=1e-6, atol=1e-6)
        assert float(before[1, 0]) == 17.0
    x = ops.embed_streams(to(w["embed"]), _step(dev, [3], [0]), 2.5, copies)          # no pairs: the rows alone, scaled
    np.testing.assert_allclose((x if copies is None else x[:, 0]).cpu().numpy(), np.repeat(w["embed"][:1] * 2.5, 3, axis=0), rtol=1e-6)


@pytest.mark.parametrize("s,W", [(1, 50), (2, 96), (3, 51), (4, 1000), (4, 2048), (5, 64), (6, 1500), (7, 33), (8, 72), (16, 40), (4, 12800)])
def test_streams_are_mixed_and_read_as_one_sum(dev, s, W):
    """A term (whole, and as a stack of partial sums) joins the streams, which mix all at once from the old ones ([from, to]: the mix is not
    symmetric), and their weighted sum is normed for the reader; each half alone; chosen rows without a stream written."""
    import sllm_b200.ops as ops
    rng = np.random.default_rng(s * W)
    T, eps, mult = 7, 1e-2, 0.6
    x, y = rng.standard_normal((T, s, W)) * 2, rng.standard_normal((3, T, W))
    w = {"in": rng.standard_normal(s) * 0.3, "mix": rng.standard_normal((s, s)), "out": rng.standard_normal(s)}
    gain, into = rng.standard_normal(W) * 0.3, rng.standard_normal(s) * 0.05
    to = _to(dev)
    new = plain.connect(x.transpose(1, 0, 2), w, "", mult, lambda u: y.sum(0)).transpose(1, 0, 2)
    want_h = plain.norm_around_zero(np.einsum("tsw,s->tw", new, into), gain, eps)
    args = (to(w["mix"]), to(w["out"] * mult), to(into), to(1 + gain), eps)
    for term in (to(y.sum(0)), to(y)):
        for dtype in (torch.float32, torch.bfloat16):
            streams = to(x)
            h = ops.streams_step(streams, term, *args, dtype)
            assert h.dtype == dtype
            np.testing.assert_allclose(streams.cpu().numpy(), new, rtol=3e-5, atol=3e-5)
            tol = 5e-5 if dtype == torch.float32 else 1e-2
            np.testing.assert_allclose(h.float().cpu().numpy(), want_h, rtol=tol, atol=tol)
        streams = to(x)
        rows = torch.tensor([6, 0, 3], dtype=torch.int32, device=dev)
        h = ops.streams_step(streams, term, *args, torch.float32, rows=rows)
        np.testing.assert_allclose(h.cpu().numpy(), want_h[[6, 0, 3]], rtol=5e-5, atol=5e-5)
        np.testing.assert_array_equal(streams.cpu().numpy(), x.astype(np.float32))
        assert ops.streams_step(streams, term, args[0], args[1], None, None, 0.0, None) is None
        np.testing.assert_allclose(streams.cpu().numpy(), new, rtol=3e-5, atol=3e-5)
    streams = to(x)
    h = ops.streams_step(streams, None, None, None, *args[2:], torch.float32)
    np.testing.assert_allclose(h.cpu().numpy(), plain.norm_around_zero(np.einsum("tsw,s->tw", x, into), gain, eps), rtol=5e-5, atol=5e-5)
    np.testing.assert_array_equal(streams.cpu().numpy(), x.astype(np.float32))


def test_distance_buckets():
    """The whole-number form against the formula's logarithms (where those are not within rounding of a border), and on borders that are exact:
    with 16 buckets up to 128, distances 16, 32 and 64 each open the bucket that 8 times a power of sqrt 2 names."""
    from sllm_b200.parts.side_by_side import distance_buckets
    for B, D in ((16, 111), (16, 128), (32, 1000), (8, 5), (2, 2), (2, 50), (64, 100), (6, 4000), (12, 7), (5, 30)):
        got = distance_buckets(B, D)
        assert len(got) == D + 1 and got[-1] == B - 1 and all(b - a in range(B) for a, b in zip(got, got[1:]))
        for n in range(D + 1):
            if n >= B // 2:
                pos = np.log(n / (B // 2)) / np.log(D / (B // 2)) * (B - B // 2)
                if abs(pos - round(pos)) < 1e-9:
                    continue
            assert got[n] == plain.distance_bucket(n, B, D), (B, D, n)
    b = distance_buckets(16, 128)
    assert (b[15], b[16], b[31], b[32], b[63], b[64]) == (9, 10, 11, 12, 13, 14) and b[:9] == [0, 1, 2, 3, 4, 5, 6, 7, 8]
    for B, D in ((1, 10), (8, 4), (8, 3)):
        with pytest.raises(ValueError):
            distance_buckets(B, D)


def _rel(rng, nq, n, spread=1.0):
    """A table by distance whose neighbours differ: a distance that is off by one shows."""
    import sllm_b200.ops as ops
    t = rng.standard_normal((n, nq)) * spread
    return t, lambda nkv, dev: ops.DistanceBias(torch.from_numpy(t.astype(np.float32)), nkv, dev)


def _attend(kf, vf, tables, seq, pos, q, ps, nq, nkv, scale, cap, bias, window=None, sink=None):
    """One token's attention [nq, D] over its pages, plainly."""
    js = np.arange(max(0, pos - window + 1) if window else 0, pos + 1)
    kk, vv = kf[tables[seq, js // ps], :, js % ps], vf[tables[seq, js // ps], :, js % ps]
    out = []
    for h in range(nq):
        s = kk[:, h // (nq // nkv)] @ q[h] * scale
        if cap:
            s = cap * np.tanh(s / cap)
        if bias is not None:
            s = s + bias[np.minimum(pos - js, bias.shape[0] - 1), h]
        out.append(plain.softmax(s, None if sink is None else sink[h]) @ vv[:, h // (nq // nkv)])
    return np.stack(out)


@pytest.mark.parametrize("D,ps,dtype,nq,nkv,cap,n,spread", [
    (27, 4, "float32", 3, 1, 4.0, 10, 2.0), (64, 16, "bfloat16", 8, 2, 6.0, 117, 2.0), (64, 16, "bfloat16", 24, 1, 30.0, 65, 1.0),
    (128, 32, "bfloat16", 6, 3, 0.0, 300, 1.0), (32, 8, "bfloat16", 2, 2, 7.0, 33, 2.0), (56, 16, "float32", 4, 4, 0.0, 64, 2.0),
    (16, 16, "bfloat16", 5, 1, 3.0, 1, 1.0), (128, 64, "bfloat16", 16, 2, 20.0, 17, 3.0), (64, 8, "bfloat16", 3, 3, 0.0, 2, 2.0),
    (80, 16, "bfloat16", 4, 2, 8.0, 900, 1.0), (64, 16, "bfloat16", 8, 2, 6.0, 90, 30.0)])
def test_scores_with_a_bias_by_distance_over_keys_near_and_far(dev, D, ps, dtype, nq, nkv, cap, n, spread):
    """Every attention form (single tokens and portions in one step, scattered pages) with a bias per head and distance behind scale and cap, tables
    shorter than a key tile, longer than every context, and of one row; with a spread that the bounded maximum of the tcgen05 form would not
    take (30: another form runs).  For every query one key stands out in its first head: the first token, one a page back, one at
    the table's last own distance, its own."""
    import sllm_b200.ops as ops
    if dev == "cpu" and dtype != "float32":
        pytest.skip("the stand-ins are float32")
    rng = np.random.default_rng(D + nq + n)
    scale = 0.3
    cases = [(1, 1), (1, 2), (1, 700), (1, 3 * ps), (1, 3 * ps + 1), (2, 2), (5, 5), (2, 2 * ps + 1), (ps + 3, 4 * ps + 2), (3, 333), (150, 150),
             (130, 400), (1, 64), (1, 65)]
    q_lens, ctx = [c[0] for c in cases], [c[1] for c in cases]
    k, v, tables, g = _paged(dev, nkv, D, ps, ctx, rng)
    T = sum(q_lens)
    q = rng.standard_normal((T, nq, D)).astype(np.float32)
    bias, make = _rel(rng, nq, n, spread)
    rel = make(nkv, dev)
    assert rel.narrow == (spread < 30)
    step = _step(dev, q_lens, list(range(len(cases))), ctx, g)
    pos, seq = step.positions.cpu().numpy(), step.seq_of_token.cpu().numpy()
    for t in range(T):
        j = (0, max(pos[t] - ps, 0), max(pos[t] - n + 2, 0), pos[t])[t % 4]
        k[tables[seq[t], j // ps], 0, j % ps] = q[t, 0] * (12.0 / np.sqrt(D))
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    qd, kd, vd = (torch.from_numpy(a).to(dev).to(td).contiguous() for a in (q.reshape(T, nq * D), k, v))
    got = ops.paged_attention(qd, kd, vd, step, 0, nq, nkv, D, scale, None, softcap=cap, rel=rel).float().cpu().numpy().reshape(T, nq, D)
    qf, kf, vf = (a.float().cpu().numpy().astype(np.float64) for a in (qd, kd, vd))
    tol = 3e-5 if dtype == "float32" else 3e-2
    for t in range(T):
        want = _attend(kf, vf, tables, seq[t], pos[t], qf.reshape(T, nq, D)[t], ps, nq, nkv, scale, cap, bias)
        np.testing.assert_allclose(got[t], want, rtol=tol, atol=tol, err_msg=f"token {t} (position {pos[t]})")


@pytest.mark.gpu
@pytest.mark.parametrize("D,nq,nkv,q_len,ctx,n", [(64, 4, 1, 40, 2500, 129), (128, 8, 2, 33, 2304, 1500), (64, 4, 4, 1, 5000, 700), (128, 4, 2, 1, 3001, 65), (32, 4, 2, 1, 2100, 100)])
def test_a_bias_by_distance_over_a_context_cut_into_ranges(D, nq, nkv, q_len, ctx, n):
    """Few rows over thousands of keys: ranges of the context run as CTAs of their own, some of them all far, some near."""
    import sllm_b200.ops as ops
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    dev, ps, cap, scale = "cuda:0", 16, 9.0, 0.4
    rng = np.random.default_rng(ctx)
    k, v, tables, g = _paged(dev, nkv, D, ps, [ctx, 70], rng)
    q_lens, T = [q_len, 1], q_len + 1
    q = rng.standard_normal((T, nq, D)).astype(np.float32)
    step = _step(dev, q_lens, [0, 1], [ctx, 70], g)
    pos, seq = step.positions.cpu().numpy(), step.seq_of_token.cpu().numpy()
    for t in range(q_len):
        j = 7 + 31 * t
        k[tables[0, j // ps], 0, j % ps] = q[t, 0] * (16.0 / np.sqrt(D))
    bias, make = _rel(rng, nq, n, 2.0)
    qd, kd, vd = (torch.from_numpy(a).to(dev).bfloat16().contiguous() for a in (q.reshape(T, nq * D), k, v))
    got = ops.paged_attention(qd, kd, vd, step, 0, nq, nkv, D, scale, None, softcap=cap, rel=make(nkv, dev)).float().cpu().numpy().reshape(T, nq, D)
    qf, kf, vf = (a.float().cpu().numpy().astype(np.float64) for a in (qd, kd, vd))
    for t in range(T):
        np.testing.assert_allclose(got[t], _attend(kf, vf, tables, seq[t], pos[t], qf.reshape(T, nq, D)[t], ps, nq, nkv, scale, cap, bias), rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("H,G,dk,dv,ps,dtype,buckets,limit,every", [
    (6, 2, 24, 40, 4, "float32", 8, 30, 16), (3, 3, 10, 7, 8, "float32", 16, 115, 5), (8, 2, 64, 48, 16, "bfloat16", 16, 60, 32), (4, 1, 96, 128, 16, "bfloat16", 32, 90, 7),
    (2, 2, 16, 16, 16, "bfloat16", 2, 9, 64), (1, 1, 33, 12, 16, "float32", 6, 200, 1), (4, 2, 144, 100, 16, "bfloat16", 12, 40, 20)])
def test_attention_and_a_second_layer_on_the_same_keys_and_values(dev, H, G, dk, dv, ps, dtype, buckets, limit, every):
    """The whole mixer through its part: biases, norms over all of the query and all of the key, the query's factor across many of its steps,
    the bias by distance; then a second mixer without keys and values that reads what the first one cached, with a scale, cap, factor, buckets and limit of
    its own.  Two requests in portions down to one token on scattered pages; eps counts beside the projections' size."""
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import MIXERS, GroupView, LayerCache
    if dev == "cpu" and dtype != "float32":
        pytest.skip("the stand-ins are float32")
    rng = np.random.default_rng(dk + H)
    W, eps = 72, 0.05
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    m1 = _att(H, G, dk, dv, 0.5 / np.sqrt(dk) * 3, limit, 4.0, (0.5, every))
    m2 = _att(H, G, dk, dv, 0.3, limit + 5, None, (-0.2, every + 3), kv_from=0)

    def weights(own, B):
        w = {"m.q": rng.standard_normal((H * dk, W)) * 0.1, "m.q.b": rng.standard_normal(H * dk) * 0.5, "m.q.norm": 1 + 0.3 * rng.standard_normal(H * dk),
             "m.rel": rng.standard_normal((B, H)), "m.o": rng.standard_normal((W, H * dv)) * 0.2, "m.o.b": rng.standard_normal(W)}
        if own:
            w.update({"m.k": rng.standard_normal((G * dk, W)) * 0.1, "m.k.b": rng.standard_normal(G * dk) * 0.5, "m.k.norm": 1 + 0.3 * rng.standard_normal(G * dk),
                      "m.v": rng.standard_normal((G * dv, W)) * 0.3, "m.v.b": rng.standard_normal(G * dv)})
        return _bf16_exact(w)

    def build(m, w, shared):
        spec = {"hidden_size": W, "heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": m["scale"], "eps": eps, "norm_over": "projection", "bias": True,
                "out_bias": True, "softcap": m.get("softcap"), "q_temp": m["q_temp"], "distance_bias": m["bias_max"], "shared_kv": shared,
                "rotary": None, "max_positions": 512}
        return _bind(MIXERS.build(PartSpec("normed_attention", spec), dtype=td, device=dev), w, "m.")
    w1, w2 = weights(True, buckets), weights(False, buckets + 4)
    first, second = build(m1, w1, False), build(m2, w2, True)
    assert first.cache_need() == second.cache_need() and first.cache_need().head_dim >= max(dk, dv)
    lens = {0: 110, 1: 37}
    xs = {s: _bf16_exact({"x": rng.standard_normal((n, W))})["x"] for s, n in lens.items()}
    want = {}
    for s, x in xs.items():
        kv = plain.keys_values(x, w1, "m.", m1, eps)
        want[s] = np.concatenate([plain.attention(x, w1, "m.", m1, eps, kv), plain.attention(x, w2, "m.", m2, eps, kv)], axis=1)
    D = first.cache_need().head_dim
    _, _, tables, _ = _paged(dev, G, D, ps, list(lens.values()), rng)
    kc, vc = (torch.full((int(tables.max()) + 1, G, ps, D), 3.0, dtype=td, device=dev) for _ in range(2))
    cache = LayerCache(group=0, k=kc, v=vc)
    to = _to(dev)
    row = {s: i for i, s in enumerate(lens)}

    def run(rows, step):
        slot_map = np.concatenate([[tables[row[s], p // ps] * ps + p % ps for p in range(a, b)] for s, a, b in rows]).astype(np.int32)
        step.groups = [GroupView(ps, torch.from_numpy(tables[[row[s] for s, _, _ in rows]]).to(dev), torch.from_numpy(slot_map).to(dev))]
        x = to(np.concatenate([xs[s][a:b] for s, a, b in rows])).to(td)
        return np.concatenate([_term(first.forward(x, step, cache, None)), _term(second.forward(x, step, cache, None, write_cache=False))], axis=1)
    got = _portions(dev, lens, {0: 0, 1: 1}, CUTS, run)
    for s in lens:
        for part in (slice(0, W), slice(W, 2 * W)):
            if dtype == "float32":
                np.testing.assert_allclose(got[s][:, part], want[s][:, part], rtol=5e-4, atol=5e-4)
            else:
                e = _relative(got[s][:, part], want[s][:, part])
                assert e.max() < 0.05 and np.quantile(e, 0.9) < 0.02, (s, float(e.max()), int(e.argmax()))


@pytest.mark.parametrize("H,dk,dr,dv,q_rank,rank,window,dims,ps,dtype", [
    (4, 24, 8, 40, 36, 48, 19, 8, 4, "float32"), (3, 10, 6, 14, 9, 21, 1, 4, 8, "float32"), (8, 16, 16, 32, 64, 48, 16, 16, 16, "bfloat16"),
    (2, 32, 32, 32, 48, 96, 33, 32, 16, "bfloat16"), (1, 16, 2, 16, 12, 30, 2, 2, 16, "float32"), (2, 64, 64, 64, 96, 192, 40, 64, 16, "bfloat16"),
    (5, 12, 0, 8, 16, 16, 7, 0, 16, "float32"), (4, 128, 64, 128, 128, 512, 50, 64, 16, "bfloat16"), (3, 16, 8, 24, 40, 40, None, 6, 8, "float32")])
def test_latent_attention_in_a_window(dev, H, dk, dr, dv, q_rank, rank, window, dims, ps, dtype):
    """Queries through a latent of their own, pairs of neighbouring channels rotated (all, part or none of the shared key part), a window whose edge
    single tokens and portions meet at every place in a page, a sink, a gate per channel.  Pages the window has passed are poisoned.  Scores are
    several units wide, so that for some tokens the key at the window's edge takes most of the weight and an edge that is off by one shows."""
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import MIXERS, GroupView, LayerCache
    if dev == "cpu" and dtype != "float32":
        pytest.skip("the stand-ins are float32")
    rng = np.random.default_rng(rank + H)
    W, eps, base = 72, 0.02, 300.0
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    m = _lat(H, dk, dr, dv, q_rank, rank, 4.0 / np.sqrt(dk + dr), window, (base, dims) if dims else None)
    w = _bf16_exact({"m.dq": rng.standard_normal((q_rank, W)) * 0.2, "m.dq.norm": 1 + 0.3 * rng.standard_normal(q_rank),
                     "m.uq": rng.standard_normal((H * (dk + dr), q_rank)) * q_rank ** -0.5, "m.dkv": rng.standard_normal((rank + dr, W)) * 0.12,
                     "m.dkv.norm": 1 + 0.3 * rng.standard_normal(rank), "m.uk": rng.standard_normal((H * dk, rank)) * rank ** -0.5,
                     "m.uv": rng.standard_normal((H * dv, rank)) * rank ** -0.5, "m.sink": rng.standard_normal(H) * 2,
                     "m.g": rng.standard_normal((H * dv, W)) * 0.2, "m.o": rng.standard_normal((W, H * dv)) * 0.2})
    spec = {"hidden_size": W, "heads": H, "dim": dk, "vdim": dv, "q_rank": q_rank, "kv_rank": rank, "scale": m["scale"], "eps": eps, "gate": "element",
            "sink": True, "rot_dim": dr, "window": window,
            "rotary": {"theta": base, "rotary_dim": dims, "interleaved": True, "max_positions": 512} if dims else None}
    mixer = _bind(MIXERS.build(PartSpec("latent_attention", spec), dtype=td, device=dev), w, "m.")
    need = mixer.cache_need()
    assert need.window == window and need.head_dim >= rank + dr
    lens = {0: 110, 1: 37}
    xs = {s: _bf16_exact({"x": rng.standard_normal((n, W))})["x"] for s, n in lens.items()}
    want = {s: plain.latent_attention(x, w, "m.", m, eps) for s, x in xs.items()}
    if dtype == "float32":                          # the queries' norm alone (a layer that writes no latents of its own runs it so)
        import sllm_b200.ops as ops
        z = rng.standard_normal((5, q_rank + 9))
        got = ops.norm_cols(_to(dev)(z), 4, q_rank, _to(dev)(w["m.dq.norm"]), eps, torch.float32).cpu().numpy()
        np.testing.assert_allclose(got, plain.norm(z[:, 4:4 + q_rank], w["m.dq.norm"], eps), rtol=2e-5, atol=2e-5)
    if window is not None and window > 1:           # the edge matters here: one key more or less changes rows by more than the tolerance
        for other in (window - 1, window + 1):
            d = _relative(plain.latent_attention(xs[0], w, "m.", dict(m, mask={"size": other}), eps), want[0])
            assert np.quantile(d[window + 1:], 0.95) > 0.03 and d.max() > 0.2
    D = need.head_dim
    _, _, tables, _ = _paged(dev, 1, D, ps, list(lens.values()), rng)
    kc = torch.full((int(tables.max()) + 1, 1, ps, D), 3.0, dtype=td, device=dev)
    cache = LayerCache(group=0, k=kc, v=kc)
    to = _to(dev)
    row = {s: i for i, s in enumerate(lens)}

    def run(rows, step):
        bt = tables.copy()
        for s, a, b in rows:
            gone = max(0, a - (window or 1 << 30) + 1) // ps
            kc[torch.from_numpy(bt[row[s], :gone].astype(np.int64)).to(dev)] = float("nan")
            bt[row[s], :gone] = -1
        slot_map = np.concatenate([[tables[row[s], p // ps] * ps + p % ps for p in range(a, b)] for s, a, b in rows]).astype(np.int32)
        step.groups = [GroupView(ps, torch.from_numpy(bt[[row[s] for s, _, _ in rows]]).to(dev), torch.from_numpy(slot_map).to(dev))]
        return _term(mixer.forward(to(np.concatenate([xs[s][a:b] for s, a, b in rows])).to(td), step, cache, None))
    got = _portions(dev, lens, {0: 0, 1: 1}, CUTS, run)
    for s in lens:
        if dtype == "float32":
            np.testing.assert_allclose(got[s], want[s], rtol=5e-4, atol=5e-4)
        else:
            e = _relative(got[s], want[s])
            assert e.max() < 0.08 and np.quantile(e, 0.9) < 0.03, (s, float(e.max()), int(e.argmax()))


@pytest.mark.parametrize("D,ps,dtype,nq,nkv,window", [
    (27, 4, "float32", 3, 1, 10), (64, 16, "bfloat16", 8, 2, 100), (64, 16, "bfloat16", 24, 1, 64), (128, 32, "bfloat16", 6, 3, 33), (32, 8, "bfloat16", 2, 2, 21),
    (128, 16, "bfloat16", 16, 1, 130), (64, 8, "bfloat16", 4, 4, 1), (160, 16, "bfloat16", 6, 1, 50), (128, 64, "bfloat16", 5, 1, 17)])
def test_window_with_a_sink_over_every_form(dev, D, ps, dtype, nq, nkv, window):
    """Single tokens and portions in one step, hundreds of tokens into a request; pages the window has passed are given back and poisoned.  For every
    query the key at the window's edge, the one just outside, or its own stands out in its first head."""
    import sllm_b200.ops as ops
    if dev == "cpu" and dtype != "float32":
        pytest.skip("the stand-ins are float32")
    rng = np.random.default_rng(D + nq + window)
    scale = 0.3
    cases = [(1, 1), (1, 2), (1, 700), (1, 3 * ps + 1), (2, 2), (5, 5), (2, 2 * ps + 1), (ps + 3, 4 * ps + 2), (3, 333), (150, 150), (130, 400), (40, 640), (1, window), (1, window + 1)]
    q_lens, ctx = [c[0] for c in cases], [c[1] for c in cases]
    k, v, tables, g = _paged(dev, nkv, D, ps, ctx, rng)
    T = sum(q_lens)
    q = rng.standard_normal((T, nq, D)).astype(np.float32)
    full = tables.copy()
    for s, (n, c) in enumerate(cases):
        gone = max(0, c - n - window + 1) // ps
        k[tables[s, :gone]] = v[tables[s, :gone]] = np.nan
        tables[s, :gone] = -1
    g.block_tables.copy_(torch.from_numpy(tables))
    step = _step(dev, q_lens, list(range(len(cases))), ctx, g)
    pos, seq = step.positions.cpu().numpy(), step.seq_of_token.cpu().numpy()
    for t in range(T):
        j = (max(pos[t] - window + 1, 0), max(pos[t] - window, 0), pos[t])[t % 3]
        if tables[seq[t], j // ps] >= 0:
            k[tables[seq[t], j // ps], 0, j % ps] = q[t, 0] * (12.0 / np.sqrt(D))
    sink = rng.standard_normal(nq) * 2
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    qd, kd, vd = (torch.from_numpy(a).to(dev).to(td).contiguous() for a in (q.reshape(T, nq * D), k, v))
    got = ops.paged_attention(qd, kd, vd, step, 0, nq, nkv, D, scale, window, sink=_to(dev)(sink)).float().cpu().numpy().reshape(T, nq, D)
    qf, kf, vf = (a.float().cpu().numpy().astype(np.float64) for a in (qd, kd, vd))
    tol = 3e-5 if dtype == "float32" else 3e-2
    for t in range(T):
        want = _attend(kf, vf, full, seq[t], pos[t], qf.reshape(T, nq, D)[t], ps, nq, nkv, scale, 0.0, None, window, sink)
        np.testing.assert_allclose(got[t], want, rtol=tol, atol=tol, err_msg=f"token {t} (position {pos[t]})")


def _state_space_case(rng, dev, H, dv, N, G, taps, parts, W=40, eps=1e-2):
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import MIXERS, LayerCache
    inner, C = H * dv, H * dv + 2 * G * N
    # decays from one that forgets at once to one that all but never does, steps from tiny to large
    w = _bf16_exact({"m.in": rng.standard_normal((inner + C + H, W)) * 0.25, "m.conv": rng.standard_normal((C, taps)) * 0.5, "m.conv.b": rng.standard_normal(C) * 0.5,
                     "m.dt_bias": rng.standard_normal(H), "m.A_log": np.linspace(-9.0, 2.5, H) if H > 1 else np.array([-5.0]), "m.D": rng.standard_normal(H),
                     "m.norm": 1 + 0.3 * rng.standard_normal(inner), "m.o": rng.standard_normal((W, inner)) * inner ** -0.5})
    m = _ssm(H, dv, N, G, taps, parts)
    mixer = _bind(MIXERS.build(PartSpec("mamba2", dict(m, hidden_size=W, eps=eps)), dtype=torch.float32, device=dev), w, "m.")
    slots = 5
    cache = LayerCache(states={"ssm": torch.zeros((slots, H, N, dv), dtype=torch.float32, device=dev)})
    if taps > 1:
        cache.states["conv"] = torch.zeros((slots, C, taps - 1), dtype=torch.float32, device=dev)
    return w, m, mixer, cache, W, eps


@pytest.mark.parametrize("H,dv,N,G,taps,parts", [(1, 64, 64, 1, 4, 1), (6, 16, 20, 3, 3, 4), (5, 10, 7, 5, 5, 5), (2, 130, 12, 1, 2, 2), (80, 16, 16, 8, 4, 1),
                                                 (4, 32, 128, 2, 1, 4), (2, 128, 128, 2, 4, 1), (1, 80, 256, 1, 4, 2), (3, 96, 160, 1, 6, 3)])
def test_state_space_in_portions_and_slots(dev, H, dv, N, G, taps, parts):
    """The mixer through its part (convolution with bias, step sizes, decays, grouped B and C, the skip, the gate before the norm in parts) in
    portions down to one token; one slot's states stay untouched."""
    rng = np.random.default_rng(N + H)
    w, m, mixer, cache, W, eps = _state_space_case(rng, dev, H, dv, N, G, taps, parts)
    assert len(mixer.cache_need()) == (2 if taps > 1 else 1)
    lens, slots = {0: 110, 1: 21}, {0: 1, 1: 2}
    xs = {s: rng.standard_normal((n, W)) for s, n in lens.items()}
    to = _to(dev)
    run = lambda rows, step: _term(mixer.forward(to(np.concatenate([xs[s][a:b] for s, a, b in rows])), step, cache, None))
    got = _portions(dev, lens, slots, CUTS, run)
    for s in lens:
        np.testing.assert_allclose(got[s], plain.mamba2(xs[s], w, "m.", m, eps), rtol=1e-3, atol=1e-3)
    assert all(float(st[0].abs().max()) == 0.0 for st in cache.states.values())


@pytest.mark.parametrize("H,dv,N,G,taps,parts", [(2, 64, 64, 1, 4, 1), (3, 30, 48, 3, 4, 1), (4, 128, 128, 2, 2, 4), (6, 100, 16, 2, 3, 2), (2, 64, 100, 1, 4, 1), (3, 7, 33, 1, 5, 3),
                                                 (1, 24, 200, 1, 4, 1), (8, 64, 128, 1, 4, 2)])
def test_state_space_over_long_portions_beside_short_ones(dev, H, dv, N, G, taps, parts):
    """Long portions run in chunks on the GPU, short ones and single tokens token by token: portions that end beside a chunk's border and on either
    side of where chunks begin to be used, alone and beside others in one step, each going on from its state rows."""
    rng = np.random.default_rng(N + dv)
    w, m, mixer, cache, W, eps = _state_space_case(rng, dev, H, dv, N, G, taps, parts)
    cuts = [(200, 1, 64), (1, 129, 95), (97, 1, 96), (1, 2, 65), (127, 128, 1), (95, 192, 1)]
    lens, slots = {s: sum(c[s] for c in cuts) for s in range(3)}, {0: 2, 1: 0, 2: 3}
    xs = {s: rng.standard_normal((n, W)) for s, n in lens.items()}
    to = _to(dev)
    run = lambda rows, step: _term(mixer.forward(to(np.concatenate([xs[s][a:b] for s, a, b in rows])), step, cache, None))
    got = _portions(dev, lens, slots, cuts, run)
    for s in lens:
        np.testing.assert_allclose(got[s], plain.mamba2(xs[s], w, "m.", m, eps), rtol=1e-3, atol=1e-3)
    assert all(float(st[1].abs().max()) == 0.0 for st in cache.states.values())


@pytest.mark.parametrize("n,groups,off", [(48, 1, 0), (60, 4, 3), (2048, 2, 0), (4096, 64, 8), (33, 33, 1)])
def test_the_gate_comes_before_the_norm_in_parts(dev, n, groups, off):
    import sllm_b200.ops as ops
    rng = np.random.default_rng(n)
    T, eps = 9, 1e-2
    y, z, gain = rng.standard_normal((T, n)) * 0.3, rng.standard_normal((T, n + off + 2)), rng.standard_normal(n)
    v = y * plain.silu(z[:, off:off + n])
    want = plain.unit_rms(v.reshape(T, groups, -1), eps).reshape(T, n) * gain
    got = ops.gated_group_norm(_to(dev)(y), _to(dev)(z), off, _to(dev)(gain), eps, groups, torch.float32).cpu().numpy()
    np.testing.assert_allclose(got, want, rtol=3e-5, atol=3e-5)


@pytest.mark.parametrize("W,ff,T", [(36, 20, 41), (64, 72, 9), (40, 17, 30), (128, 256, 70)])
def test_two_matrices_with_the_exact_gelu(dev, W, ff, T):
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import FEED_FORWARDS
    rng = np.random.default_rng(ff)
    w = _bf16_exact({"up": rng.standard_normal((ff, W)) * 0.3, "down": rng.standard_normal((W, ff)) * 0.3})
    h = rng.standard_normal((T, W))
    part = _bind(FEED_FORWARDS.build(PartSpec("plain_dense", {"hidden_size": W, "intermediate_size": ff, "activation": "gelu"}), dtype=torch.float32, device=dev), w)
    np.testing.assert_allclose(_term(part.forward(_to(dev)(h), None)), plain.feed_forward(h, w, "", {"kind": "dense"}), rtol=2e-4, atol=2e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("M", [1, 8, 12, 30, 40, 64, 100, 128, 200, 300])
@pytest.mark.parametrize("N,K", [(384, 256), (24, 328), (8448, 2048), (9000, 512), (30, 64), (33, 44)])
def test_gelu_that_leaves_with_the_products_tile(M, N, K):
    """The exact gelu behind every form of the bfloat16 product against float64 arithmetic on the same operands."""
    import sllm_b200.ops as ops
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    gen = torch.Generator(device="cuda:0")
    gen.manual_seed(M * 7 + N)
    x = torch.randn(M, K, device="cuda:0", generator=gen).bfloat16()
    w = (torch.randn(N, K, device="cuda:0", generator=gen) * K ** -0.5).bfloat16()
    want = torch.nn.functional.gelu(x.double() @ w.double().t())
    got = ops.linear_plain_act(x, w, torch.bfloat16, "gelu").double()
    assert float(((got - want).abs() - 2 ** -7 * want.abs()).max()) < 1e-3 and float((got - want).norm() / want.norm()) < 4e-3
    ops.check_tcgen05_status()


@pytest.mark.parametrize("E,top,ff,shared", [(6, 2, 40, 24), (4, 4, 17, 9), (8, 1, 8, 16), (3, 2, 24, None), (16, 5, 16, 40), (31, 3, 12, 20), (5, 2, 10, 14)])
def test_mixture_behind_a_biased_router_beside_a_gated_expert(dev, E, top, ff, shared):
    """The bias decides who is chosen (large enough to change many choices) and enters the weights; the shared expert, of another size, is
    weighed by a number of its own.  A token alone gets what it gets in the batch."""
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import FEED_FORWARDS
    rng = np.random.default_rng(E * ff)
    W, T = 36, 41
    mlp = _moe(E, top, ff, shared)
    w = {"router": rng.standard_normal((E, W)) * 0.3, "router.b": rng.standard_normal(E) * 2.0}
    for e in [f"e{i}" for i in range(E)] + (["shared"] if shared else []):
        f = shared if e == "shared" else ff
        w[f"{e}.gate"], w[f"{e}.up"], w[f"{e}.down"] = (rng.standard_normal(s) * 0.5 for s in ((f, W), (f, W), (W, f)))
    if shared:
        w["shared.sg"] = rng.standard_normal((1, W)) * 0.5
    w = _bf16_exact(w)
    h = rng.standard_normal((T, W))
    want = plain.experts(h, w, "", mlp)
    if top < E:
        assert np.abs(want - plain.experts(h, dict(w, **{"router.b": w["router.b"] * 0}), "", mlp)).max() > 0.1
    part = _bind(FEED_FORWARDS.build(PartSpec("gated_experts", {"hidden_size": W, "experts": E, "top": top, "expert_ff": ff, "activation": "silu", "router_bias": True,
                                                                "shared_ff": shared or 0}), dtype=torch.float32, device=dev), w)
    assert {s.name for s in part.tensor_specs()} == set(w)
    got = _term(part.forward(_to(dev)(h), None))
    np.testing.assert_allclose(got, want, rtol=3e-4, atol=3e-4)
    np.testing.assert_allclose(_term(part.forward(_to(dev)(h[7:8]), None)), got[7:8], rtol=2e-6, atol=2e-5)
    dense, idx, wts = part.route(_to(dev)(h))
    assert dense.shape[1] == E + (1 if shared else 0)
    np.testing.assert_allclose(dense[:, :E].sum(1).cpu().numpy(), 1.0, rtol=1e-5)
    if shared:
        np.testing.assert_allclose(dense[:, E].cpu().numpy(), plain.sigmoid(h @ w["shared.sg"].T)[:, 0], rtol=1e-4)


# ---- the whole model through the engine: every cutting against the plain implementation ---------------------------

@pytest.mark.parametrize("which", ["A", "odd"])
def test_sum_of_the_streams_after_every_layer(tmp_path, dev, which):
    """The streams after each layer (float32), with the term the layer hands on."""
    from sllm_b200.engine import Engine, StepEntry, build_model
    config = CONFIGS[which][0]
    d = make_model(tmp_path, config)
    cfg, w = plain.load_model(d)
    ids = _requests(config["vocab"], (19,))["r0"]
    after = []
    want = plain.forward(ids, cfg, w, after)
    model, _ = build_model(d, "float32", dev)
    seen = []
    for layer in model.layers:
        inner = layer.block.forward

        def forward(streams, *a, _inner=inner, **kw):
            out = _inner(streams, *a, **kw)
            c, x = out.connection, streams.clone()
            x = torch.einsum("tsw,sr->trw", x, c.mix) + c.share[None, :, None] * (out.term.sum(0) if out.term.dim() == 3 else out.term)[:, None]
            seen.append(x.sum(1).cpu().numpy())
            return out
        layer.block.forward = forward
    eng = Engine(model, page_size=8, num_pages=8, max_requests=1)
    got = eng.step([StepEntry("a", ids, list(range(len(ids))))]).cpu().numpy()
    np.testing.assert_allclose(got, want, rtol=3e-4, atol=3e-4)
    assert len(seen) == len(after) == len(config["layers"])
    for i, (a, b) in enumerate(zip(seen, after)):
        np.testing.assert_allclose(a, b, rtol=3e-4, atol=3e-4, err_msg=f"after layer {i}")


@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_every_cutting_against_plain(tmp_path, dev, which):
    """Whole prompts; most of a prompt and the rest token by token; portions of changing size down to two tokens; up to
    four requests at a time, portions beside single tokens.  The pools hold the trace's peak only and freed pages are
    poisoned, so pages and state slots are used again and a read of a page no longer held would show."""
    from sllm_b200.engine import Engine, build_model
    config, page = CONFIGS[which]
    reqs = _requests(config["vocab"], (70, 37, 100, 1, 45, 64, 23))
    for dtype, d, want, margins in models_for(tmp_path, config, dev, reqs):
        model, _ = build_model(d, dtype, dev)
        for mode in ("whole", "tail_decode", "portions", "mixed"):
            tr = getattr(traces, mode)(reqs)
            eng = Engine(model, page_size=page, num_pages=max(tr.max_tokens // page, 1), max_requests=4, poison_freed=True)
            out = traces.replay_engine(tr, eng)
            compare(tr, out, want, dtype, f"{which}/{dtype}/{mode}", margins)
            eng.cache.check()
            assert not eng.cache.requests and all(g.pool.used_count == 0 for g in eng.cache.groups)
            if mode == "mixed" and eng.cache.groups:
                assert eng.cache.reuse_count > 0


def test_batch_of_unequal_requests_equals_each_alone(tmp_path, dev):
    from sllm_b200.engine import Engine, StepEntry, build_model
    d = make_model(tmp_path, CONFIG_A)
    reqs = _requests(CONFIG_A["vocab"], (33, 2, 19, 50), seed=8)
    model, _ = build_model(d, "float32", dev)
    alone = {}
    for r, ids in reqs.items():
        eng = Engine(model, page_size=16, num_pages=8, max_requests=2)
        a = eng.step([StepEntry(r, ids[:-1], [len(ids) - 2])])
        b = eng.step([StepEntry(r, ids[-1:], [0])])
        alone[r] = torch.cat([a, b]).cpu().numpy()
    eng = Engine(model, page_size=16, num_pages=16, max_requests=5)
    eng.step([StepEntry("warm", [1, 2, 3], [])])            # takes slot 0 and the first page, then leaves
    eng.finish("warm")
    order = ["r3", "r1", "r0", "r2"]
    a = eng.step([StepEntry(r, reqs[r][:-1], [len(reqs[r]) - 2]) for r in order]).cpu().numpy()
    b = eng.step([StepEntry(r, reqs[r][-1:], [0]) for r in order]).cpu().numpy()
    for i, r in enumerate(order):
        np.testing.assert_allclose(np.stack([a[i], b[i]]), alone[r], rtol=3e-5, atol=3e-5)


def test_a_slot_that_is_used_again_starts_from_nothing(tmp_path, dev):
    """Four state slots, nine requests one after another and side by side: a request that gets a slot and pages another
    one left behind must not see that one's states, keys, values or last token."""
    from sllm_b200.engine import Engine, StepEntry, build_model
    d = make_model(tmp_path, ODD)
    reqs = _requests(ODD["vocab"], (12, 30, 7, 18, 3, 25, 9, 14, 2), seed=17)
    want = plain_logits(d, reqs)
    model, _ = build_model(d, "float32", dev)
    eng = Engine(model, page_size=8, num_pages=16, max_requests=4, poison_freed=True)
    names = list(reqs)
    for a in range(0, len(names), 3):
        group = names[a:a + 3]
        first = eng.step([StepEntry(r, reqs[r][:-1], [len(reqs[r]) - 2]) for r in group]).cpu().numpy()
        last = eng.step([StepEntry(r, reqs[r][-1:], [0]) for r in group]).cpu().numpy()
        for i, r in enumerate(group):
            np.testing.assert_allclose(first[i], want[r][-2], rtol=3e-4, atol=3e-4)
            np.testing.assert_allclose(last[i], want[r][-1], rtol=3e-4, atol=3e-4)
            eng.finish(r)
    assert eng.cache.reuse_count > 0


LONG_MEMORY = _config(150, 128, 3, 0.8, [           # every mixer can hold on to what lies far back
    _layer(_att(4, 2, 32, 32, 0.5, 60, 15.0, (0.3, 64)), _dense(96)),
    _layer(_ssm(4, 32, 64, 2, 4, 2), None),
    _layer(_att(4, 2, 32, 32, 0.4, 30, 18.0, None, kv_from=0), _dense(64)),
    _layer(_lat(4, 16, 16, 32, 48, 48, 0.6, 37, (10000.0, 16)), None),
], pairs=(500, 7, 11))


def _sharp(t):
    """Mixers that weigh more than the other terms, states that all but never forget: a lost key, a window that is a token off or a dropped
    state changes the logits by far more than the tolerance."""
    for n in list(t):
        if n.endswith("A_log"):
            t[n] = torch.full_like(t[n], -7.0)
        if n.endswith("mix.o"):
            t[n] *= 2.0
        if n.endswith("mlp.down"):
            t[n] *= 0.3


def test_keys_far_back_at_page_borders_window_edges_and_a_long_memory(tmp_path, dev):
    """Sharpened weights (`_sharp`): a prompt of several hundred tokens, cut at and beside page borders and the window's edge, then decoded
    token by token across more of them; every position wanted."""
    from sllm_b200.engine import Engine, build_model
    config, page = LONG_MEMORY, 16
    reqs = _requests(config["vocab"], (260,), seed=12)
    ids = reqs["r0"]
    for dtype, d, want, margins in models_for(tmp_path, config, dev, reqs, seed=11, edit=_sharp):
        cfg, w = plain.load_model(d)
        cut = plain.forward(ids[150:], cfg, w)              # the memory matters: without the first 150 tokens the end differs
        assert np.abs(cut[-1] - want["r0"][-1]).max() > 0.05
        other = json.loads(json.dumps(cfg))
        other["layers"][3]["mixer"]["mask"]["size"] += 1    # and so does the window's edge
        d1 = plain.forward(ids, other, w) - want["r0"]
        assert np.quantile(np.abs(d1[60:]).max(-1), 0.5) > 0.01
        model, _ = build_model(d, dtype, dev)
        tr = traces.Trace()
        at = 0
        for n in (15, 1, 1, 16, 3, 1, 1, 11, 1, 1, 2, 45, 1, 2, 3, 25):     # up to, onto and over page borders and the window
            tr.step([("r0", at, ids[at:at + n], range(n))])
            at += n
        while at < len(ids):
            tr.step([("r0", at, ids[at:at + 1], [0])], end=["r0"] if at == len(ids) - 1 else [])
            at += 1
        eng = Engine(model, page_size=page, num_pages=tr.max_tokens // page, max_requests=1, poison_freed=True)
        compare(tr, traces.replay_engine(tr, eng), want, dtype, f"far/{dtype}", margins)


def test_long_decoding_from_a_short_prompt(tmp_path, dev):
    """Three tokens of prompt, then 150 tokens one at a time: the states and the cache carry everything, across many
    pages; every step's logits against the plain implementation.  The first tokens of the sequence are wanted too (the
    empty states, no token before, a softmax over one key)."""
    from sllm_b200.engine import Engine, build_model
    reqs = _requests(CONFIG_A["vocab"], (153,), seed=42)
    for dtype, d, want, margins in models_for(tmp_path, CONFIG_A, dev, reqs, seed=41):
        model, _ = build_model(d, dtype, dev)
        tr = traces.tail_decode(reqs, tail=150)
        eng = Engine(model, page_size=8, num_pages=tr.max_tokens // 8, max_requests=1)
        compare(tr, traces.replay_engine(tr, eng), want, dtype, f"long/{dtype}", margins)
        if dtype == "float32":
            tr = traces.Trace()
            tr.step([("r0", 0, reqs["r0"][:1], [0])])
            tr.step([("r0", 1, reqs["r0"][1:2], [0])])
            tr.step([("r0", 2, reqs["r0"][2:5], [0, 1, 2])], end=["r0"])
            eng = Engine(model, page_size=8, num_pages=8, max_requests=1)
            compare(tr, traces.replay_engine(tr, eng), want, dtype, f"first/{dtype}", margins)


def test_greedy_generation_through_the_entry_point(tmp_path, dev):
    """`LLM.generate`: admission, the token budget, prompts in portions, decoding (from captured graphs on the GPU, whose steps
    are chained on the device: the token before is the device's own), sampling on the device; against greedy decoding with the plain
    implementation."""
    from sllm_b200.engine import build_model
    from sllm_b200.engine.llm import LLM
    from sllm_b200.sampling import SamplingParams
    d = make_model(tmp_path, CONFIG_A, seed=21)
    cfg, w = plain.load_model(d)
    prompts = list(_requests(CONFIG_A["vocab"], (9, 40, 17, 3, 26), seed=22).values())
    new = 10
    model, _ = build_model(d, "float32", dev)
    llm = LLM(model=model, block_size=16, num_pages=40, max_num_seqs=3, chunk_size=16, max_batch_tokens=48, max_model_len=128)
    res = llm.generate(prompts, SamplingParams(max_new=new))
    for pr, r in zip(prompts, res):
        ids, out = list(pr), []
        for _ in range(new):
            logits = plain.forward(ids, cfg, w)[-1]
            top = np.sort(logits)[-2:]
            out.append(int(np.argmax(logits)))
            ids.append(out[-1])
            if top[1] - top[0] < 1e-3:      # a tie the rounding may break either way: compare up to here
                break
        assert r.ids[:len(out)] == out, (len(pr), r.ids, out)
    llm.engine.cache.check()
    assert not llm.engine.cache.requests


def test_command_line_with_random_weights(tmp_path, capsys, dev, monkeypatch):
    import sllm_b200.engine.llm as llm_mod
    from sllm_b200.serving import main as cli
    recipe = "tiny-muzulorn"
    if dev == "cpu":
        import yaml
        real = llm_mod.LLM
        monkeypatch.setattr(llm_mod, "LLM", lambda model_dir, **kw: real(model_dir, **dict(kw, device="cpu")))
        with open(os.path.join(cli.RECIPES_DIR, "tiny-muzulorn.yaml")) as f:
            raw = yaml.safe_load(f)
        raw["memory"] = {"kv_device_bytes": 1 << 20}
        recipe = os.path.join(str(tmp_path), "tiny-muzulorn.yaml")
        with open(recipe, "w") as f:
            yaml.safe_dump(raw, f)
    assert cli.main([recipe]) == 0
    out = capsys.readouterr().out
    assert "Muzulorn: 4 layers" in out
    assert cli.main([recipe, "--mode", "run", "--random-weights", "4", "--prompt-ids", "5,17,3,150,42", "--max-new", "5",
                     "--dtype", "float32", "--log-level", "ERROR"]) == 0
    got = [int(t) for t in capsys.readouterr().out.strip().split(",")]
    assert len(got) == 5 and all(0 <= t < 260 for t in got)


@pytest.mark.gpu
def test_weights_drawn_on_the_device():
    """A model without a folder (`build_random_model`, what the benchmarks use), a prompt and decode steps through it."""
    from sllm_b200.engine import Engine, StepEntry, build_random_model
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    for config in (MID, ODD):
        model, _ = build_random_model(config, seed=1, dtype="bfloat16", device="cuda:0")
        eng = Engine(model, page_size=16, num_pages=16, max_requests=2)
        ids = _requests(config["vocab"], (150,))["r0"]
        out = [eng.step([StepEntry("a", ids[:140], [139])])] + [eng.step([StepEntry("a", ids[p:p + 1], [0])]) for p in range(140, 150)]
        assert all(bool(torch.isfinite(o).all()) for o in out)


@pytest.mark.gpu
def test_replay_program_on_a_model_folder(tmp_path):
    """bin/trace_run as a user runs it: the model class chosen by config.json, all four cuttings in one trace, four state slots."""
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    reqs = _requests(CONFIG_B["vocab"], (40, 75, 9, 120, 51), seed=32)
    tr = traces.all_modes(reqs)
    for dtype, d, want, margins in models_for(tmp_path, CONFIG_B, "cuda:0", reqs, seed=31):
        want = traces.tagged(want)
        out = traces.replay_subprocess(tr, d, dtype, os.path.join(str(tmp_path), f"out_{dtype}"), 16)
        compare(tr, out, want, dtype, f"replay/{dtype}", margins)
