"""Mumopel on the device against the plain implementation in ``plain_mumopel.py``: every mechanism alone, then whole
models of several shapes through the replay session (whole prompts, decoding token by token, portions down to two
tokens, mixed batches with pages used again) and greedy generation through the engine and its scheduler."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_mumopel as P
import replay_util as U

pytestmark = pytest.mark.gpu

TDT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _att(heads, kv_heads, dim, vdim, chunk=None, dims=None, scale=None, base=700.0):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5}
    if chunk:
        out["mask"] = {"size": chunk}
    if dims is None or dims > 0:
        out["rot"] = {"base": base, "dims": dim // 2 * 2 if dims is None else dims}
    return out


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, limit=1.1, shared=None, shared_limit=0.8):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def _layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _cfg(layers, width=48, vocab=101, streams=2, loop=None, cap=6.0, eps=1e-5):
    out = {"architecture": "Mumopel", "vocab": vocab, "width": width, "streams": streams, "logit_softcap": cap,
           "norm": {"eps": eps}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # dense, routed and no feed-forward; value heads shorter and longer than key heads, rotation over a part of the head,
    # chunks of several sizes and none, a loop in the middle
    "loop_inside": _cfg([_layer(_att(4, 2, 24, 40, chunk=17, dims=16), _moe(6, 2, 24, shared=40)),
                         _layer(_att(6, 2, 24, 24, chunk=32, dims=8), _dense(72)),
                         _layer(_att(2, 1, 40, 16, dims=40), _moe(5, 3, 40, shared=16)),
                         _layer(_att(3, 3, 32, 16, chunk=20), None)], loop=(1, 3, 3)),
    # the values a model may happen to make equal or one: one stream, one head everywhere, as many kv heads as heads, one
    # expert, all experts, a loop of one turn, chunks of one position, no rotation
    "equal_or_one": _cfg([_layer(_att(1, 1, 32, 32, chunk=32), _moe(1, 1, 64, shared=64, shared_limit=1.1)),
                          _layer(_att(2, 2, 32, 32, chunk=1), _dense(64)),
                          _layer(_att(1, 1, 32, 32, dims=0), _moe(3, 3, 64))], width=64, vocab=131, streams=1, loop=(0, 3, 1)),
    # sizes that no fast path takes: a width that is no multiple of 4, heads of 20 and 9, odd experts, nine streams
    "odd_sizes": _cfg([_layer(_att(3, 1, 20, 12, chunk=13, dims=10), _moe(7, 3, 18, shared=9)),
                       _layer(_att(2, 2, 9, 13, chunk=25, dims=6), _dense(50)),
                       _layer(_att(5, 1, 20, 20, dims=2), _moe(4, 1, 10, shared=21))], width=38, vocab=50, streams=9, loop=(2, 3, 2)),
    # everything loops, five streams, no shared expert, no cap
    "all_loops": _cfg([_layer(_att(4, 1, 48, 16, chunk=24, dims=32), _dense(40)),
                       _layer(_att(2, 2, 16, 80, chunk=48, dims=4), _moe(4, 2, 16))], width=40, streams=5, loop=(0, 2, 2), cap=None),
    # layers of a mixer only, and no loop
    "mixers_only": _cfg([_layer(_att(4, 2, 16, 16, chunk=40)), _layer(_att(5, 1, 16, 32, dims=8)),
                         _layer(_att(2, 2, 48, 48, chunk=16), _dense(30))], width=56, streams=3),
    # sizes that every fast path takes in bfloat16: heads of 64 and 128 (tcgen05 attention), widths and experts in steps of 16
    "fast_paths": _cfg([_layer(_att(4, 2, 64, 64, chunk=48, dims=32), _dense(128)),
                        _layer(_att(8, 2, 64, 64, dims=64), _moe(4, 2, 64, shared=32)),
                        _layer(_att(8, 4, 128, 128, chunk=64, dims=32), _moe(6, 2, 32)),
                        _layer(_att(2, 1, 128, 64, chunk=80, dims=128), _dense(96))], width=64, vocab=97, streams=4, loop=(1, 3, 2)),
}


def _decide_by_the_bias(w, cfg):
    """The choice of experts is made one that rounding cannot turn: the routers' biases are far apart and their matrices
    small.  The weights still depend on the token."""
    for i, L in enumerate(cfg["layers"]):
        if L.get("mlp") is not None and L["mlp"]["kind"] == "moe":
            w[f"l{i}.mlp.router"] *= 0.25
            b = w[f"l{i}.mlp.router.b"]
            E = b.numel()
            step = 3 if E % 3 else 5
            b[:] = torch.tensor([1.5 * ((e * step + i) % E) for e in range(E)], dtype=b.dtype)


def _model_dir(tmp_path, name, cfg, seed=1, static_choice=False, edit=None):
    w = P.random_weights(cfg, seed)
    if static_choice:
        _decide_by_the_bias(w, cfg)
    if edit is not None:
        edit(w)
    w = {k: v.to(torch.bfloat16).double() for k, v in w.items()}              # what the file will hold
    U.write_model_dir(str(tmp_path / name), cfg, {k: v.float() for k, v in w.items()}, torch.bfloat16)
    return str(tmp_path / name), w


def _session(model_dir, dtype, max_tokens, block=16, max_requests=4):
    from firefly_b200.replay import ReplaySession
    return ReplaySession(model_dir, dtype=dtype, max_tokens=max_tokens, block_size=block, max_requests=max_requests)


def _check(got, plain, dtype, what):
    """32-bit: every row within the tolerance.  bfloat16: most rows within it and every row near it."""
    if dtype == "float32":
        U.compare(got, plain, U.TOL[dtype], what)
        return
    errs = sorted(U.rel_err(row, plain[rid.split("#")[0]][pos]) for (rid, pos), row in got.rows.items())
    assert errs and all(e == e for e in errs), what
    tol = U.TOL[dtype]
    assert errs[-1] <= 2 * tol and errs[int(0.9 * (len(errs) - 1))] <= tol, \
        f"{what}: worst {errs[-1]:.3e}, 90% {errs[int(0.9 * (len(errs) - 1))]:.3e}, tol {tol:g}"


# ------------------------------------------------------------------ whole models, every cutting --
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_replay_in_every_cutting_matches_the_plain_model(tmp_path, name, dtype):
    cfg = CONFIGS[name]
    model_dir, w = _model_dir(tmp_path, name, cfg, static_choice=dtype == "bfloat16")
    reqs = U.make_requests(cfg["vocab"], [70, 3, 45, 1, 33, 58], 5)
    plain = {rid: P.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}
    twice = dict(reqs, **{"r0#2": reqs["r0"], "r4#2": reqs["r4"]})       # a request once more, on pages used before
    for label, steps in (("whole", U.trace_whole(reqs)), ("decode", U.trace_tail_decode(reqs, tail=40)),
                         ("portions", U.trace_portions(reqs, sizes=(17, 5, 2, 9, 2, 31, 3, 2))),
                         ("mixed", U.trace_mixed(twice, seed=3, max_live=4, sizes=(13, 2, 7, 21, 3, 2, 16)))):
        sess = _session(model_dir, dtype, U.peak_tokens(steps), block=16 if label != "portions" else 8)
        _check(U.run_trace(sess, steps), plain, dtype, f"{name}/{dtype}/{label}")
        sess.cache.check()
        assert not sess.cache.live


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_requests_at_middling_sizes(tmp_path, dtype):
    """Requests of hundreds of tokens over many chunks, whole, with a decoded tail, and mixed on reused pages."""
    cfg = _cfg([_layer(_att(6, 2, 80, 80, chunk=200, dims=48), _moe(6, 2, 48, shared=80)),
                _layer(_att(4, 2, 64, 64, chunk=128, dims=64), _dense(128)),
                _layer(_att(8, 1, 64, 64, dims=16), _moe(4, 1, 96, shared=64)),
                _layer(_att(2, 1, 40, 112, chunk=70, dims=32), None)], width=96, vocab=211, streams=3, loop=(0, 2, 2))
    model_dir, w = _model_dir(tmp_path, "middling", cfg, seed=3, static_choice=dtype == "bfloat16")
    reqs = U.make_requests(cfg["vocab"], [600, 260, 90], 9)
    plain = {rid: P.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}
    twice = dict(reqs, **{"r1#2": reqs["r1"]})
    for label, steps in (("whole", U.trace_whole(reqs)), ("decode", U.trace_tail_decode(reqs, tail=48)),
                         ("mixed", U.trace_mixed(twice, seed=5, max_live=3, sizes=(64, 2, 129, 31, 3, 200)))):
        sess = _session(model_dir, dtype, U.peak_tokens(steps))
        _check(U.run_trace(sess, steps), plain, dtype, f"middling/{dtype}/{label}")
        sess.cache.check()
        assert not sess.cache.live


@pytest.mark.parametrize("name", ["loop_inside", "mixers_only", "odd_sizes"])
def test_the_streams_sum_matches_after_every_layer_run(tmp_path, name):
    from firefly_b200.parts.streams import stream_sum
    cfg = CONFIGS[name]
    model_dir, w = _model_dir(tmp_path, "stream", cfg)
    toks = U.make_requests(cfg["vocab"], [45], 8)["r0"]
    want, got, steps = [], [], []
    P.forward(cfg, w, toks, sums=want)
    sess = _session(model_dir, "float32", 64)
    build = sess.runner.build_context
    sess.runner.build_context = lambda *a, **k: steps.append(build(*a, **k)) or steps[-1]
    sess.model.after_run = lambda i, res, pending: got.append(stream_sum(res, pending, steps[-1], cfg["streams"]).cpu().double().clone())
    sess.run_step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": [0]}], "end": ["a"]})
    assert len(got) == len(want) == len(P.layer_order(cfg))
    for i, g in enumerate(got):
        assert float((g - want[i]).abs().max()) < 2e-5 * float(want[i].abs().max()), f"after layer run {i}"


def test_a_looped_layer_has_a_cache_for_every_turn(tmp_path):
    """With the first turn's queries and the second's told apart by the streams, one cache for both turns would show: the
    plain model with its turns' keys swapped gives other logits."""
    cfg = CONFIGS["all_loops"]
    model_dir, w = _model_dir(tmp_path, "turns", cfg)
    sess = _session(model_dir, "float32", 64)
    assert len(sess.model.cache_slot_specs()) == 4
    once = dict(cfg, loop={"start": 0, "stop": 2, "times": 1})
    toks = U.make_requests(cfg["vocab"], [30], 8)["r0"]
    two, one = P.forward(cfg, w, toks), P.forward(once, w, toks)
    assert float((two - one).abs().max()) > 0.1 * float(two.abs().max())


# ------------------------------------------------------------------ mechanisms alone --
def _one_layer(tmp_path, layer, width=48, dtype="float32", seed=2, max_tokens=1024, block=16, edit=None):
    cfg = _cfg([layer], width=width)
    model_dir, w = _model_dir(tmp_path, "one", cfg, seed, edit=edit)
    return cfg, w, _session(model_dir, dtype, max_tokens, block=block)


def _step_context(sess, seqs):
    """A StepContext for sequences given as (request id, new tokens): admits, grows, builds."""
    from firefly_b200.engine.runner import StepEntry
    entries = []
    for rid, n in seqs:
        rc = sess.live.get(rid) or sess.cache.admit(rid)
        sess.live[rid] = rc
        assert sess.cache.grow(rc, rc.num_tokens + n)
        entries.append(StepEntry(rc, [0] * n, []))
    return sess.runner.build_context(entries), entries


def _run_cut(sess, call, x, cuts, rid):
    """``call(rows, ctx)`` on the portions of x one after the other, as one request; its pages then go to the next cutting."""
    rows, p = [], 0
    for n in cuts:
        ctx, entries = _step_context(sess, [(rid, n)])
        rows.append(call(x[p:p + n].cuda().contiguous(), ctx).float().cpu())
        for e in entries:
            sess.cache.advance(e.cache, len(e.tokens))
        p += n
    sess.runner.check_status()
    sess.cache.free(sess.live.pop(rid))
    return torch.cat(rows).double()


def _mixer(sess):
    m = sess.model.blocks[0].mixer
    return lambda rows, ctx: m.forward(rows, ctx, 0, True)


CUTS = ([57], [20, 2, 1, 1, 30, 3], [1] * 57, [2] * 28 + [1])
ATT_SHAPES = [(4, 2, 24, 40, 16, 16), (2, 2, 16, 16, 7, 16), (3, 1, 20, 12, 30, 10), (4, 2, 64, 64, 32, 32), (2, 1, 128, 128, None, 128),
              (34, 2, 16, 16, 20, 2), (2, 1, 192, 96, 11, 96), (1, 1, 100, 256, 57, 48), (6, 6, 32, 32, 1, 0), (16, 1, 64, 32, 29, 64),
              (5, 1, 96, 96, 12, 40), (9, 3, 9, 9, 13, 4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", ATT_SHAPES)
def test_attention_alone(tmp_path, dtype, shape):
    """The norms over all heads, the rotation of neighbouring pairs, the chunks and the sinks together."""
    heads, kv, dim, vdim, chunk, dims = shape
    m = _att(heads, kv, dim, vdim, chunk=chunk, dims=dims, scale=dim ** -0.5 * 1.2)
    cfg, w, sess = _one_layer(tmp_path, _layer(m), dtype=dtype)
    eps = cfg["norm"]["eps"]
    x = torch.randn(57, 48, generator=torch.Generator().manual_seed(0)).to(TDT[dtype])
    want = P.attention(x.double(), w, "l0.mix", m, eps)
    # the test can tell: without the sinks, with chunks one longer, without the rotation
    others = [(w["l0.mix.sink"] - 30.0, m)]
    if chunk and chunk < 50:
        others.append((w["l0.mix.sink"], dict(m, mask={"size": chunk + 1})))
    if dims and chunk != 1:
        others.append((w["l0.mix.sink"], dict(m, rot=None)))
    for sink, other in others:
        far = P.attention(x.double(), dict(w, **{"l0.mix.sink": sink}), "l0.mix", other, eps)
        assert float((far - want).abs().max()) > 0.02 * float(want.abs().max())
    tol = 3e-5 if dtype == "float32" else 3e-2
    for cuts in CUTS:
        got = _run_cut(sess, _mixer(sess), x, cuts, f"r{len(cuts)}")
        assert float((got - want).abs().max()) <= tol * float(want.abs().max()), cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", [16, 48, 64, 96, 128, 256])
@pytest.mark.parametrize("chunk", [None, 300, 64, 50])
def test_a_sink_s_score_is_taken_in_once_however_the_keys_are_split(dtype, d, chunk):
    """The attention kernels alone, every head with a sink of its own (far below, among and far above the scores): one token
    a sequence with its keys in one range, in many ranges and in ranges shared out by length, and portions with their keys
    walked by one block or shared out over several; a step of both."""
    from firefly_b200.ops import kernels as K
    H, G, block = 6, 2, 16
    lens = [1, 5, 64, 65, 400, 1300]
    gen = torch.Generator().manual_seed(d)
    dev, dt = "cuda", TDT[dtype]
    sink = torch.tensor([-20.0, 0.0, 3.0, 9.0, -1.5, 40.0], dtype=torch.float64)
    sink_d = sink.float().cuda()
    per = -(-max(lens) // block)
    pages = torch.zeros(len(lens) * per + 1, 2, G, block, d, dtype=dt, device=dev)
    table = (torch.arange(len(lens) * per, dtype=torch.int32).view(len(lens), per) + 1).flip(0).contiguous()
    data, wants = [], []
    scale = 1.5 * d ** -0.5
    for s, n in enumerate(lens):
        q, k, v = (torch.randn(n, heads, d, generator=gen).to(dt) for heads in (H, G, G))
        for j in range(n):
            pages[table[s, j // block], 0, :, j % block] = k[j].to(dev)
            pages[table[s, j // block], 1, :, j % block] = v[j].to(dev)
        data.append(q)
        wants.append(P.sink_softmax_attention(q.double(), k.double(), v.double(), scale, P.chunk_mask(n, chunk), sink))
    table = table.to(dev)
    tol = 2e-5 if dtype == "float32" else 2e-2

    class Scratch:
        def get(self, tag, shape, dtype):
            return torch.empty(shape, dtype=dtype, device=dev)

    def run(q_lens, by_length=False):
        ctx_lens = [n - ql for n, ql in zip(lens, q_lens)]
        q = torch.cat([data[s][n - ql:] for s, (n, ql) in enumerate(zip(lens, q_lens))]).reshape(-1, H * d).to(dev).contiguous()
        T = q.shape[0]
        cu = torch.tensor([0] + list(np.cumsum(q_lens)), dtype=torch.int32, device=dev)
        ctx = SimpleNamespace(
            cu_q=cu, ctx_lens=torch.tensor(ctx_lens, dtype=torch.int32, device=dev), num_seqs=len(lens), q_lens=q_lens,
            token_seq=torch.repeat_interleave(torch.arange(len(lens), dtype=torch.int32), torch.tensor(q_lens)).to(torch.int32).to(dev),
            positions=torch.cat([torch.arange(c, c + ql) for c, ql in zip(ctx_lens, q_lens)]).to(torch.int32).to(dev),
            ctx_lens_host=ctx_lens, num_decode_seqs=next((i for i, ql in enumerate(q_lens) if ql > 1), len(lens)),
            max_kv_len=max(lens), ranges_by_length=by_length, workspace=Scratch(), captured=False, memo={},
            key_share_level=0, status=torch.zeros(1, dtype=torch.int32, device=dev))
        out = torch.empty(T, H * d, dtype=dt, device=dev)
        torch.cuda.synchronize()
        K.paged_attention(q, H * d, pages, table, ctx, out, H, G, d, scale, -chunk if chunk else 0, sink=sink_d)
        assert int(ctx.status[0]) == 0
        want = torch.cat([wants[s][n - ql:] for s, (n, ql) in enumerate(zip(lens, q_lens))]).reshape(T, H * d)
        err = (out.double().cpu() - want).abs().view(T, H, d).amax(dim=(0, 2))
        big = want.abs().view(T, H, d).amax(dim=(0, 2))                        # head by head: a high sink makes small rows
        assert bool((err <= tol * torch.clamp(big, min=1e-12) + 1e-30).all()), (q_lens, by_length, err / big)
    run([1] * 6)
    run([1] * 6, by_length=True)
    run(lens)
    run([1, 1, 1, 3, 70, 2])                                                   # a short portion behind many keys: shares
    run([1, 1, 1, 1, 1, 9])


# ------------------------------------------------------------------ far keys and chunk borders --
def _queries_against_keys(w, m):
    """Every query head becomes minus the key head it reads, on the elements that do not turn (those that turn are made
    small), with plain norms.  A row that is minus an earlier row then has a query along that row's key and against its
    own: that one score stands far above the others, and an attention that loses that key gives another result."""
    p, d, rep, dims = "l0.mix", m["dim"], m["heads"] // m["kv_heads"], m["rot"]["dims"] if m.get("rot") else 0
    for h in range(m["heads"]):
        kh = h // rep
        w[p + ".q"][h * d:(h + 1) * d] = -w[p + ".k"][kh * d:(kh + 1) * d]
        if dims:
            w[p + ".q"][h * d:h * d + dims] *= 0.02
    w[p + ".q.norm"][:] = 1.0
    w[p + ".k.norm"][:] = 1.0


def _far_case(tmp_path, m, far, query, dtype, seen):
    cfg, w, sess = _one_layer(tmp_path, _layer(m), dtype=dtype, edit=lambda w: _queries_against_keys(w, m))
    x = torch.randn(query + 1, 48, generator=torch.Generator().manual_seed(far))
    x[query] = -x[far]
    x = x.to(TDT[dtype])
    eps = cfg["norm"]["eps"]
    want = P.attention(x.double(), w, "l0.mix", m, eps)
    y = x.double().clone()
    y[far] = 0.0
    without = P.attention(y, w, "l0.mix", m, eps)
    moved = float((without[-1] - want[-1]).abs().max()) / float(want[-1].abs().max())
    if seen:
        assert moved > 0.2                                                     # the test can tell
    else:
        assert moved == 0.0                                                    # the key is not read,
        open_m = dict(m, mask=None)
        assert float((P.attention(x.double(), w, "l0.mix", open_m, eps)[-1] - want[-1]).abs().max()) > 0.2 * float(want[-1].abs().max())
    T = query + 1
    tol = 3e-5 if dtype == "float32" else 4e-2
    for cuts in ([T], [T - 1, 1], [far + 1, T - far - 1], [max(1, T - 9)] + [1] * min(9, T - 1), [T - 2, 2]):
        got = _run_cut(sess, _mixer(sess), x, [c for c in cuts if c], f"r{len(cuts)}")
        assert float((got - want).abs().max()) <= tol * float(want.abs().max()), cuts
        assert float((got[-1] - want[-1]).abs().max()) <= tol * float(want[-1].abs().max()), cuts


SIZES = [(4, 2, 24, 16, 8), (4, 2, 64, 48, 16), (2, 2, 128, 128, 32), (6, 1, 96, 96, 32)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("chunk,far,query", [(None, 0, 700), (None, 15, 700), (None, 255, 700), (512, 512, 700), (512, 515, 1000), (701, 16, 700),
                                             (64, 64, 127), (96, 192, 287), (300, 1, 299), (48, 3, 40), (33, 33, 34)])
def test_a_key_far_back_is_found(tmp_path, dtype, sizes, chunk, far, query):
    """A key that stands out among hundreds, at and off page borders, the first of a sequence or of its chunk, with the query
    at its chunk's end; the query inside a prompt, at the start of a portion, and decoded."""
    heads, kv, dim, vdim, dims = sizes
    _far_case(tmp_path, _att(heads, kv, dim, vdim, chunk=chunk, dims=dims, scale=14.0 / dim), far, query, dtype, True)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("chunk,far,query", [(512, 511, 700), (64, 63, 64), (64, 63, 127), (96, 191, 287), (100, 99, 100), (16, 15, 17), (33, 32, 40)])
def test_a_key_of_the_chunk_in_front_is_not_read(tmp_path, dtype, sizes, chunk, far, query):
    heads, kv, dim, vdim, dims = sizes
    _far_case(tmp_path, _att(heads, kv, dim, vdim, chunk=chunk, dims=dims, scale=14.0 / dim), far, query, dtype, False)


def test_the_first_tokens_see_themselves_and_the_sink(tmp_path):
    """Position 0, and the first position of every chunk: one key and the sink share the softmax."""
    m = _att(2, 1, 16, 16, chunk=5)
    cfg, w, sess = _one_layer(tmp_path, _layer(m))
    x = torch.randn(21, 48, generator=torch.Generator().manual_seed(9))
    want = P.attention(x.double(), w, "l0.mix", m, cfg["norm"]["eps"])
    for cuts in ([21], [1] * 21, [5, 5, 5, 6], [4, 2, 15]):
        got = _run_cut(sess, _mixer(sess), x, cuts, f"r{len(cuts)}")
        for t in (0, 5, 10, 15, 20):
            assert float((got[t] - want[t]).abs().max()) <= 3e-5 * float(want[t].abs().max()), (cuts, t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,true,dims", [(24, 24, 0), (24, 16, 16), (64, 64, 32), (96, 40, 32), (128, 128, 128), (256, 256, 64), (20, 20, 10), (9, 9, 4)])
def test_one_norm_over_all_heads(dtype, d, true, dims):
    """Rows whose heads differ in size by far, so that a norm a head would show; heads filled up with zeros; queries only."""
    from firefly_b200.ops import kernels as K
    nq, nkv, T, block = 5, 2, 11, 8
    g = torch.Generator().manual_seed(d)
    dt = TDT[dtype]
    freq = torch.rand(dims // 2, generator=g, dtype=torch.float64) if dims else None
    positions = torch.tensor([0, 1, 5, 6, 7, 40, 41, 1000, 1001, 77, 30], dtype=torch.int32)
    table = torch.randperm(200, generator=g).to(torch.int32).view(1, 200).cuda() + 1
    ctx = SimpleNamespace(positions=positions.cuda(), token_seq=torch.zeros(T, dtype=torch.int32, device="cuda"),
                          status=torch.zeros(1, dtype=torch.int32, device="cuda"))
    freq_d = freq.cuda() if dims else None
    v = torch.randn(T, nq + 2 * nkv, d, generator=g) * torch.logspace(-1, 1, nq + 2 * nkv)[None, :, None]
    v[..., true:] = 0.0
    v = v.to(dt).double()
    qw, kw = (torch.randn(n, d, generator=g) for n in (nq, nkv))

    def finish(z, wt):
        n = z.shape[1]
        rms = torch.sqrt((z * z).sum(dim=(1, 2), keepdim=True) / (n * true) + 1e-5)
        z = z / rms * wt.double()[None]
        if not dims:
            return z
        ang = positions.double()[:, None] * freq[None, :]
        c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
        out = z.clone()
        out[..., 0:dims:2] = z[..., 0:dims:2] * c - z[..., 1:dims:2] * s
        out[..., 1:dims:2] = z[..., 1:dims:2] * c + z[..., 0:dims:2] * s
        return out
    q, k = finish(v[:, :nq], qw), finish(v[:, nq:nq + nkv], kw)
    qwd, kwd = qw.reshape(-1).cuda(), kw.reshape(-1).cuda()
    tol = 3e-6 if dtype == "float32" else 5e-3
    torch.cuda.synchronize()
    for keys in (nkv, 0):
        got = v[:, :nq + 2 * keys].reshape(T, -1).to(dt).cuda().contiguous()
        pages = torch.zeros(202, 2, nkv, block, d, dtype=dt, device="cuda")
        torch.cuda.synchronize()
        K.head_finish(got, nq, keys, d, true, 1e-5, freq_d, 1.0, ctx, table if keys else None, pages if keys else None, interleaved=True,
                      q_norm_w=qwd, k_norm_w=kwd if keys else None, norm_all=True)
        assert int(ctx.status[0]) == 0
        back = got.cpu().double()[:, :nq * d].view(T, nq, d)
        assert float((back - q).abs().max()) <= tol * float(q.abs().max())
        if keys:
            pg = pages.cpu().double()
            for t in range(T):
                pos = int(positions[t])
                page = int(table[0, pos // block])
                assert float((pg[page, 0, :, pos % block] - k[t]).abs().max()) <= tol * float(k.abs().max())
                assert torch.equal(pg[page, 1, :, pos % block], v[t, nq + nkv:])
            assert int((pg.abs().sum(dim=(1, 2, 4)) > 0).sum()) == T          # and nothing else was written


# ------------------------------------------------------------------ streams --
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 8, 9, 32])
@pytest.mark.parametrize("T,W", [(1, 48), (5, 352), (3, 1024), (2, 2052), (1, 16388), (4, 37)])
def test_the_seam_between_two_parts(dtype, S, T, W):
    """The write with a tensor or with routed rows, in place and from equal streams, the read, the norm of both kinds, the
    sum of the streams for chosen rows."""
    from firefly_b200.ops import kernels as K
    g = torch.Generator().manual_seed(W + S)
    dt = TDT[dtype]
    X = torch.randn(T, S, W, generator=g) * torch.linspace(0.5, 3.0, S)[None, :, None]
    x0 = torch.randn(T, W, generator=g)
    mix, ow, iw = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    wn, bn = torch.randn(W, generator=g), torch.randn(W, generator=g)
    y = torch.randn(T, W, generator=g).to(dt)
    top = 3
    rows, wts, shared = torch.randn(T * top, W, generator=g), torch.rand(T, top, generator=g), torch.randn(T, W, generator=g)
    row_of = torch.randperm(T * top, generator=g).to(torch.int32)
    dev = {n: t.cuda() for n, t in dict(X=X, x0=x0, mix=mix, ow=ow, iw=iw, wn=wn, bn=bn, y=y, rows=rows, wts=wts, shared=shared, row_of=row_of).items()}
    torch.cuda.synchronize()              # weights are read before the kernel waits for what is in front of it in the stream
    routed = (wts.double()[:, :, None] * rows.double()[row_of.long().view(T, top)]).sum(dim=1)
    tol = 4e-6 if dtype == "float32" else 5e-3

    def norm(u, center):
        if center:
            return P.layer_norm(u, wn.double(), bn.double(), 1e-5)
        return P.rms_norm(u, wn.double(), 1e-5) + bn.double()
    for what, kw, yy in (("none", {}, None), ("tensor", dict(y=dev["y"]), y.double()),
                         ("routed", dict(routed=(dev["rows"], dev["row_of"], dev["wts"], None)), routed),
                         ("shared", dict(routed=(dev["rows"], dev["row_of"], dev["wts"], dev["shared"])), routed + shared.double())):
        for same in (False, True):
            old = (x0[:, None, :].expand(T, S, W) if same else X).double().permute(1, 0, 2)
            new = old if yy is None else P.streams_write(old, mix.double(), ow.double(), yy)
            src = dev["x0"] if same else dev["X"].clone()
            weights = {} if yy is None else dict(mix=dev["mix"], out_w=dev["ow"])
            dst = None if yy is None else (torch.empty(T, S, W, device="cuda") if same else src)
            center = what != "tensor"
            out = torch.empty(T, W, dtype=dt, device="cuda")
            K.stream_seam(src, out, streams=S, in_w=dev["iw"], w=dev["wn"], b=dev["bn"], eps=1e-5, center=center, dst=dst, **weights, **kw)
            want = norm(P.streams_read(new, iw.double()), center)
            assert float((out.cpu().double() - want).abs().max()) <= tol * float(want.abs().max()), (what, same)
            if dst is not None:
                got = dst.cpu().double().permute(1, 0, 2)
                assert float((got - new).abs().max()) <= 4e-6 * float(new.abs().max()), (what, same)
            # the model's end: nothing kept, the plain sum, chosen rows, and the sum itself
            src = dev["x0"] if same else dev["X"]
            pick = torch.tensor([T - 1, 0], dtype=torch.int32, device="cuda")
            out = torch.empty(2, W, dtype=dt, device="cuda")
            K.stream_seam(src, out, streams=S, w=dev["wn"], b=dev["bn"], eps=1e-5, row_idx=pick, **weights, **kw)
            want = norm(new.sum(dim=0), True)[[T - 1, 0]]
            assert float((out.cpu().double() - want).abs().max()) <= tol * float(want.abs().max()), (what, same)
            total = torch.empty(T, W, device="cuda")
            K.stream_seam(src, total, streams=S, **weights, **kw)
            assert float((total.cpu().double() - new.sum(dim=0)).abs().max()) <= 4e-6 * float(new.abs().sum(dim=0).max()), (what, same)
            assert torch.equal(dev["X"].cpu(), X) and torch.equal(dev["x0"].cpu(), x0)


def test_the_mix_is_read_from_and_to(tmp_path):
    """A mix that only feeds the second stream from the first, and parts that write into one stream only: the transposed
    matrix gives another model."""
    cfg = _cfg([_layer(_att(2, 1, 16, 16, chunk=12), _dense(24)), _layer(_att(2, 2, 16, 16), _moe(3, 1, 16))], streams=3)

    def edit(w):
        for k in [k for k in w if k.endswith(".mix") and ".hc" in k]:
            w[k][:] = torch.tensor([[1.0, 1.0, 0.0], [0.0, 0.5, 2.0], [0.0, 0.0, 1.0]])
            w[k[:-3] + "out"][:] = torch.tensor([1.0, 0.0, 0.0])
    model_dir, w = _model_dir(tmp_path, "mix", cfg, edit=edit)
    toks = U.make_requests(cfg["vocab"], [30], 2)["r0"]
    want = P.forward(cfg, w, toks)
    turned = P.forward(cfg, {k: (v.T if k.endswith(".mix") and ".hc" in k else v) for k, v in w.items()}, toks)
    assert float((turned - want).abs().max()) > 0.1 * float(want.abs().max())
    sess = _session(model_dir, "float32", 64)
    U.compare(U.run_trace(sess, U.trace_whole({"r0": toks})), {"r0": want.numpy()}, U.TOL["float32"], "mix")


# ------------------------------------------------------------------ feed-forward, router, logits --
@pytest.mark.parametrize("E,top,groups,keep", [(14, 3, 1, 1), (1, 1, 1, 1), (7, 7, 1, 1), (40, 5, 1, 1), (16, 4, 4, 2), (130, 8, 1, 1)])
def test_the_softmax_over_the_chosen_logits(E, top, groups, keep):
    from firefly_b200.ops import kernels as K
    T = 33
    g = torch.Generator().manual_seed(E)
    z, b = torch.randn(T, E, generator=g) * 4, torch.randn(E, generator=g) * 3
    z[5] += 400.0                                                              # a softmax over all of these would not do
    z[6] -= 400.0
    zd, bd = z.cuda(), b.cuda()
    ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    torch.cuda.synchronize()
    for bias in (None, bd):
        K.moe_route(zd, ids, wts, groups, keep, score=K.ROUTE_CHOSEN_SOFTMAX, renormalize=False, bias=bias)
        full = z.double() + (b.double() if bias is not None else 0.0)
        if groups > 1:
            per = full.view(T, groups, E // groups)
            shut = torch.ones(T, groups, dtype=torch.bool).scatter(1, per.max(dim=2).values.topk(keep, dim=1).indices, False)
            pickable = per.masked_fill(shut[:, :, None], -float("inf")).view(T, E)
        else:
            pickable = full
        best = pickable.topk(top, dim=1)
        assert torch.equal(ids.cpu().long().sort(dim=1).values, best.indices.sort(dim=1).values)
        want = torch.zeros(T, E, dtype=torch.float64).scatter(1, best.indices, torch.softmax(best.values, dim=1))
        got = torch.zeros(T, E, dtype=torch.float64).scatter(1, ids.cpu().long(), wts.cpu().double())
        assert float((got - want).abs().max()) < 3e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens", [1, 5, 65, 300])
@pytest.mark.parametrize("shape", [(6, 2, 24, 40), (5, 1, 40, 16), (1, 1, 16, 16), (9, 9, 8, None), (4, 3, 18, 9), (8, 1, 136, None)])
def test_routed_experts_alone(tmp_path, dtype, tokens, shape):
    """As rows handed on, as a delta and added into a stream; both limits bite; the bias turns choices and weights."""
    from firefly_b200.parts.moe import RoutedRows
    E, top, ff, shared = shape
    mlp = _moe(E, top, ff, limit=0.7, shared=shared, shared_limit=0.45)
    cfg, w, sess = _one_layer(tmp_path, _layer(_att(1, 1, 8, 8), mlp), dtype=dtype)
    x = (torch.randn(tokens, 48, generator=torch.Generator().manual_seed(tokens)) * 1.5).to(TDT[dtype])
    want = P.moe_ff(x.double(), w, "l0.mlp", mlp)
    if tokens >= 65:
        others = [(w, dict(mlp, expert=dict(mlp["expert"], limit=0.9)))]
        if shared:
            others.append((w, dict(mlp, shared=dict(mlp["shared"], limit=0.7))))
        if top < E:
            others.append((dict(w, **{"l0.mlp.router.b": w["l0.mlp.router.b"] * 0}), mlp))
        for ww, other in others:
            assert float((P.moe_ff(x.double(), ww, "l0.mlp", other) - want).abs().max()) > 0.03 * float(want.abs().max())
    ctx, _ = _step_context(sess, [("a", tokens)])
    part = sess.model.blocks[0].feed_forward
    got = part.forward(x.cuda(), ctx).double().cpu()
    res = torch.full((tokens, 48), 0.5, device="cuda")
    assert part.forward(x.cuda(), ctx, accumulate_into=res, residual_scale=0.25) is None
    handed = part.forward(x.cuda(), ctx, as_rows=True)
    assert isinstance(handed, RoutedRows)
    row_of = handed.row_of.cpu().long()[:tokens * top].view(tokens, top)
    summed = (handed.wts.cpu().double()[:, :, None] * handed.rows.cpu().double()[row_of]).sum(dim=1)
    if handed.shared is not None:
        summed = summed + handed.shared.cpu().double()
    # a token whose choice is a matter of rounding may go either way in bfloat16
    z = x.double() @ w["l0.mlp.router"].T + w["l0.mlp.router.b"]
    clear = torch.ones(tokens, dtype=torch.bool)
    if top < E and dtype == "bfloat16":
        srt = z.sort(dim=1, descending=True).values
        clear = srt[:, top - 1] - srt[:, top] > 1e-3
    assert int(clear.sum()) >= 0.9 * tokens
    tol = 3e-5 if dtype == "float32" else 2e-2
    for a in (got, summed):
        assert float((a - want)[clear].abs().max()) <= tol * float(want.abs().max())
    assert float((res.double().cpu() - 0.5 - 0.25 * want)[clear].abs().max()) <= tol * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens", [1, 2, 64, 65, 150])
@pytest.mark.parametrize("width,ff", [(48, 72), (38, 21), (128, 320)])
def test_the_dense_feed_forward_alone(tmp_path, dtype, tokens, width, ff):
    cfg, w, sess = _one_layer(tmp_path, _layer(_att(1, 1, 8, 8), _dense(ff)), width=width, dtype=dtype)
    x = torch.randn(tokens, width, generator=torch.Generator().manual_seed(tokens)).to(TDT[dtype])
    want = P.dense_ff(x.double(), w, "l0.mlp")
    ctx, _ = _step_context(sess, [("a", tokens)])
    got = sess.model.blocks[0].feed_forward.forward(x.cuda(), ctx).double().cpu()
    assert float((got - want).abs().max()) <= (3e-5 if dtype == "float32" else 2e-2) * float(want.abs().max())


def test_the_cap_on_the_logits():
    from firefly_b200.ops import kernels as K
    x = torch.cat([torch.linspace(-80, 80, 4001), torch.tensor([0.0, 1e-6, -1e4, 1e4])])
    for cap in (0.5, 15.0, 40.0):
        y = x.cuda()
        K.softcap_(y, cap)
        want = cap * torch.tanh(x.double() / cap)
        assert float((y.cpu().double() - want).abs().max()) <= 2e-6 * cap


# ------------------------------------------------------------------ long decoding, batches, generation --
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(tmp_path, dtype):
    cfg = CONFIGS["loop_inside"]
    model_dir, w = _model_dir(tmp_path, "long", cfg, seed=4, static_choice=dtype == "bfloat16")
    toks = U.make_requests(cfg["vocab"], [300], 3)["r0"]
    plain = {"r0": P.forward(cfg, w, toks).numpy()}
    sess = _session(model_dir, dtype, 320)
    _check(U.run_trace(sess, U.trace_tail_decode({"r0": toks}, tail=290)), plain, dtype, f"long decoding {dtype}")
    sess.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_of_unequal_requests_gives_each_its_own_logits(tmp_path, dtype):
    """All requests in one step, then a decoded token of each beside a portion of another, against each alone."""
    cfg = CONFIGS["fast_paths"]
    model_dir, w = _model_dir(tmp_path, "batch", cfg, seed=8, static_choice=True)
    reqs = U.make_requests(cfg["vocab"], [130, 2, 40, 71], 4)
    alone = U.run_trace(_session(model_dir, dtype, 256), U.trace_whole(reqs)).rows
    heads = {"r0": 100, "r1": 1, "r2": 39, "r3": 70}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": reqs[r][:n], "want": list(range(n))} for r, n in heads.items()], "end": []},
             {"step": 1, "entries": [{"id": r, "tokens": reqs[r][n:], "want": list(range(len(reqs[r]) - n))} for r, n in heads.items()],
              "end": list(reqs)}]
    got = U.run_trace(_session(model_dir, dtype, 384), steps).rows
    assert set(got) == set(alone)
    for key, row in got.items():
        assert U.rel_err(row, alone[key]) <= (2e-5 if dtype == "float32" else 3e-2), key


def test_tensors_of_a_half_that_a_layer_does_not_have_may_lie_in_the_file(tmp_path):
    cfg = CONFIGS["mixers_only"]
    S, W = cfg["streams"], cfg["width"]
    w = P.random_weights(cfg, 2)
    toks = U.make_requests(cfg["vocab"], [20], 2)["r0"]
    plain = {"r0": P.forward(cfg, w, toks).numpy()}
    more = dict(w, **{"l1.norm2": torch.ones(W), "l1.norm2.b": torch.ones(W), "l1.hc2.in": torch.ones(S), "l1.hc2.out": torch.ones(S),
                      "l1.hc2.mix": torch.ones(S, S)})
    U.write_model_dir(str(tmp_path / "more"), cfg, {k: v.float() for k, v in more.items()}, torch.bfloat16)
    sess = _session(str(tmp_path / "more"), "float32", 64)
    U.compare(U.run_trace(sess, U.trace_whole({"r0": toks})), plain, U.TOL["float32"], "unused tensors")


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", ["loop_inside", "odd_sizes", "equal_or_one"])
def test_greedy_generation_through_the_engine(tmp_path, name, graphs):
    from firefly_b200 import LLM
    cfg = CONFIGS[name]
    model_dir, w = _model_dir(tmp_path, "gen", cfg, seed=6)
    prompts = [v for v in U.make_requests(cfg["vocab"], [19, 3, 41, 8, 27], 11).values()]
    llm = LLM(model_dir, dtype="float32", max_batch_size_limit=3, kv_block_size=8, num_kv_blocks=40,
              max_prefill_chunk_size=16, eos_token_ids=[], use_cuda_graphs=graphs)
    outs = llm.generate(prompts, max_tokens=10, ignore_eos=True)
    llm.engine.cache.check()
    for p, o in zip(prompts, outs):
        assert len(o) == 10
        rows = P.forward(cfg, w, list(p) + o[:-1])
        for i, tok in enumerate(o):
            row = rows[len(p) - 1 + i]
            top2 = torch.topk(row, 2).values
            assert tok == int(row.argmax()) or float(top2[0] - top2[1]) < 1e-4 * float(row.abs().max()), (i, tok)


def test_generation_in_bfloat16_with_graphs_stays_near_the_plain_model_s_best(tmp_path):
    from firefly_b200 import LLM
    cfg = CONFIGS["fast_paths"]
    model_dir, w = _model_dir(tmp_path, "genbf", cfg, seed=7, static_choice=True)
    prompts = [v for v in U.make_requests(cfg["vocab"], [90, 5, 33], 12).values()]
    llm = LLM(model_dir, dtype="bfloat16", max_batch_size_limit=4, num_kv_blocks=64, max_prefill_chunk_size=64,
              eos_token_ids=[], use_cuda_graphs=True)
    outs = llm.generate(prompts, max_tokens=12, ignore_eos=True)
    llm.engine.cache.check()
    for p, o in zip(prompts, outs):
        rows = P.forward(cfg, w, list(p) + o[:-1])
        for i, tok in enumerate(o):
            row = rows[len(p) - 1 + i]
            assert float(row.max() - row[tok]) <= 5e-2 * float(row.abs().max()), (i, tok)


def _program(name):
    return os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "bin", name)


def test_the_command_line_generates_from_a_folder_and_from_a_configuration(tmp_path):
    model_dir, _ = _model_dir(tmp_path, "cli", CONFIGS["loop_inside"])
    out = subprocess.run([sys.executable, _program("firefly"), model_dir, "--prompt-ids", "5,9,2", "--max-tokens", "4", "--ignore-eos"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    assert len(json.loads(out.stdout.strip().splitlines()[-1])["tokens"]) == 4
    conf = tmp_path / "c.json"
    conf.write_text(json.dumps(CONFIGS["odd_sizes"]))
    out = subprocess.run([sys.executable, _program("firefly"), "--random", str(conf), "--prompt-len", "9", "--num-prompts", "2",
                          "--max-tokens", "3", "--ignore-eos"], capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr


def test_the_trace_program_replays_a_mixed_schedule(tmp_path):
    cfg = CONFIGS["loop_inside"]
    model_dir, w = _model_dir(tmp_path, "prog", cfg, seed=9)
    reqs = U.make_requests(cfg["vocab"], [40, 9, 77, 2, 31], 3)
    plain = {rid: P.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}
    steps = U.trace_mixed(reqs, seed=1, max_live=4)
    out = tmp_path / "out"
    run = subprocess.run([sys.executable, _program("trace_run"), "--model", model_dir, "--dtype", "float32", "--out", str(out),
                          "--max-tokens", str(U.peak_tokens(steps))], input="".join(json.dumps(s) + "\n" for s in steps),
                         capture_output=True, text=True, timeout=900)
    assert run.returncode == 0, run.stderr
    assert [ln for ln in run.stdout.splitlines() if ln.startswith("done ")] == [f"done {s['step']}" for s in steps]
    done = {}
    for rec in steps:
        arr = np.fromfile(out / f"{rec['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        k = 0
        for ent in rec["entries"]:
            base = done.get(ent["id"], 0)
            for wpos in ent["want"]:
                assert U.rel_err(arr[k], plain[ent["id"]][base + wpos]) <= U.TOL["float32"], (rec["step"], ent["id"], wpos)
                k += 1
            done[ent["id"]] = base + len(ent["tokens"])
        assert k == arr.shape[0]
