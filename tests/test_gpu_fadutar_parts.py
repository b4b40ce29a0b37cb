"""The mechanisms of the Fadutar decoder one by one, each kernel or part against the plain function of the same
mechanism (tests/plain/fadutar.py): norms stored around zero, the softmax with learned sinks within chunks on every
attention kernel (edge keys made to stand out, scores so low that the sink takes all), attention that reads another
layer's keys, latent attention with sinks, the gated linear recurrence (its kernels apart and the part in prompts,
portions and single tokens) and the feed-forward with a limited gate and biases on every product."""
import numpy as np
import pytest
import torch

from plain import fadutar as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _t(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device=DEV).contiguous()


def _ints(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def _close(got, want, tol):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape
    if got.size:
        assert np.abs(got - want).max() <= tol * max(1.0, np.abs(want).max()), np.abs(got - want).max()


def _bf16(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32).to(torch.bfloat16).float().numpy()


# ------------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_norm_weights_are_a_difference_from_one(dtype):
    from xeno_rt_b200.core import parse_dtype
    from xeno_rt_b200.parts import part_class
    from xeno_rt_b200.parts.norm import WeightedParts
    rng = np.random.default_rng(1)
    width, eps = 72, 1e-5
    w, w2 = _bf16(rng.normal(0, 0.02, width)), _bf16(rng.normal(0, 0.3, width))
    mk = lambda v: part_class("norm", "rmsnorm")({"width": width, "eps": eps, "offset": 1.0}, {"weight": _t(v).to(DT[dtype])},
                                                 parse_dtype(dtype), DEV)
    norm, then = mk(w), mk(w2)
    x, y = rng.normal(size=(5, width)).astype(np.float32), rng.normal(0.3, 2.0, size=(5, width)).astype(np.float32)
    # 1 + w is a 32-bit sum: rounded to bfloat16 it would lose most of these weights
    _close(norm.forward_f32(_t(x)).cpu().numpy(), plain.offset_norm(x, w, eps), 2e-6)
    _close(norm.forward(_t(x)).float().cpu().numpy(), plain.offset_norm(x, w, eps), 2e-6 if dtype == "float32" else 8e-3)
    bias = rng.normal(size=width).astype(np.float32)
    residual = _t(x)
    h = norm.add_into(residual, WeightedParts(_t(y), bias=_t(bias)), then=then)
    new = x + plain.offset_norm(y + bias, w, eps)
    _close(residual.cpu().numpy(), new, 3e-6)
    _close(h.float().cpu().numpy(), plain.offset_norm(new, w2, eps), 3e-6 if dtype == "float32" else 8e-3)


# ------------------------------------------------------------------------------------------------ chunks and sinks
def _cache_of(k, v, kv, size, dtype, order):
    kp = torch.zeros((max(order) + 1, kv, 64, size), dtype=dtype, device=DEV)
    vp = torch.zeros_like(kp)
    for pos in range(k.shape[0]):
        kp[order[pos // 64], :, pos % 64] = _t(k[pos]).to(dtype)
        vp[order[pos // 64], :, pos % 64] = _t(v[pos]).to(dtype)
    return kp, vp


def _plain_attend(q, k, v, scale, chunk, sinks):
    n, heads, _ = q.shape
    group = heads // k.shape[1]
    out = np.zeros((n, heads, v.shape[2]))
    for t in range(n):
        js = plain.visible(t, chunk)
        for a in range(heads):
            p = plain.sink_weights(k[js.start:js.stop, a // group] @ q[t, a] * scale, sinks[a])
            out[t, a] = p @ v[js.start:js.stop, a // group]
    return out.reshape(n, -1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,size,chunk", [(4, 2, 16, 40), (6, 2, 32, 90), (3, 3, 48, 5), (2, 1, 64, 64), (12, 1, 96, 130),
                                                 (4, 1, 128, 1), (6, 2, 128, 70), (4, 4, 128, 150), (8, 1, 256, 129),
                                                 (2, 2, 32, 0), (2, 1, 128, 0), (16, 1, 160, 0)])
def test_softmax_with_learned_sinks_within_chunks(dtype, heads, kv, size, chunk):
    """Random q and k of unit size would give flat weights that hide a key that is wrongly seen or missed.  So at chosen
    query positions (the first of a chunk, the last, one inside) the first key of the chunk and the key just before it
    line up with the query and have values of their own.  Other queries are turned away from all their keys: there the
    sink holds nearly all of the weight.  Chunk 0 = every key: a key 300 tokens back stands out instead."""
    from xeno_rt_b200.csrc import ops
    rng = np.random.default_rng(5)
    n = 330
    tdt = DT[dtype]
    scale = 6.0 / np.sqrt(size)
    unit = lambda a: a / np.sqrt((a * a).mean(-1, keepdims=True))
    q, k = unit(rng.normal(size=(n, heads, size))), unit(rng.normal(size=(n, kv, size)))
    v = rng.normal(size=(n, kv, size))
    sinks = rng.normal(2.0, 2.0, heads).astype(np.float32)
    reach = chunk or 330
    edges = [c * reach for c in range(1, n // reach + 1) if c * reach < n][:6]
    for first in edges:
        for i in (first, min(n, first + reach) - 1, min(n, first + reach) - 1 - reach // 2):
            for j in (first, first - 1):
                if j <= i and j != i:
                    k[j] = q[i, ::heads // kv] * 0.98 + 0.02 * k[j]
    if not chunk:
        k[3] = q[329, ::heads // kv]
    u = unit(rng.normal(size=(kv, size)))
    k = k + 2.0 * u
    lonely = [151, 328]
    for i in lonely:
        least = min(float(u[g] @ k[j, g]) for j in plain.visible(i, chunk) for g in range(kv))
        assert least > 0
        q[i] = np.repeat(-u * (30.0 / (least * scale)), heads // kv, axis=0)
    if dtype == "bfloat16":
        q, k, v = _bf16(q), _bf16(k), _bf16(v)
    want = _plain_attend(q, k, v, scale, chunk, sinks)
    without = _plain_attend(q, k, v, scale, chunk, np.full(heads, -1e5))
    assert min(np.abs(want[i]).max() for i in lonely) < 0.05 and np.abs(without[lonely[0]]).max() > 0.2
    tol = 3e-5 if dtype == "float32" else 2.5e-2
    if chunk > 1:
        assert np.abs(_plain_attend(q, k, v, scale, chunk + 1, sinks) - want).max() > 0.2  # the inputs show the edge
    order = [5, 1, 4, 0, 2, 7]  # the sequence's blocks are scattered over the pool
    kp, vp = _cache_of(k, v, kv, size, tdt, order)
    table = torch.full((3, 8), -1, dtype=torch.int32, device=DEV)
    table[2, :6] = _ints(order)
    qd, sd = _t(q.reshape(n, heads * size)).to(tdt), _t(sinks)
    out = torch.empty_like(qd)
    ops.attention_reference(out, qd, kp, vp, _ints([2] * n), _ints(range(n)), table, heads, kv, size, scale, sink=sd,
                            mask_chunk=chunk)
    _close(out.float().cpu().numpy(), want, tol)
    if dtype == "float32":
        return
    # prompts: the whole sequence as one step, and its tail as a step that continues it; a block that no query of the
    # step sees any more may be gone from the table
    kernels = [ops.attention_prefill] + ([ops.attention_prefill_tcgen05] if size == 128 else [])
    for kernel in kernels:
        for start in (0, 64, 150, 327):
            seen = table.clone()
            if chunk:
                seen[2, :(start - start % chunk) // 64] = -1
            out = torch.zeros((n - start, heads * size), dtype=tdt, device=DEV)
            sink = {"sink": sd} if kernel is ops.attention_prefill else {"sinks": sd}
            kernel(out, qd[start:].contiguous(), kp, vp, _ints([0, n - start]), _ints([2]), _ints([start]), seen, n - start,
                   heads, kv, size, scale, mask_chunk=chunk, **sink)
            _close(out.float().cpu().numpy(), want[start:], tol)
    # single tokens: every position as a step's one new token, the visible keys cut into splits or not, merged by a
    # second kernel, by the last block and as clusters; a row of no sequence gives zeros
    slots = _ints([2] * (n - 1) + [-1])
    for chunk_keys, splits in ((64, 7), (128, 4), (448, 1)):
        if chunk_keys * splits < reach + 63:
            continue
        for fused, clusters in ((False, False), (True, False), (False, True)):
            if clusters and n * kv > ops.tuning().decode_cluster_pairs:  # few pairs only: take some rows
                rows = [0, 1, 63, 64, 128, 151, 200, 328] + [e for e in edges] + [e - 1 for e in edges]
            else:
                rows = list(range(n))
            rows = sorted(set(rows))
            out = torch.empty((len(rows), heads * size), dtype=tdt, device=DEV)
            ops.attention_decode(out, qd[rows].contiguous(), kp, vp, slots[rows].contiguous(), _ints(rows), table, heads, kv,
                                 size, scale, 0, chunk_keys, splits, fused=fused, clusters=clusters, sinks=sd, mask_chunk=chunk)
            got = out.float().cpu().numpy()
            for i, r in enumerate(rows):
                _close(got[i], want[r] if r < n - 1 else np.zeros_like(want[r]), tol)
    for chunk_keys, splits in ((32, 11), (352, 1)):  # the kernel of layers with score options takes chunks and sinks too
        out = torch.empty_like(qd)
        ops.attention_decode_scored(out, qd, kp, vp, slots, _ints(range(n)), table, heads, kv, size, scale, 0, 0, 0.0, 0.0,
                                    chunk_keys, splits, sink=sd, mask_chunk=chunk)
        _close(out.float().cpu().numpy()[:-1], want[:-1], tol)
    ops.check_error_flag(DEV)


# ------------------------------------------------------------------------------------------------ parts with a cache
def _run_mixer(part, cache, dtype, hs, plan, owns=True, slots=None, advance=True):
    """Runs ``part.mix`` over sequences whose inputs are ``hs`` ([T_i, width] each); ``plan`` lists for every step how
    many tokens each sequence brings.  Returns the results a sequence and the slots (left open)."""
    from xeno_rt_b200.core import parse_dtype
    from xeno_rt_b200.engine import StepEntry, build_context
    slots = [cache.open_slot() for _ in hs] if slots is None else slots
    at, got = [0] * len(hs), [[] for _ in hs]
    for step in plan:
        live = [(i, k) for i, k in enumerate(step) if k]
        ctx, _ = build_context([StepEntry(slots[i], [0] * k) for i, k in live], cache, 10, parse_dtype(dtype), DEV)
        cache.flush_tables()
        h = torch.cat([_t(hs[i][at[i]:at[i] + k]) for i, k in live]).to(DT[dtype])
        out = part.mix(h, ctx, cache.store(0), owns).float().cpu().numpy()
        row = 0
        for i, k in live:
            got[i].append(out[row:row + k])
            row += k
            at[i] += k
            if advance:
                cache.advance(slots[i], k)
    return [np.concatenate(g) for g in got], slots


def _part(kind, params, tensors, dtype):
    from xeno_rt_b200.core import parse_dtype
    from xeno_rt_b200.parts import part_class
    cls = part_class("mixer", kind)
    kinds = {role: k for role, (_, k) in cls.weight_shapes(params).items()}
    return cls(params, {r: _t(w).to(torch.float32 if kinds[r] == "vector" else DT[dtype]) for r, w in tensors.items()},
               parse_dtype(dtype), DEV)


PLANS = [[2, 1, 3], [1, 0, 2], [60, 0, 59], [3, 0, 6], [150, 0, 0]] + [[1, 0, 0]] * 19, [[200, 0, 64]] + [[1, 1, 1]] + [[1, 0, 1]] * 5 + [[1, 0, 0]] * 29


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(3, 8, 8, 16, 24), (1, 12, 6, 20, 13), (4, 64, 64, 48, 192),
                                                     (2, 16, 32, 16, 300), (20, 8, 4, 8, 12)])
def test_latent_attention_with_sinks_in_prompts_portions_and_single_tokens(dtype, heads, dim, rot, vdim, rank):
    from xeno_rt_b200.cache import Cache
    from xeno_rt_b200.core import parse_dtype
    rng = np.random.default_rng(11)
    width, eps = 72, 1e-5
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"dims": rot, "base": 300.0},
         "scale": 1.5 / np.sqrt(dim + rot)}
    mk = lambda rows, cols, s=1.0: _bf16(rng.normal(0, s / np.sqrt(cols), (rows, cols)))
    w = {"q": mk(heads * (dim + rot), width, 2.0), "dkv": mk(rank + rot, width, 2.0), "dkv.norm": _bf16(rng.normal(1.0, 0.3, rank)),
         "uk": mk(heads * dim, rank), "uv": mk(heads * vdim, rank), "o": mk(width, heads * vdim),
         "sink": _bf16(rng.normal(3.0, 1.5, heads))}
    params = {"width": width, "n_heads": heads, "head_dim": dim, "rot_dim": rot, "v_head_dim": vdim, "kv_rank": rank, "eps": eps,
              "window": None, "scale": m["scale"], "sink": "learned",
              "position": {"kind": "blended_rotary", "params": {"rope_dim": rot, "base": 300.0, "pairing": "split_half",
                                                                "scaling": None}}}
    part = _part("latent_attention", params, {"q": w["q"], "down": w["dkv"], "down_norm": w["dkv.norm"], "up_k": w["uk"],
                                              "up_v": w["uv"], "o": w["o"], "sink": w["sink"]}, dtype)
    hs = [_bf16(rng.normal(size=(n, width))) for n in (235, 2, 70)]
    wants = [plain.latent_attention(h, w, m, eps) for h in hs]
    other = plain.latent_attention(hs[0], dict(w, sink=np.roll(w["sink"], 1) + 1.0), m, eps)
    assert np.abs(other - wants[0]).max() > 0.05 * np.abs(wants[0]).max()  # the sinks show
    tol = 3e-5 if dtype == "float32" else 3e-2
    for steps in ([[235, 2, 70]],) + PLANS:
        cache = Cache([part.cache_need()], 64 * 8, 1024, parse_dtype(dtype), DEV)
        got, slots = _run_mixer(part, cache, dtype, hs, steps)
        for g, want in zip(got, wants):
            _close(g, want[:len(g)], tol)
        for s in slots:
            cache.close_slot(s)
        cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim,own_chunk,reader_chunk,reader_heads", [(24, 40, 70, 20, 3), (64, 64, 40, 130, 6),
                                                                        (128, 128, 64, 96, 3), (16, 16, 50, 0, 9)])
def test_a_layer_reads_the_keys_and_values_another_layer_cached(dtype, dim, vdim, own_chunk, reader_chunk, reader_heads):
    """The owner writes keys and values; the reader has queries, sinks, chunks and a scale of its own and must leave the
    cache alone, in prompts, portions and single tokens (where heads of 64 and 128 have ONE kernel for the step between
    the product and attention)."""
    import dataclasses
    from xeno_rt_b200.cache import Cache
    from xeno_rt_b200.core import parse_dtype
    from xeno_rt_b200.engine import StepEntry, build_context
    rng = np.random.default_rng(14)
    width, kv = 40, 3
    mk = lambda rows, cols, s=1.5: _bf16(rng.normal(0, s / np.sqrt(cols), (rows, cols)))

    def build(heads, chunk, own):
        m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 1.5 / np.sqrt(dim)}
        if chunk:
            m["mask"] = {"size": chunk}
        w = {"q": mk(heads * dim, width), "o": mk(width, heads * vdim), "sink": _bf16(rng.normal(1.0, 1.5, heads))}
        if own:
            w.update({"k": mk(kv * dim, width), "v": mk(kv * vdim, width)})
        params = {"width": width, "n_heads": heads, "n_kv_heads": kv, "head_dim": dim, "v_head_dim": vdim, "qk_norm": False,
                  "scale": m["scale"], "sink": "learned", "chunk": chunk or None, "own_kv": own}
        return _part("attention", params, w, dtype), w, m

    owner, w_own, m_own = build(3, own_chunk, True)
    reader, w_read, m_read = build(reader_heads, reader_chunk, False)
    n = 200
    h_own, h_read = _bf16(rng.normal(size=(n, width))), _bf16(rng.normal(size=(n, width)))
    kept = plain.attention_keys_values(h_own, w_own, m_own)
    want_own, want_read = plain.attention(h_own, w_own, m_own, kept), plain.attention(h_read, w_read, m_read, kept)
    need = dataclasses.replace(owner.cache_need(), window=max(own_chunk, reader_chunk) if reader_chunk else None)
    cache = Cache([need], 64 * 6, 1024, parse_dtype(dtype), DEV)
    slot = cache.open_slot()
    got_own, got_read, at = [], [], 0
    for k in [131, 2, 3] + [1] * 64:
        ctx, _ = build_context([StepEntry(slot, [0] * k)], cache, 10, parse_dtype(dtype), DEV)
        cache.flush_tables()
        got_own.append(owner.mix(_t(h_own[at:at + k]).to(DT[dtype]), ctx, cache.store(0), True).float().cpu().numpy())
        snapshot = cache.store(0).k.clone()
        got_read.append(reader.mix(_t(h_read[at:at + k]).to(DT[dtype]), ctx, cache.store(0), False).float().cpu().numpy())
        assert torch.equal(snapshot, cache.store(0).k)
        cache.advance(slot, k)
        at += k
    tol = 3e-5 if dtype == "float32" else 3e-2
    _close(np.concatenate(got_own), want_own, tol)
    _close(np.concatenate(got_read), want_read, tol)
    cache.check()


# ------------------------------------------------------------------------------------------------ the recurrence
def _recurrence_weights(rng, width, inner, blocks, taps, lam=(-4.0, 1.5)):
    mk = lambda shape, s: _bf16(rng.normal(0, s, shape))
    size = inner // blocks
    return {"y": mk((inner, width), 1.5 / np.sqrt(width)), "y.b": mk(inner, 0.5), "x": mk((inner, width), 1.5 / np.sqrt(width)),
            "x.b": mk(inner, 0.5), "conv": mk((inner, taps), 0.7), "conv.b": mk(inner, 0.3),
            "ra": mk((blocks, size, size), 1.5 / np.sqrt(size)), "ra.b": mk((blocks, size), 0.5),
            "ri": mk((blocks, size, size), 1.5 / np.sqrt(size)), "ri.b": mk((blocks, size), 0.5),
            "lam": _bf16(rng.normal(*lam, inner)), "o": mk((width, inner), 1.0 / np.sqrt(inner))}


ROLES = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra", "r_bias": "ra.b",
         "i": "ri", "i_bias": "ri.b", "lam": "lam", "o": "o"}


def _recurrence(w, width, inner, blocks, taps, dtype):
    return _part("gated_linear_recurrence", {"width": width, "inner": inner, "blocks": blocks, "taps": taps, "decay_scale": 8.0},
                 {role: w[name] for role, name in ROLES.items()}, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("inner,blocks,taps", [(96, 4, 4), (33, 33, 5), (60, 5, 1), (48, 6, 2), (640, 2, 3), (72, 1, 9), (272, 2, 4)])
def test_the_recurrence_in_prompts_portions_and_single_tokens(dtype, inner, blocks, taps):
    """Prompts over several tiles of 64 tokens, portions down to one and two tokens (also fewer than the convolution has
    taps), sequences of unequal lengths beside each other, the tail token by token; then the slots again for other
    sequences, which must find nothing of the first."""
    from xeno_rt_b200.cache import Cache
    from xeno_rt_b200.core import parse_dtype
    rng = np.random.default_rng(21)
    width = 40
    w = _recurrence_weights(rng, width, inner, blocks, taps)
    part = _recurrence(w, width, inner, blocks, taps, dtype)
    assert part.one_launch == (dtype == "bfloat16" and inner // blocks % 8 == 0)
    hs = [_bf16(rng.normal(size=(n, width))) for n in (235, 2, 70)]
    wants = [plain.recurrent(h, w) for h in hs]
    tol = 3e-5 if dtype == "float32" else 2e-2
    cache = Cache([part.cache_need()], 64 * 8, 1024, parse_dtype(dtype), DEV, max_slots=3)
    for turn, steps in enumerate(([[235, 2, 70]],) + PLANS + ([[1, 1, 1]] * 2 + [[1, 0, 1]] * 68,)):
        slots = [cache.open_slot() for _ in hs]
        got, _ = _run_mixer(part, cache, dtype, hs, steps, slots=slots if turn % 2 else slots[::-1])
        for g, want in zip(got, wants):
            _close(g, want[:len(g)], tol)
        for s in slots:
            cache.close_slot(s)


@pytest.mark.parametrize("inner,blocks,taps", [(96, 4, 4), (640, 2, 3), (64, 8, 1), (272, 2, 9)])
def test_the_gates_are_32_bit_under_bfloat16_matrices(inner, blocks, taps):
    """The kernels alone on 32-bit branches: the gates' products take u as it is (rounded to bfloat16 first, the result
    would be 40 to 70 times this bound off), in the prompt kernels and in the one-launch step alike."""
    from xeno_rt_b200.csrc import ops
    rng = np.random.default_rng(22)
    n = 150
    w = _recurrence_weights(rng, 8, inner, blocks, taps, lam=(-6.0, 1.0))
    p = rng.normal(size=(n, 2 * inner)).astype(np.float32)
    y, x = p[:, :inner].astype(np.float64), p[:, inner:].astype(np.float64)
    u = plain.short_convolution(x + w["x.b"], w["conv"], w["conv.b"])
    gates = [plain.sigmoid(plain.block_product(u, w[m], w[m + ".b"])) for m in ("ra", "ri")]
    want = plain.linear_recurrence(u, *gates, w["lam"]) * plain.gelu_tanh(y + w["y.b"])
    rounded = [plain.sigmoid(plain.block_product(_bf16(u), w[m], w[m + ".b"])) for m in ("ra", "ri")]
    off = np.abs(plain.linear_recurrence(u, *rounded, w["lam"]) * plain.gelu_tanh(y + w["y.b"]) - want).max()
    tol = 5e-6
    assert off > 20 * tol * max(1.0, np.abs(want).max())
    part = _recurrence(w, 8, inner, blocks, taps, "bfloat16")
    assert ops.recurrence_tensor_cores(part.weights)
    new = lambda: (torch.zeros((4, inner), device=DEV), torch.full((4, taps, inner), 7.0, device=DEV))
    pd = _t(p)
    results = []
    for cuts in ([n], [1, 2, 64, 3, 80]):
        state, ring = new()
        rows, at = [], 0
        for k in cuts:
            out = torch.empty((k, inner), device=DEV)  # 32-bit results of the prompt kernels
            ops.linear_recurrence(out, pd[at:at + k].contiguous(), part.weights, state, ring, _ints([0, k]), _ints([2]), _ints([at]), k)
            rows.append(out)
            at += k
        got = torch.cat(rows).cpu().numpy()
        _close(got, want, tol)
        results.append((got, state.cpu().numpy()))
        assert not state[[0, 1, 3]].any() and bool((ring[[0, 1, 3]] == 7.0).all())  # no other slot is touched
    _close(results[1][0], results[0][0], 3e-6)
    # the one-launch step, from the first token on: its states stay beside the 32-bit ones, its results are their bfloat16
    state, ring = new()
    arrays = (_ints([2, -1]), _ints([0, 1, 2]), _ints([2, -1]))
    for t in range(n):
        out = torch.full((2, inner), 9.0, dtype=torch.bfloat16, device=DEV)
        rows = torch.cat([pd[t:t + 1], pd[t:t + 1]])
        ops.linear_recurrence_step(out, rows, part.weights, state, ring, arrays[0], _ints([t, 0]), arrays[1], arrays[2], _ints([t, 0]))
        _close(out[0].float().cpu().numpy(), want[t], 6e-3)
        assert not out[1].any()
    _close(state[2].cpu().numpy(), results[0][1][2], 1e-5)
    assert not state[[0, 1, 3]].any()


def test_decays_near_one_and_near_zero():
    """log a from -1e-6 to -60: sqrt(1 - a^2) keeps its digits near a = 1 and nothing overflows near a = 0."""
    from xeno_rt_b200.csrc import ops
    rng = np.random.default_rng(23)
    inner, n = 64, 200
    w = _recurrence_weights(rng, 8, inner, 4, 2)
    w["lam"] = _bf16(np.linspace(-15.0, 12.0, inner))
    part = _recurrence(w, 8, inner, 4, 2, "bfloat16")
    p = rng.normal(size=(n, 2 * inner)).astype(np.float32)
    u = plain.short_convolution(p[:, inner:] + w["x.b"].astype(np.float64), w["conv"], w["conv.b"])
    gates = [plain.sigmoid(plain.block_product(u, w[m], w[m + ".b"])) for m in ("ra", "ri")]
    want = plain.linear_recurrence(u, *gates, w["lam"]) * plain.gelu_tanh(p[:, :inner] + w["y.b"].astype(np.float64))
    out = torch.empty((n, inner), device=DEV)
    state, ring = torch.zeros((1, inner), device=DEV), torch.zeros((1, 2, inner), device=DEV)
    ops.linear_recurrence(out, _t(p), part.weights, state, ring, _ints([0, n]), _ints([0]), _ints([0]), n)
    err = np.abs(out.cpu().numpy() - want) / np.maximum(np.abs(want).max(0), 1e-6)  # channel by channel
    assert err.max() < 2e-5, (err.max(), int(np.argmax(err.max(0))))


# ------------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [1, 8, 19, 90, 200])
@pytest.mark.parametrize("width,inner,limit", [(64, 40, 1.5), (256, 384, 0.7), (36, 33, 3.0), (512, 520, 2.0)])
def test_the_limited_gate_with_biases_on_every_product(dtype, n, width, inner, limit):
    """Few rows (the weight-streaming products), up to 128 (split K), more (tiles), and 32-bit; gate and up sums beyond
    the limit on both sides.  The down product's bias is left for the norm that follows."""
    from xeno_rt_b200.core import parse_dtype
    from xeno_rt_b200.parts import part_class
    from xeno_rt_b200.parts.norm import WeightedParts
    rng = np.random.default_rng(31)
    w = {"gate": _bf16(rng.normal(0, 2.0 / np.sqrt(width), (inner, width))), "up": _bf16(rng.normal(0, 2.0 / np.sqrt(width), (inner, width))),
         "down": _bf16(rng.normal(0, 1.0 / np.sqrt(inner), (width, inner))), "gate.b": _bf16(rng.normal(0, 0.7, inner)),
         "up.b": _bf16(rng.normal(0, 0.7, inner)), "down.b": _bf16(rng.normal(0, 0.7, width))}
    params = {"width": width, "inner": inner, "activation": "gated_sigmoid", "limit": limit, "alpha": 1.702, "bias": True}
    tensors = {r: _t(w[r]).to(DT[dtype]) for r in ("gate", "up", "down")}
    tensors.update({r + "_bias": _t(w[r + ".b"]) for r in ("gate", "up", "down")})
    part = part_class("feed_forward", "swiglu")(params, tensors, parse_dtype(dtype), DEV)
    h = _bf16(rng.normal(size=(n, width)))
    want = plain.dense_ff(h.astype(np.float64), w, limit)
    g = h @ w["gate"].T + w["gate.b"]
    assert (g > limit).mean() > 0.02 and plain.limited_gate(limit + 1, limit + 5, limit) == plain.limited_gate(limit, limit, limit)

    class Ctx:
        then_norm = None
    y = part.apply(_t(h).to(DT[dtype]), Ctx())
    assert isinstance(y, WeightedParts)
    tol = 2e-5 if dtype == "float32" else 1.5e-2
    _close((y.parts + y.bias).cpu().numpy(), want, tol)
    out = torch.empty((n, width), device=DEV)
    _close(part.apply(_t(h).to(DT[dtype]), Ctx(), out=out).cpu().numpy(), want, tol)
    residual = torch.ones((n, width), device=DEV)
    part.forward(_t(h).to(DT[dtype]), residual, Ctx())
    _close(residual.cpu().numpy() - 1.0, want, tol)
