"""The mechanisms of the Zivovik decoder one by one, each kernel or part against the plain function of the same mechanism
(tests/plain/zivovik.py): the embedding with a row a position, the query temperature and values tied to the keys in every
kernel that prepares heads, each mixer alone through the cache (prompts, portions, single tokens, slots used again), the
scan with one decay a head (unit q and k, silu, raw and constant decays, a far token that the state must still hold), the
sum into the stream with its norms, gathered rows and the norm that follows, routing and experts on both of their paths."""
import numpy as np
import pytest
import torch

from plain import zivovik as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _t(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device=DEV).contiguous()


def _ints(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def _bf16(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32).to(torch.bfloat16).to(torch.float64).numpy()


def _close(got, want, tol):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape
    if got.size:
        assert np.isfinite(got).all() and np.abs(got - want).max() <= tol * max(1.0, np.abs(want).max()), np.abs(got - want).max()


# ------------------------------------------------------------------------------------------------ embedding
@pytest.mark.parametrize("width", [36, 64, 200])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_adds_an_unscaled_row_a_position(width, dtype):
    from xeno_rt_b200.csrc import ops
    rng = np.random.default_rng(width)
    table, pos = _bf16(rng.normal(size=(11, width))), _bf16(rng.normal(size=(300, width)))
    ids, at = rng.integers(0, 11, 9), np.array([0, 1, 63, 64, 65, 128, 200, 298, 299])
    out = torch.empty((9, width), device=DEV)
    flag = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.embedding(out, _t(table, DT[dtype]), _ints(ids), flag, 2.5, _t(pos, DT[dtype]), _ints(at))
    _close(out.cpu().numpy(), table[ids] * 2.5 + pos[at], 1e-6)
    assert int(flag) == 0
    ops.embedding(out, _t(table, DT[dtype]), _ints(ids), flag, 2.5)
    _close(out.cpu().numpy(), table[ids] * 2.5, 1e-6)
    ops.embedding(out[:2], _t(table, DT[dtype]), _ints([1, 2]), flag, 1.0, _t(pos, DT[dtype]), _ints([3, 300]))
    assert int(flag) == 1 and not bool(out[1].any())   # a position beyond the table: zeros and the error flag


# ------------------------------------------------------------------------------------------------ parts with a cache
def _run_mixer(part, cache, dtype, hs, plan, slots=None):
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
        out = part.mix(h, ctx, cache.store(0), True)
        if not isinstance(out, torch.Tensor):   # in parts: what the next kernel would add up
            from xeno_rt_b200.csrc import ops
            y, out = out, torch.zeros((h.shape[0], h.shape[1]), device=DEV)
            ops.stream_add(out, y.parts, 1.0, scales=y.scales, part_norms=y.norms, part_eps=y.eps)
        out = out.float().cpu().numpy()
        row = 0
        for i, k in live:
            got[i].append(out[row:row + k])
            row += k
            at[i] += k
            cache.advance(slots[i], k)
    return [np.concatenate(g) for g in got], slots


def _part(kind, params, tensors, dtype):
    from xeno_rt_b200.core import parse_dtype
    from xeno_rt_b200.parts import part_class
    cls = part_class("mixer", kind)
    kinds = {role: k for role, (_, k) in cls.weight_shapes(params).items()}
    assert set(kinds) == set(tensors)
    return cls(params, {r: _t(w).to(torch.float32 if kinds[r] == "vector" else DT[dtype]) for r, w in tensors.items()},
               parse_dtype(dtype), DEV)


PLANS = [[2, 1, 3], [1, 0, 2], [60, 0, 59], [3, 0, 6], [150, 0, 0]] + [[1, 0, 0]] * 19, [[200, 0, 64]] + [[1, 1, 1]] + [[1, 0, 1]] * 5 + [[1, 0, 0]] * 29


def _check_mixer(part, dtype, hs, wants, tol):
    """The mixer over its cache: whole prompts beside each other, portions, single tokens; then the slots and blocks again
    for other runs, which must find nothing of the ones before."""
    from xeno_rt_b200.cache import Cache
    from xeno_rt_b200.core import parse_dtype
    cache = Cache([part.cache_need()], 64 * 8, 1024, parse_dtype(dtype), DEV, max_slots=3)
    for turn, steps in enumerate(([[len(h) for h in hs]],) + PLANS + ([[1, 1, 1]] * 2 + [[1, 0, 1]] * 68,)):
        slots = [cache.open_slot() for _ in hs]
        got, _ = _run_mixer(part, cache, dtype, hs, steps, slots=slots if turn % 2 else slots[::-1])
        for g, want in zip(got, wants):
            _close(g, want[:len(g)], tol)
        for s in slots:
            cache.close_slot(s)
        cache.check()


def _sequences(rng, width):
    return [_bf16(rng.normal(size=(n, width))) for n in (235, 2, 70)]


def _matrices(rng):
    return lambda rows, cols, s=1.0: _bf16(rng.normal(0, s / np.sqrt(cols), (rows, cols)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,dim,temp", [(4, 2, 16, (0.5, 30)), (3, 3, 20, (1.0, 1)), (6, 1, 64, (0.7, 64)),
                                               (8, 2, 128, (0.5, 50)), (17, 1, 24, None), (2, 2, 256, (-0.2, 100)), (4, 4, 96, (0.3, 65))])
def test_attention_with_values_tied_to_the_keys(dtype, heads, kv, dim, temp):
    """Head sizes of every attention kernel; a temperature of many steps, of every position, falling and none."""
    rng = np.random.default_rng(31)
    width, eps = 40, 1e-5
    mk = _matrices(rng)
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "scale": 2.0 / np.sqrt(dim),
         "q_temp": {"coef": temp[0], "every": temp[1]} if temp else None}
    w = {"q": mk(heads * dim, width), "k": mk(kv * dim, width), "g": mk(heads * dim, width), "o": mk(width, heads * dim)}
    params = {"width": width, "n_heads": heads, "n_kv_heads": kv, "head_dim": dim, "v_head_dim": dim, "qk_norm": "unit",
              "eps": eps, "scale": m["scale"], "gate": "sigmoid", "tied_values": True, "q_temp": m["q_temp"]}
    hs = _sequences(rng, width)
    wants = [plain.tied_attention(h, w, m, eps) for h in hs]
    scale = np.abs(wants[0]).max()
    if temp:  # what a temperature that steps one position later, and none, would look like
        late = plain.tied_attention(hs[0], w, dict(m, q_temp={"coef": temp[0], "every": temp[1] + 1}), eps)
        off = plain.tied_attention(hs[0], w, dict(m, q_temp=None), eps)
        assert np.abs(late - wants[0]).max() > 1e-3 * scale and np.abs(off - wants[0]).max() > 0.02 * scale
    _check_mixer(_part("attention", params, w, dtype), dtype, hs, wants, 3e-5 if dtype == "float32" else 3e-2)


def test_tied_values_are_the_keys_before_their_norm():
    """What lies in the cache: unit keys, and beside them the keys as projected."""
    from xeno_rt_b200.cache import Cache
    from xeno_rt_b200.core import parse_dtype
    rng = np.random.default_rng(5)
    width, kv, dim, eps = 24, 2, 20, 1e-5
    mk = _matrices(rng)
    w = {"q": mk(2 * dim, width), "k": mk(kv * dim, width, 3.0), "g": mk(2 * dim, width), "o": mk(width, 2 * dim)}
    part = _part("attention", {"width": width, "n_heads": 2, "n_kv_heads": kv, "head_dim": dim, "qk_norm": "unit", "eps": eps,
                               "gate": "sigmoid", "tied_values": True}, w, "float32")
    cache = Cache([part.cache_need()], 128, 1024, parse_dtype("float32"), DEV)
    h = _bf16(rng.normal(size=(5, width)))
    _run_mixer(part, cache, "float32", [h], [[5]])
    store = cache.store(0)
    k = (h @ w["k"].T).reshape(5, kv, dim)
    block = int(store.block_table.max())
    _close(store.v[block, :, :5, :dim].permute(1, 0, 2).cpu().numpy(), k, 1e-5)
    _close(store.k[block, :, :5, :dim].permute(1, 0, 2).cpu().numpy(), plain.unit_rms(k, eps), 1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,dim,vdim,temp", [(4, 2, 24, 12, (0.5, 30)), (6, 3, 16, 40, (1.0, 64)), (8, 2, 64, 64, (0.5, 50)),
                                                    (4, 4, 128, 128, (0.4, 7)), (5, 5, 8, 8, None), (4, 1, 128, 72, (0.6, 65)),
                                                    (3, 1, 64, 64, (0.6, 40)), (6, 2, 128, 40, None), (1, 1, 256, 256, (0.5, 9))])
def test_attention_with_a_gate_a_head_and_a_temperature(dtype, heads, kv, dim, vdim, temp):
    rng = np.random.default_rng(32)
    width = 40
    mk = _matrices(rng)
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 1.5 / np.sqrt(dim),
         "q_temp": {"coef": temp[0], "every": temp[1]} if temp else None}
    w = {"q": mk(heads * dim, width, 1.3), "k": mk(kv * dim, width, 1.3), "v": mk(kv * vdim, width), "g": mk(heads, width, 2.0),
         "o": mk(width, heads * vdim)}
    params = {"width": width, "n_heads": heads, "n_kv_heads": kv, "head_dim": dim, "v_head_dim": vdim, "qk_norm": False,
              "scale": m["scale"], "gate": "sigmoid_head", "q_temp": m["q_temp"]}
    hs = _sequences(rng, width)
    wants = [plain.head_gated_attention(h, w, m) for h in hs]
    _check_mixer(_part("attention", params, w, dtype), dtype, hs, wants, 3e-5 if dtype == "float32" else 3e-2)


def _delta_weights(rng, width, heads, kv, dim, vdim, taps):
    mk = _matrices(rng)
    w = {"q": mk(kv * dim, width, 1.5), "k": mk(kv * dim, width, 1.5), "v": mk(heads * vdim, width, 1.5),
         "b": mk(heads, width, 1.5), "a": mk(heads, width), "A_log": _bf16(rng.normal(0, 0.7, heads)),
         "dt_bias": _bf16(rng.normal(-3.5, 1.5, heads)), "g": mk(heads * vdim, width), "norm": _bf16(rng.normal(1.0, 0.2, vdim)),
         "o": mk(width, heads * vdim)}
    for name, rows in (("q", kv * dim), ("k", kv * dim), ("v", heads * vdim)):
        w[name + ".conv"] = _bf16(rng.normal(0, 0.7, (rows, taps)))
    return w


def _delta_tensors(w):
    return {(r[0] + "_conv" if r.endswith(".conv") else r): t for r, t in w.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,dim,vdim,taps", [(4, 2, 16, 32, 4), (3, 3, 12, 20, 1), (2, 1, 128, 128, 4), (6, 2, 40, 9, 5),
                                                    (2, 2, 64, 200, 2), (2, 2, 150, 33, 9)])
def test_the_delta_rule_with_one_decay_a_head(dtype, heads, kv, dim, vdim, taps):
    rng = np.random.default_rng(33)
    width, eps = 40, 1e-5
    w = _delta_weights(rng, width, heads, kv, dim, vdim, taps)
    params = {"width": width, "n_heads": heads, "n_qk_heads": kv, "key_dim": dim, "value_dim": vdim, "taps": taps, "eps": eps,
              "gate_act": "silu"}
    part = _part("gated_delta_rule", params, _delta_tensors(w), dtype)
    hs = _sequences(rng, width)
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim}
    wants = [plain.delta_rule(h, w, m, eps) for h in hs]
    _check_mixer(part, dtype, hs, wants, 5e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim,decay", [(16, 24, [0.5, 0.9, 0.99]), (12, 20, [1.0, 0.25]), (128, 64, [0.999, 0.97]),
                                            (50, 8, [0.8]), (4, 130, [0.9, 0.99, 0.3, 0.999])])
def test_linear_attention_with_a_constant_decay_a_head(dtype, dim, vdim, decay):
    rng = np.random.default_rng(34)
    width, eps, heads = 40, 1e-5, len(decay)
    mk = _matrices(rng)
    w = {"q": mk(heads * dim, width, 1.5), "k": mk(heads * dim, width, 1.5), "v": mk(heads * vdim, width, 1.5),
         "g": mk(heads * vdim, width), "norm": _bf16(rng.normal(1.0, 0.2, heads * vdim)), "o": mk(width, heads * vdim)}
    params = {"width": width, "n_heads": heads, "key_dim": dim, "value_dim": vdim, "decay": decay, "eps": eps}
    hs = _sequences(rng, width)
    wants = [plain.lightning(h, w, {"heads": heads, "decay": decay}, eps) for h in hs]
    _check_mixer(_part("constant_decay_linear_attention", params, w, dtype), dtype, hs, wants, 5e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_mean_of_two_mixers_normed_one_by_one(dtype):
    from zivovik_cases import attn, delta, layer, model, temp
    from xeno_rt_b200.config import config_from_dict
    rng = np.random.default_rng(35)
    width, eps = 48, 1e-5
    mixer = {"left": attn(4, 2, 24, 0.4, temp(0.5, 20), vdim=16), "right": delta(4, 2, 16, 24, 4)}
    arch, cfg = config_from_dict(model(10, width, [layer("parallel", mixer, None)], eps=eps))
    spec = arch.build_spec(cfg).layers[0].parts["mixer"][1]
    mk = _matrices(rng)
    w = {f"right.{r}": t for r, t in _delta_weights(rng, width, 4, 2, 16, 24, 4).items()}
    w.update({"left.q": mk(96, width), "left.k": mk(48, width), "left.v": mk(32, width), "left.g": mk(4, width), "left.o": mk(width, 64, 5.0),
              "left.out": _bf16(rng.normal(1.0, 0.3, width)), "right.out": _bf16(rng.normal(1.0, 0.3, width))})
    tensors = {role: w[name[len("l0.mix."):]] for role, name in spec.weights.items()}
    hs = _sequences(rng, width)
    wants = [plain.parallel(h, w, mixer, eps) for h in hs]
    _check_mixer(_part("side_by_side", spec.params, tensors, dtype), dtype, hs, wants, 5e-5 if dtype == "float32" else 4e-2)


# ------------------------------------------------------------------------------------------------ the scan alone
@pytest.mark.parametrize("dim,vdim,heads,kv", [(16, 16, 2, 1), (128, 128, 4, 4), (96, 40, 2, 2), (64, 64, 160, 160), (260, 12, 1, 1),
                                               (600, 20, 2, 1), (33, 7, 3, 3)])
@pytest.mark.parametrize("kind", ["delta", "plain"])
def test_the_scan_holds_a_far_token_exactly(kind, dim, vdim, heads, kv):
    """One write stands out at the first token and its key is asked for again after hundreds of tokens, in one portion and
    in portions and single tokens (the state between them); rows of no sequence are left alone."""
    from xeno_rt_b200.csrc import ops
    rng = np.random.default_rng(dim + heads)
    n = 150
    q, k = rng.normal(size=(n, kv, dim)), rng.normal(size=(n, kv, dim))
    v = rng.normal(size=(n, heads, vdim))
    v[0] *= 200.0
    q[-1] = k[0]
    raw, beta = rng.normal(-7.0, 0.5, (n, heads)), rng.normal(0.0, 1.5, (n, heads))
    a_log, dt_bias, const = rng.normal(0, 0.3, heads), rng.normal(0, 0.3, heads), rng.uniform(0.99, 1.0, heads)
    group = heads // kv
    f32 = lambda a: np.asarray(a, np.float32).astype(np.float64)
    q, k, v, raw, beta, a_log, dt_bias, const = map(f32, (q, k, v, raw, beta, a_log, dt_bias, const))
    if kind == "delta":
        qu, ku = plain.unit_vectors(q) * dim ** -0.5, plain.unit_vectors(k)
        g, b = plain.head_decay(raw, a_log, dt_bias), plain.sigmoid(beta)
        want = np.stack([plain.delta_scan(qu[:, a // group], ku[:, a // group], v[:, a], g[:, a], b[:, a]) for a in range(heads)], 1)
        options = dict(decay_raw=raw, beta=beta, a_log=_t(a_log), dt_bias=_t(dt_bias), q_scale=dim ** -0.5, unit_eps=plain.UNIT_EPS)
    else:
        s = plain.silu
        want = np.stack([plain.constant_decay_scan(s(q[:, a // group]), s(k[:, a // group]), s(v[:, a]), const[a]) for a in range(heads)], 1)
        options = dict(decay=_t(const), silu=True)
    for cuts in ([150], [1, 2, 17, 64, 1, 1, 30, 33, 1]):
        state = torch.zeros((3, heads, vdim, dim), device=DEV)
        state[0] = 5.0
        at, got = 0, []
        for c in cuts:
            now = {key: (_t(val[at:at + c]) if isinstance(val, np.ndarray) else val) for key, val in options.items()}
            pad = lambda t: torch.cat([_t(t[at:at + c].reshape(c, -1)), torch.ones((2, t[0].size), device=DEV)])
            for key in ("decay_raw", "beta"):
                if key in now:
                    now[key] = torch.cat([now[key], torch.ones((2, heads), device=DEV)])
            out = torch.full((c + 2, heads * vdim), 3.0, device=DEV)
            ops.head_scan(out, pad(q), pad(k), pad(v), state, _ints([0, c, c]), _ints([2, -1]), heads, kv, dim, vdim, max_new=c, **now)
            assert bool((out[c:] == 3.0).all())
            got.append(out[:c].cpu().numpy())
            at += c
        assert bool((state[0] == 5.0).all()) and not bool(state[1].any())
        got = np.concatenate(got).reshape(n, heads, vdim)
        for rows in (slice(0, 1), slice(1, n - 1), slice(n - 1, n)):
            _close(got[rows], want[rows], 2e-5)


# ------------------------------------------------------------------------------------------------ sums into the stream
@pytest.mark.parametrize("width", [36, 64, 250, 1024, 3000, 2050])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_results_enter_the_stream_times_a_number_with_the_next_norm(width, out_dtype):
    from xeno_rt_b200.csrc import ops
    rng = np.random.default_rng(width)
    n, parts, eps, mult = 7, 3, 1e-5, 0.35
    x = rng.normal(size=(n, width)).astype(np.float32)
    y = (rng.normal(size=(parts, n, width)) * np.array([1.0, 30.0, 0.01])[:, None, None]).astype(np.float32)
    w2, norms = rng.normal(1.0, 0.2, width).astype(np.float32), rng.normal(1.0, 0.3, (parts, width)).astype(np.float32)
    scales, row_scales = rng.uniform(0.1, 2.0, parts).astype(np.float32), rng.uniform(0.1, 2.0, (n, parts)).astype(np.float32)
    rows = rng.permutation(n * parts)
    pool = np.zeros((n * parts, width), np.float32)
    pool[rows.reshape(n, parts)] = y.transpose(1, 0, 2)
    normed = np.stack([plain.rms_norm(y[p], norms[p], eps) for p in range(parts)])
    y64 = y.astype(np.float64)
    forms = [
        (y, {}, y64.sum(0)),
        (y[1], {}, y64[1]),
        (y, {"scales": _t(scales)}, np.einsum("p,ptw->tw", scales.astype(np.float64), y64)),
        (y, {"scales": _t(scales), "part_norms": _t(norms), "part_eps": eps}, np.einsum("p,ptw->tw", scales.astype(np.float64), normed)),
        (y, {"part_norms": _t(norms), "part_eps": eps}, normed.sum(0)),
        (y, {"row_scales": _t(row_scales)}, np.einsum("tp,ptw->tw", row_scales.astype(np.float64), y64)),
        (pool, {"rows": _ints(rows), "row_scales": _t(row_scales)}, np.einsum("tp,ptw->tw", row_scales.astype(np.float64), y64)),
    ]
    for given, options, total in forms:
        want = x + mult * total
        for weight in (None, torch.float32, torch.bfloat16):
            stream, out = _t(x), torch.empty((n, width), dtype=out_dtype, device=DEV)
            w = _t(w2).to(weight) if weight else None
            ops.stream_add(stream, _t(given), mult, then=(w, eps, out) if weight else None, **options)
            _close(stream.cpu().numpy(), want, 2e-6)
            if weight:
                _close(out.float().cpu().numpy(), plain.rms_norm(want, w.double().cpu().numpy(), eps), 3e-6 if out_dtype == torch.float32 else 1e-2)


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens", [1, 5, 150])
@pytest.mark.parametrize("width,ff,experts,top", [(64, 24, 6, 2), (40, 33, 5, 5), (64, 40, 3, 1), (36, 16, 12, 4)])
def test_experts_weighted_by_softmax_scores_over_the_chosen(dtype, tokens, width, ff, experts, top):
    """Few tokens (every pair by itself) and many (rows sorted by expert, gathered where they are added up)."""
    from xeno_rt_b200.core import parse_dtype
    from xeno_rt_b200.parts import part_class
    from xeno_rt_b200.parts.context import StepContext
    from xeno_rt_b200.parts.norm import WeightedParts
    rng = np.random.default_rng(tokens + width)
    mk = _matrices(rng)
    params = {"width": width, "inner": ff, "experts": experts, "top": top, "activation": "gated_silu", "routing": "scores",
              "scores": "softmax", "normalize": True, "sum_eps": 1e-20, "router_bias": False}
    w = {"router": mk(experts, width, 4.0)}
    for e in range(experts):
        w.update({f"e{e}.gate": mk(ff, width), f"e{e}.up": mk(ff, width), f"e{e}.down": mk(width, ff)})
    roles = {"router": w["router"], **{f"{r}{e}": w[f"e{e}.{r}"] for e in range(experts) for r in ("gate", "up", "down")}}
    part = part_class("feed_forward", "routed_experts")(params, {r: _t(t).to(DT[dtype]) for r, t in roles.items()}, parse_dtype(dtype), DEV)
    h = _bf16(rng.normal(size=(tokens, width)))
    want = plain.experts_ff(h, w, {"router": {"top": top}})
    ctx = StepContext(n_tokens=tokens, n_seqs=1, token_ids=None, tok_pos=None, tok_slot=None, cu_seqlens=None, seq_slot=None,
                      seq_start=None, new_lens=[tokens], starts=[0], all_single=tokens == 1, max_new=tokens, max_context=tokens,
                      dtype=parse_dtype(dtype))
    add = part_class("add", "scaled")({"width": width, "factor": 0.5}, {}, parse_dtype(dtype), DEV)
    y = part.apply_rows(_t(h).to(DT[dtype]), ctx)
    assert isinstance(y, WeightedParts) and (y.rows is not None) == (tokens * top >= 4 * experts)
    stream = torch.zeros((tokens, width), device=DEV)
    assert add.add_into(stream, y) is None
    tol = 2e-5 if dtype == "float32" else 2e-2
    _close(stream.cpu().numpy(), 0.5 * want, tol)
    summed = part.apply(_t(h).to(DT[dtype]), ctx)
    _close(summed.sum(0).cpu().numpy(), want, tol)
