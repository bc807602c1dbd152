"""Python face of the decoders whose model is a folder (fc_decoder*): one class for every design. Token ids in,
logits / scores / token ids out; every method is a thin ctypes call into the library.

CudaDecoder has the calls of CudaLlama (caches of one's own) and, on a cache it keeps itself, the three
calls CudaBackend makes of a model: generate_tokens, generate_sampled and score_requests.
"""
import ctypes as C
import weakref

import numpy as np

from . import _lib
from ._lib import FerrumCudaError, check
from .engine import Score, _ids, _ptr, sampling

DEFAULT_CTX = 4096


def probe(path):
    """Sizes of a model folder; validates configuration and tensors without a GPU."""
    info = _lib.FcDecoderInfo()
    check(_lib.lib().fc_decoder_probe(str(path).encode(), C.byref(info)))
    return info


class DecoderCache:
    """What one sequence holds: cached rows and states of every layer, and the position."""

    def __init__(self, model):
        self.model = model
        self._h = C.c_void_p()
        check(_lib.lib().fc_decoder_cache_create(model._h, C.byref(self._h)))
        model._caches.append(weakref.ref(self))

    def close(self):
        if self._h:
            _lib.lib().fc_decoder_cache_free(self._h)
            self._h = C.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def clear(self):
        check(_lib.lib().fc_decoder_cache_clear(self._h))

    def pos(self):
        return _lib.lib().fc_decoder_cache_pos(self._h)

    @property
    def last_decode_ms(self):
        return _lib.lib().fc_decoder_last_decode_ms(self._h)


def dir_architecture(path):
    """Architecture of a model folder, read by the library."""
    buf = C.create_string_buffer(256)
    check(_lib.lib().fc_model_dir_architecture(str(path).encode(), buf, len(buf)))
    return buf.value.decode()


class CudaDecoder:
    """A model folder on one GPU. math_mode: FC_MATH_BF16 or FC_MATH_FP32; ctx: positions a cache holds."""

    architecture = None        # a design's class takes folders of that design only

    def __init__(self, path, device=0, math_mode=_lib.FC_MATH_BF16, ctx=DEFAULT_CTX):
        self._h = C.c_void_p()
        self._caches = []
        self._own = None
        if self.architecture is not None and dir_architecture(path) != self.architecture:
            raise FerrumCudaError(_lib.FC_E_FORMAT, f"{path} holds no {self.architecture} model")
        check(_lib.lib().fc_decoder_load(str(path).encode(), device, math_mode, ctx, C.byref(self._h)))
        self.info = _lib.FcDecoderInfo()
        check(_lib.lib().fc_decoder_get_info(self._h, C.byref(self.info)))

    def close(self):
        self._own = None
        for ref in self._caches:                 # caches go first: they hold device memory of this model's context
            cache = ref()
            if cache is not None:
                cache.close()
        self._caches = []
        if self._h:
            _lib.lib().fc_decoder_free(self._h)
            self._h = C.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def new_cache(self):
        return DecoderCache(self)

    def _cache(self):
        if self._own is None:
            self._own = self.new_cache()
        return self._own

    # ---- forward ---------------------------------------------------------------------------
    def feed(self, ids, cache, want=()):
        """The next tokens of the cache's sequence, any number of them; logits [len(want)][vocab] of the wanted places."""
        ids, want = _ids(ids), _ids(want)
        out = np.empty((want.size, self.info.vocab), dtype=np.float32)
        check(_lib.lib().fc_decoder_feed(cache._h, _ptr(ids), ids.size, _ptr(want) if want.size else None, want.size,
                                         _ptr(out) if want.size else None))
        return out

    def feed_layers(self, ids, cache):
        """One portion; the residual stream after every layer [layers][n][width]."""
        ids = _ids(ids)
        out = np.empty((self.info.n_layers, ids.size, self.info.width), dtype=np.float32)
        check(_lib.lib().fc_decoder_feed_layers(cache._h, _ptr(ids), ids.size, _ptr(out)))
        return out

    def forward_tokens(self, ids):
        """Logits [n][vocab] of a sequence of its own."""
        ids = _ids(ids)
        cache = self._cache()
        cache.clear()
        return self.feed(ids, cache, np.arange(ids.size))

    def forward_one(self, token, cache, want_logits=True):
        return self.feed([token], cache, [0])[0] if want_logits else self.feed([token], cache)

    @property
    def last_forward_ms(self):
        return _lib.lib().fc_decoder_last_forward_ms(self._h)

    # ---- scoring ---------------------------------------------------------------------------
    def score_from(self, ids, start, per_token=False):
        """Score of ids[start..] given what precedes it, in one pass over the sequence."""
        ids = _ids(ids)
        sc = _lib.FcScore()
        lp = np.zeros(max(ids.size - 1, 1), dtype=np.float32)
        gr = np.zeros(max(ids.size - 1, 1), dtype=np.uint8)
        check(_lib.lib().fc_decoder_score(self._cache()._h, _ptr(ids), ids.size, start, C.byref(sc), _ptr(lp), _ptr(gr)))
        score = Score(sc.logprob, sc.n_tokens, bool(sc.greedy))
        return (score, lp[:max(ids.size - 1, 0)], gr[:max(ids.size - 1, 0)].astype(bool)) if per_token else score

    def score_requests(self, requests, batch_windows=0):
        """One Score per (ids, first scored target); batch_windows is the other models' knob and has no meaning here."""
        return [self.score_from(ids, start) for ids, start in requests]

    # ---- generation ------------------------------------------------------------------------
    def _generate(self, prompt, max_new, params, stops, rng_state, cache, cancel_p):
        prompt = _ids(prompt)
        stops_a = np.ascontiguousarray(stops, dtype=np.int32)
        out = np.zeros(max(max_new, 1), dtype=np.int32)
        n_out = C.c_int(0)
        state = C.c_uint64(rng_state)
        rc = _lib.lib().fc_decoder_generate(cache._h, _ptr(prompt), prompt.size, max_new, C.byref(params),
                                            _ptr(stops_a) if stops_a.size else None, stops_a.size, C.byref(state), cancel_p,
                                            _ptr(out), C.byref(n_out))
        return rc, out[:n_out.value].copy(), state.value

    def generate(self, prompt, max_new, params, stops=(), rng_state=1, cache=None, cancel=None):
        """(new token ids, advanced generator state); a stop id ends the generation and is kept."""
        rc, out, state = self._generate(prompt, max_new, params, stops, rng_state, cache or self._cache(),
                                        None if cancel is None else C.cast(C.byref(cancel), C.c_void_p))
        check(rc)
        return out, state

    def generate_sampled(self, prompt, max_tokens, params, rng_state, eos=-1, cancel=None):
        """As CudaSlm.generate_sampled: the end token is not part of the result; cancel is a numpy int32[1]."""
        rc, out, state = self._generate(prompt, max_tokens, params, () if eos < 0 else (eos,), rng_state, self._cache(),
                                        None if cancel is None else _ptr(cancel))
        if rc != _lib.FC_E_CANCELLED:
            check(rc)
        if eos >= 0 and out.size and out[-1] == eos:
            out = out[:-1]
        return out, state

    def generate_tokens(self, prompt, max_tokens, eos=-1, cancel=None):
        """Greedy ids as CudaSlm.generate_tokens: (ids, whether the caller cancelled)."""
        out, _ = self.generate_sampled(prompt, max_tokens, sampling(temperature=0.0), 1, eos=eos, cancel=cancel)
        return out, bool(cancel is not None and int(cancel[0]))


class CudaNurinex(CudaDecoder):
    """Layers of attention with mixed heads, a linear-attention recurrence and a dense feed-forward side by side."""
    architecture = "Nurinex"


class CudaZogevik(CudaDecoder):
    """Layers of windowed attention (latent, or grouped-query with caches that layers may share) and routed experts."""
    architecture = "Zogevik"


__all__ = ["CudaDecoder", "CudaNurinex", "CudaZogevik", "DecoderCache", "dir_architecture", "probe", "FerrumCudaError"]
