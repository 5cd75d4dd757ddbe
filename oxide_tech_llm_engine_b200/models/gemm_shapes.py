"""Launch shapes of the tcgen05 projections, shared by the device models."""
from __future__ import annotations

import os

from .. import ops


class GemmShapes:
    """Mixin: needs `_gemm_cfg` (a dict that caches the choices), `_sms` and `tp`."""

    def _gemm_shape(self, m: int, n: int, k: int, *, swiglu: bool = False, routed: bool = False,
                    store: bool = False) -> dict:
        """Tile width, rows per tile, split-K factor and split-K mode of one projection. Steps of
        129 to 256 rows (large decode batches) keep every row with the CTA that streams a weight
        tile and split K to fill the SMs, combined inside the kernel; a routed projection on one GPU
        adds its splits straight into the fp32 accumulator instead. Other steps use 128-row tiles."""
        key = (m, n, k, swiglu, routed, store)
        c = self._gemm_cfg.get(key)
        if c is not None:
            return c
        # the in-kernel split-K costs about 10 us of partial-tile traffic and barrier: it pays for the
        # large weight streams (gate/up, down), not for the small ones (QKV, O), measured in situ
        big = n * k * 2 >= (48 << 20)
        if 128 < m <= 256 and big and os.environ.get("OXB_DECODE_GEMM", "1") != "0":
            bn, mt, sp = ops.pick_decode_cfg(m, n, k, swiglu=swiglu, sms=self._sms)
            fixup = sp > 1 and not (routed and self.tp == 1)
        else:
            m_tiles = (m + 127) // 128
            bn = ops.pick_bn(n, m_tiles, can_split=not swiglu)
            mt = 1
            sp = 1 if swiglu else ops.pick_splits(m, n, k, bn, self._sms)
            fixup = False
            if sp > 1 and (store or (routed and self.tp > 1)):
                # these epilogues cannot add into an fp32 accumulator: combine the splits in the kernel
                # when the launch is one wave, else do not split
                fits = (((n + bn - 1) // bn) * m_tiles * sp <= self._sms
                        and sp <= ops.max_fixup_splits(bn, 1, False))
                fixup = fits
                if not fits:
                    sp = 1
        c = dict(bn=bn, mt=mt, splits=sp, fixup=fixup)
        self._gemm_cfg[key] = c
        return c
