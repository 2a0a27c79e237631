"""What every model handle of the library (femto_handle) offers, whichever model it holds."""
from __future__ import annotations

import ctypes as C

from . import _lib


class Handle:
    def __init__(self):
        self.h = None

    def refresh_weights(self, theta) -> None:
        _lib.check(_lib.lib().femto_refresh_weights(self.h, _lib.ptr(theta), _lib.stream_ptr()))

    def status_word(self) -> int:
        out = C.c_int32(0)
        _lib.check(_lib.lib().femto_status_word(self.h, C.byref(out)))
        return out.value

    def launch_count(self) -> int:
        return int(_lib.lib().femto_launch_count(self.h))

    def close(self) -> None:
        if self.h:
            _lib.lib().femto_destroy(self.h)
            self.h = None

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass
