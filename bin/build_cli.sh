# Sourced by the programs of this folder, which set $prog: brings that program and the libraries up to date (make, one caller at a
# time) unless they are there already.  The compilers' output goes to standard error.
pkg="$here/gretacore-v3_b200"
if [ ! -x "$pkg/build/$prog" ] || [ ! -f "$pkg/libgreta_host.so" ] || [ ! -f "$pkg/libgreta_cuda.so" ]; then
  mkdir -p "$pkg/build" || exit 1
  (
    flock 9 || exit 1
    exec make -s -C "$pkg/csrc" -j "$(nproc 2>/dev/null || echo 4)" "$pkg/build/$prog" >&2
  ) 9> "$pkg/build/.lock" || exit 1
fi
