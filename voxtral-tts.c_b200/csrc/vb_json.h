/*
 * vb_json.h - a small JSON reader for model folders (config.json, the header of a safetensors
 * file). Values are immutable trees; a malformed text is reported, never guessed at.
 */
#ifndef VB_JSON_H
#define VB_JSON_H

#include <stddef.h>

#include <string>
#include <utility>
#include <vector>

namespace vb {

struct Json {
    enum Kind { NIL, BOOL, NUMBER, STRING, ARRAY, OBJECT };
    Kind kind = NIL;
    bool truth = false;
    double number = 0.0;
    std::string text;
    std::vector<Json> items;                            /* ARRAY */
    std::vector<std::pair<std::string, Json>> members;  /* OBJECT, in file order */

    /* Member of an object, or null when it is absent (or this is not an object). A member whose
     * value is JSON null counts as absent. */
    const Json *get(const char *key) const;
};

/* false (and a message) when text[0, n) is not one JSON value. */
bool json_parse(const char *text, size_t n, Json *out, std::string *err);

} // namespace vb

#endif
